// A routed feed-forward: a router that picks `top` of the experts per token, gated experts, experts that hand their
// input through unchanged, and a gate on a shared expert.
//
//   eg_moe_route     logits = R h (float32); s = softmax(logits) over all router outputs; the `top` largest of
//                    s + correction are chosen (ties: the lower index); their weights are s itself, not renormalised.
//                    Also g[t] = sigmoid(w_g . h), the gate of the shared expert, when w_g is given.
//   eg_moe_hidden    a[t, k, :] = silu(G_e h) * (U_e h) for the k-th chosen expert e of token t (skipped for router
//                    outputs >= experts: those stand for the identity)
//   eg_moe_combine   out[t, :] = sum_k weight[t, k] * (D_e a[t, k, :]  or  h[t, :] for an identity choice)
//                                + g[t] * shared[t, :]                   (float32)
//
// eg_moe_hidden and eg_moe_combine read each chosen expert's weights per token: the form for steps of few tokens.
// Where several tokens of a small step may share an expert, eg_moe_matvec takes one expert's rows for all of its (token, choice) pairs
// at once (a warp reads a weight row once for up to four pairs): the first product with its activation, or the second into float32
// rows per pair, which eg_moe_sum adds up per token.
// For steps of many tokens the rows are sorted by expert instead, so that every expert's weights meet all of its rows in
// one grouped product on the tensor cores (eg_gemm_tcgen05_grouped):
//   eg_moe_dispatch  counts the rows of every expert, gives each expert a run of rows that starts at a multiple of 128,
//                    says which expert every tile of 128 rows belongs to, and copies each token's row to its places
//   eg_moe_gather    out[t, :] = sum_k weight[t, k] * (y[row_of[t, k], :] or h[t, :]) + g[t] * shared[t, :]
// The sizes of the runs stay on the device: nothing here waits for the host.
// Products accumulate in float32; the router is float32 throughout.
//
// Variants, each a parameter: `groups` > 1 cuts the outputs into that many equal runs of neighbours, a group counting the sum of its
// two largest s + correction, and only outputs of the `keep` best groups can be chosen (ties: the lower group); `normalize` divides
// a token's weights by their sum (+ 1e-20); `activation` 2 is an expert without a gate, a = gelu(U_e h) (then GU [experts, ff, width]); `scoring` 1 takes s = sigmoid(logits) instead of the softmax (the correction may then be null);
// `activation` 1 is the clamped gate g' = min(g, limit), u' = clamp(u, -limit, limit), a = g' sigmoid(1.702 g') (u' + 1);
// `input_weights` (eg_moe_hidden, eg_moe_dispatch) multiply an expert's INPUT row, expert(w h), and eg_moe_combine / eg_moe_gather
// then get null weights (every term counts once); a null gate adds the shared expert's output as it is.
#include "common.cuh"

namespace {

// grid (token, chunk of eight router outputs): a warp per output computes its logit (the output past the last one is the
// shared expert's gate), so that a step of few tokens still fills the SMs
template <typename T>
__global__ void __launch_bounds__(256) moe_logits_kernel(const T* __restrict__ h, long long ld, const float* __restrict__ router,
                                                         const float* __restrict__ gate_w, float* __restrict__ logits, float* __restrict__ gate, int width,
                                                         int outputs) {
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int e = blockIdx.y * (blockDim.x >> 5) + warp;
    if (e >= outputs + (gate_w ? 1 : 0)) return;
    const float* w = e < outputs ? router + (size_t)e * width : gate_w;
    const T* row = h + (size_t)t * ld;
    float acc = 0.f;
#pragma unroll 8
    for (int j = lane; j < width; j += 32) acc = fmaf(w[j], to_f32<T>(row[j]), acc);
    acc = warp_sum(acc);
    if (lane == 0) {
        if (e < outputs) logits[(size_t)t * outputs + e] = acc;
        else gate[t] = 1.0f / (1.0f + expf(-acc));
    }
}

// The same for steps of many tokens (bfloat16 rows, widths that are multiples of 64): a block computes 32 tokens x 32 outputs, 2 x 4 of
// them a thread, from tiles of 64 input channels in shared memory, the next tile's loads in flight meanwhile; every logit is one
// running sum over the channels in order, in float32.
__global__ void __launch_bounds__(128) moe_logits_tiled_kernel(const bf16* __restrict__ h, long long ld, const float* __restrict__ router,
                                                               const float* __restrict__ gate_w, float* __restrict__ logits, float* __restrict__ gate, int tokens,
                                                               int width, int outputs) {
    constexpr int CH = 64;
    __shared__ __align__(16) float hs[CH][34], ws[CH][36];        // [channel][token], [channel][output]
    const int t0 = blockIdx.x * 32, e0 = blockIdx.y * 32, all = outputs + (gate_w ? 1 : 0);
    const int tx = threadIdx.x & 7, ty = threadIdx.x >> 3;        // outputs 4 tx .. + 3, tokens 2 ty, 2 ty + 1
    // what this thread brings in: channels 16 part .. + 15 of one token and one output (the last ones again past the end)
    const int row = threadIdx.x >> 2, part = threadIdx.x & 3;
    const int e = min(e0 + row, all - 1);
    const uint4* hsrc = reinterpret_cast<const uint4*>(h + (size_t)min(t0 + row, tokens - 1) * ld + 16 * part);
    const float4* wsrc = reinterpret_cast<const float4*>((e < outputs ? router + (size_t)e * width : gate_w) + 16 * part);
    float acc[2][4] = {};
    uint4 hn[2];
    float4 wn[4];
    auto fetch = [&](int c0) {
#pragma unroll
        for (int i = 0; i < 2; ++i) hn[i] = __ldg(hsrc + c0 / 8 + i);
#pragma unroll
        for (int i = 0; i < 4; ++i) wn[i] = __ldg(wsrc + c0 / 4 + i);
    };
    fetch(0);
    for (int c0 = 0; c0 < width; c0 += CH) {
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float2 f = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&hn[i])[q]);
                hs[16 * part + 8 * i + 2 * q][row] = f.x;
                hs[16 * part + 8 * i + 2 * q + 1][row] = f.y;
            }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            ws[16 * part + 4 * i][row] = wn[i].x;
            ws[16 * part + 4 * i + 1][row] = wn[i].y;
            ws[16 * part + 4 * i + 2][row] = wn[i].z;
            ws[16 * part + 4 * i + 3][row] = wn[i].w;
        }
        __syncthreads();
        if (c0 + CH < width) fetch(c0 + CH);
#pragma unroll 16
        for (int c = 0; c < CH; ++c) {
            const float2 a = *reinterpret_cast<const float2*>(&hs[c][2 * ty]);
            const float4 b = *reinterpret_cast<const float4*>(&ws[c][4 * tx]);
            acc[0][0] = fmaf(a.x, b.x, acc[0][0]);
            acc[0][1] = fmaf(a.x, b.y, acc[0][1]);
            acc[0][2] = fmaf(a.x, b.z, acc[0][2]);
            acc[0][3] = fmaf(a.x, b.w, acc[0][3]);
            acc[1][0] = fmaf(a.y, b.x, acc[1][0]);
            acc[1][1] = fmaf(a.y, b.y, acc[1][1]);
            acc[1][2] = fmaf(a.y, b.z, acc[1][2]);
            acc[1][3] = fmaf(a.y, b.w, acc[1][3]);
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = t0 + 2 * ty + i, o = e0 + 4 * tx + j;
            if (t >= tokens || o >= all) continue;
            if (o < outputs) logits[(size_t)t * outputs + o] = acc[i][j];
            else gate[t] = 1.0f / (1.0f + expf(-acc[i][j]));
        }
}

// a warp per token: softmax over the logits, then the `top` largest of score + correction, within the
// `keep` best groups; shared memory: `outputs` floats per warp (the scores), and `groups` more (with groups > 1)
__global__ void __launch_bounds__(128) moe_select_kernel(const float* __restrict__ logits, const float* __restrict__ correction, int* __restrict__ ids,
                                                         float* __restrict__ weights, int tokens, int outputs, int top, int scoring, int groups, int keep,
                                                         int normalize) {
    extern __shared__ float group_scores[];
    const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= tokens) return;
    float* logit = group_scores + (size_t)(threadIdx.x >> 5) * (outputs + groups);
    const float* from = logits + (size_t)t * outputs;
    for (int e = lane; e < outputs; e += 32) logit[e] = from[e];
    __syncwarp();
    if (scoring == 1) {
        for (int e = lane; e < outputs; e += 32) logit[e] = 1.0f / (1.0f + expf(-logit[e]));      // now the scores s
    } else {
        float top_logit = -INFINITY;
        for (int e = lane; e < outputs; e += 32) top_logit = fmaxf(top_logit, logit[e]);
        top_logit = warp_max(top_logit);
        float sum = 0.f;
        for (int e = lane; e < outputs; e += 32) sum += expf(logit[e] - top_logit);
        sum = warp_sum(sum);
        for (int e = lane; e < outputs; e += 32) logit[e] = expf(logit[e] - top_logit) / sum;      // now the scores s
    }
    __syncwarp();
    const int per = outputs / groups;
    float* group = logit + outputs;
    if (groups > 1) {
        const bool in_step = per <= 32 && (per & (per - 1)) == 0;
        if (in_step) {                           // a lane per output: the two largest of a run by halving
            for (int e0 = 0; e0 < outputs; e0 += 32) {
                const int e = e0 + lane;
                float first = e < outputs ? logit[e] + (correction ? correction[e] : 0.f) : -INFINITY, second = -INFINITY;
                for (int o = 1; o < per; o <<= 1) {
                    const float of = __shfl_xor_sync(0xffffffffu, first, o), os = __shfl_xor_sync(0xffffffffu, second, o);
                    second = fmaxf(fminf(first, of), fmaxf(second, os));
                    first = fmaxf(first, of);
                }
                if (e < outputs && (lane & (per - 1)) == 0) group[e / per] = per > 1 ? first + second : first;
            }
        }
        for (int g = lane; !in_step && g < groups; g += 32) {
            float first = -INFINITY, second = -INFINITY;
            for (int e = g * per; e < (g + 1) * per; ++e) {
                const float v = logit[e] + (correction ? correction[e] : 0.f);
                if (v > first) { second = first; first = v; }
                else if (v > second) second = v;
            }
            group[g] = per > 1 ? first + second : first;
        }
        __syncwarp();
        unsigned long long kept = 0ull;          // bit i for the lane's group lane + 32 i: fewer than `keep` groups come before it
        for (int g = lane, i = 0; g < groups; g += 32, ++i) {
            const float mine = group[g];
            int before = 0;
            for (int o = 0; o < groups; ++o) before += group[o] > mine || (group[o] == mine && o < g);
            if (before < keep) kept |= 1ull << i;
        }
        __syncwarp();
        for (int g = lane, i = 0; g < groups; g += 32, ++i) group[g] = (kept >> i) & 1ull ? 1.f : 0.f;
        __syncwarp();
    }
    float sum_chosen = 0.f, my_weight = 0.f;
    int my_id = 0;
    unsigned long long taken = 0ull;             // a lane tracks which of its own outputs are taken: bit k for e = lane + 32 k
    if (groups > 1)                              // outputs of the groups that are left out count as taken
        for (int e = lane, i = 0; e < outputs; e += 32, ++i)
            if (group[e / per] == 0.f) taken |= 1ull << i;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int arg = 0x7fffffff;
        for (int e = lane, i = 0; e < outputs; e += 32, ++i) {
            if ((taken >> i) & 1ull) continue;
            const float v = logit[e] + (correction ? correction[e] : 0.f);
            if (v > best) { best = v; arg = e; }
        }
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
            if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
        }
        if (arg != 0x7fffffff && arg % 32 == lane) taken |= 1ull << (arg / 32);
        // choice k stays with lane k % 32 until 32 of them are written together; the sum is every lane's (the scores lie in shared memory)
        const float s = arg == 0x7fffffff ? 0.f : logit[arg];
        sum_chosen += s;
        if (k % 32 == lane) {
            my_id = arg == 0x7fffffff ? outputs : arg;
            my_weight = s;
        }
        if (k % 32 == 31 || k == top - 1) {
            const int at = k / 32 * 32 + lane;
            if (at <= k) {
                ids[(size_t)t * top + at] = my_id;
                weights[(size_t)t * top + at] = normalize && top <= 32 ? my_weight / (sum_chosen + 1e-20f) : my_weight;
            }
        }
    }
    if (normalize && top > 32) {
        __syncwarp();
        for (int k = lane; k < top; k += 32) weights[(size_t)t * top + k] /= sum_chosen + 1e-20f;       // each lane what it wrote itself
    }
}

// grid (token, choice, chunk of ff); a warp per hidden unit; GU [experts, 2 ff, width] with the gate row of unit f at
// 2 f and its up row at 2 f + 1, or without a gate (GATED false) [experts, ff, width]
template <typename T, bool GATED>
__global__ void __launch_bounds__(256) moe_hidden_kernel(const T* __restrict__ h, long long ld, const T* __restrict__ GU, const int* __restrict__ ids,
                                                         const float* __restrict__ input_weights, T* __restrict__ act, int width, int ff, int top,
                                                         int experts, int activation, float limit) {
    extern __shared__ float row[];
    const int t = blockIdx.x, k = blockIdx.y;
    const int e = ids[(size_t)t * top + k];
    if (e >= experts) return;
    for (int j = threadIdx.x; j < width; j += blockDim.x) row[j] = to_f32<T>(h[(size_t)t * ld + j]);
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int f = blockIdx.z * warps + warp;
    if (f >= ff) return;
    const T* g = GU + (GATED ? (size_t)e * 2 * ff + 2 * f : (size_t)e * ff + f) * width;
    const T* u = GATED ? g + width : g;
    float ag = 0.f, au = 0.f;
    if (sizeof(T) == 2 && width % 8 == 0) {                      // eight weights a load
        const uint4* g8 = reinterpret_cast<const uint4*>(g);
        const uint4* u8 = reinterpret_cast<const uint4*>(u);
#pragma unroll 2
        for (int j = lane; j < width / 8; j += 32) {
            const uint4 gv = g8[j], uv = GATED ? u8[j] : gv;
            const __nv_bfloat162* gp = reinterpret_cast<const __nv_bfloat162*>(&gv);
            const __nv_bfloat162* up = reinterpret_cast<const __nv_bfloat162*>(&uv);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float2 gf = __bfloat1622float2(gp[q]), uf = __bfloat1622float2(up[q]);
                ag = fmaf(gf.x, row[8 * j + 2 * q], ag);
                ag = fmaf(gf.y, row[8 * j + 2 * q + 1], ag);
                if (GATED) {
                    au = fmaf(uf.x, row[8 * j + 2 * q], au);
                    au = fmaf(uf.y, row[8 * j + 2 * q + 1], au);
                }
            }
        }
    } else {
        for (int j = lane; j < width; j += 32) {
            ag = fmaf(to_f32<T>(g[j]), row[j], ag);
            if (GATED) au = fmaf(to_f32<T>(u[j]), row[j], au);
        }
    }
    ag = warp_sum(ag);
    if (GATED) au = warp_sum(au);
    if (input_weights) {                                         // the expert reads w h: its two products are w times these
        const float wgt = input_weights[(size_t)t * top + k];
        ag *= wgt;
        au *= wgt;
    }
    float a;
    if (!GATED) {
        a = gelu_erf(ag);
    } else if (activation == 1) {
        ag = fminf(ag, limit);
        au = fminf(fmaxf(au, -limit), limit);
        a = ag / (1.0f + expf(-1.702f * ag)) * (au + 1.0f);
    } else {
        a = ag / (1.0f + expf(-ag)) * au;
    }
    if (lane == 0) act[((size_t)t * top + k) * ff + f] = from_f32<T>(a);
}

// grid (token, chunk of width); a warp per output value; Dn [experts, width, ff]
template <typename T>
__global__ void __launch_bounds__(256) moe_combine_kernel(const T* __restrict__ h, long long ld, const T* __restrict__ act, const T* __restrict__ Dn,
                                                          const int* __restrict__ ids, const float* __restrict__ weights, const void* __restrict__ shared,
                                                          int shared_dtype, const float* __restrict__ gate, float* __restrict__ out, int width, int ff,
                                                          int top, int experts) {
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int j = blockIdx.y * warps + warp;
    if (j >= width) return;
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
        const int e = ids[(size_t)t * top + k];
        const float wgt = weights ? weights[(size_t)t * top + k] : 1.0f;
        if (e >= experts) {
            total += wgt * to_f32<T>(h[(size_t)t * ld + j]);
            continue;
        }
        const T* d = Dn + ((size_t)e * width + j) * ff;
        const T* a = act + ((size_t)t * top + k) * ff;
        float acc = 0.f;
        if (sizeof(T) == 2 && ff % 8 == 0) {                     // eight weights a load
            const uint4* d8 = reinterpret_cast<const uint4*>(d);
            const uint4* a8 = reinterpret_cast<const uint4*>(a);
#pragma unroll 2
            for (int f = lane; f < ff / 8; f += 32) {
                const uint4 dv = d8[f], av = a8[f];
                const __nv_bfloat162* dp = reinterpret_cast<const __nv_bfloat162*>(&dv);
                const __nv_bfloat162* ap = reinterpret_cast<const __nv_bfloat162*>(&av);
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const float2 df = __bfloat1622float2(dp[q]), af = __bfloat1622float2(ap[q]);
                    acc = fmaf(df.x, af.x, acc);
                    acc = fmaf(df.y, af.y, acc);
                }
            }
        } else {
            for (int f = lane; f < ff; f += 32) acc = fmaf(to_f32<T>(d[f]), to_f32<T>(a[f]), acc);
        }
        total += wgt * warp_sum(acc);
    }
    if (shared) {
        const size_t i = (size_t)t * width + j;
        total += (gate ? gate[t] : 1.0f) * (shared_dtype == EG_BF16 ? __bfloat162float(((const bf16*)shared)[i]) : ((const float*)shared)[i]);
    }
    if (lane == 0) out[(size_t)t * width + j] = total;
}

}  // namespace

// ids [T, top] int32 (router outputs; those >= the number of experts stand for the identity), weights [T, top] float32,
// gate [T] float32 (only with gate_w); logits [T, outputs] float32 is scratch
EG_API int eg_moe_route(cudaStream_t stream, int dtype, const void* h, long long ld, const float* router, const float* correction, const float* gate_w,
                        float* logits, int* ids, float* weights, float* gate, int tokens, int width, int outputs, int top, int scoring, int groups, int keep,
                        int normalize) {
    if (tokens <= 0) return 0;
    if (groups < 1 || outputs % groups || keep < 1 || keep > groups) return (int)cudaErrorInvalidValue;
    if (top < 1 || top > outputs || outputs > 2048 || !logits || scoring < 0 || scoring > 1) return (int)cudaErrorInvalidValue;
    const int all = outputs + (gate_w ? 1 : 0);
    dim3 grid(tokens, (all + 7) / 8), tiled((tokens + 31) / 32, (all + 31) / 32);
    // as many tokens as make the tiles fill a good part of the SMs
    if (tokens >= 256 && dtype == EG_BF16 && width % 64 == 0 && ld % 8 == 0 && (uintptr_t)h % 16 == 0 && (uintptr_t)router % 16 == 0 && (uintptr_t)gate_w % 16 == 0)
        moe_logits_tiled_kernel<<<tiled, 128, 0, stream>>>((const bf16*)h, ld, router, gate_w, logits, gate, tokens, width, outputs);
    else if (dtype == EG_BF16) moe_logits_kernel<bf16><<<grid, 256, 0, stream>>>((const bf16*)h, ld, router, gate_w, logits, gate, width, outputs);
    else moe_logits_kernel<float><<<grid, 256, 0, stream>>>((const float*)h, ld, router, gate_w, logits, gate, width, outputs);
    const size_t smem = (size_t)4 * (outputs + groups) * sizeof(float);
    if (smem > 48 * 1024) {
        static bool configured = false;
        if (!configured) {
            const cudaError_t e = cudaFuncSetAttribute(moe_select_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 4 * 2 * 2048 * (int)sizeof(float));
            if (e != cudaSuccess) return (int)e;
            configured = true;
        }
    }
    moe_select_kernel<<<(tokens + 3) / 4, 128, smem, stream>>>(logits, correction, ids, weights, tokens, outputs, top, scoring, groups, keep, normalize);
    return eg_launch_status();
}

// act [T, top, ff] in the compute dtype; rows of identity choices (ids >= experts) are left untouched
EG_API int eg_moe_hidden(cudaStream_t stream, int dtype, const void* h, long long ld, const void* gate_up, const int* ids, const float* input_weights,
                         void* act, int tokens, int width, int ff, int top, int experts, int activation, float limit) {
    if (tokens <= 0 || experts <= 0) return 0;
    const size_t smem = (size_t)width * sizeof(float);
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    dim3 grid(tokens, top, (ff + 7) / 8);
#define EG_HIDDEN(T, G) moe_hidden_kernel<T, G><<<grid, 256, smem, stream>>>((const T*)h, ld, (const T*)gate_up, ids, input_weights, (T*)act, width, ff, top, experts, activation, limit)
    if (dtype == EG_BF16) { if (activation == 2) EG_HIDDEN(bf16, false); else EG_HIDDEN(bf16, true); }
    else { if (activation == 2) EG_HIDDEN(float, false); else EG_HIDDEN(float, true); }
#undef EG_HIDDEN
    return eg_launch_status();
}

// out [T, width] float32; shared [T, width] (shared_dtype) with gate [T], or null
EG_API int eg_moe_combine(cudaStream_t stream, int dtype, const void* h, long long ld, const void* act, const void* down, const int* ids,
                          const float* weights, const void* shared, int shared_dtype, const float* gate, float* out, int tokens, int width, int ff,
                          int top, int experts) {
    if (tokens <= 0) return 0;
    dim3 grid(tokens, (width + 7) / 8);
    if (dtype == EG_BF16)
        moe_combine_kernel<bf16><<<grid, 256, 0, stream>>>((const bf16*)h, ld, (const bf16*)act, (const bf16*)down, ids, weights, shared, shared_dtype, gate,
                                                          out, width, ff, top, experts);
    else
        moe_combine_kernel<float><<<grid, 256, 0, stream>>>((const float*)h, ld, (const float*)act, (const float*)down, ids, weights, shared, shared_dtype,
                                                           gate, out, width, ff, top, experts);
    return eg_launch_status();
}

namespace {
// One expert's matrix [rows, K] for all pairs that chose it (bfloat16).  grid (blocks of 32 rows, expert); a warp works on four rows by
// itself: it looks at all ids, and takes up to four of its expert's pairs at a time (their input rows come from the L1, which the
// block's warps share; the weights pass it by).  MODE 0: rows interleaved (gate, up), out bfloat16 [pairs, rows / 2] with the gate's
// activation; 1: out bfloat16 [pairs, rows] = gelu; 2: out float32 [pairs, rows].  A dot product is one running sum per lane over its
// pieces of eight channels in order, then a sum over the lanes: the same for a pair whatever else chose the expert.
constexpr int MATVEC_PAIRS = 4, MATVEC_MOST = 512;
__device__ __forceinline__ uint4 load_once(const uint4* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];\n" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
template <int NP>
__device__ __forceinline__ void matvec_rows(const uint4* const (&w)[4], const uint4* const (&x)[MATVEC_PAIRS], int pieces, int lane, float (&acc)[4][MATVEC_PAIRS]) {
#pragma unroll 2
    for (int c = lane; c < pieces; c += 32) {
        uint4 wv[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) wv[r] = load_once(w[r] + c);
#pragma unroll
        for (int p = 0; p < NP; ++p) {
            const uint4 xv = __ldg(x[p] + c);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float2 xf = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&xv)[q]);
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    const float2 wf = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&wv[r])[q]);
                    acc[r][p] = fmaf(wf.x, xf.x, acc[r][p]);
                    acc[r][p] = fmaf(wf.y, xf.y, acc[r][p]);
                }
            }
        }
    }
}
template <int MODE>
__global__ void __launch_bounds__(256) moe_matvec_kernel(const bf16* __restrict__ xs, long long ldx, int pairs_per_row, const bf16* __restrict__ W,
                                                            const int* __restrict__ ids, const float* __restrict__ input_weights, void* __restrict__ out, int pairs,
                                                            int rows, int K, int activation, float limit) {
    const int e = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r0 = (blockIdx.x * 8 + warp) * 4, pieces = K / 8;
    if (r0 >= rows) return;
    // bit i of a lane's mask: pair lane + 32 i chose this expert
    unsigned mine = 0;
    for (int i = 0; lane + 32 * i < pairs; ++i) mine |= (unsigned)(ids[lane + 32 * i] == e) << i;
    if (!__any_sync(0xffffffffu, mine)) return;
    const uint4* w[4];
#pragma unroll
    for (int r = 0; r < 4; ++r) w[r] = reinterpret_cast<const uint4*>(W + ((size_t)e * rows + min(r0 + r, rows - 1)) * K);
    while (true) {
        // up to four pairs, lowest first
        int pair[MATVEC_PAIRS], np = 0;
        const uint4* x[MATVEC_PAIRS];
#pragma unroll
        for (int p = 0; p < MATVEC_PAIRS; ++p) {
            const unsigned first = mine ? (unsigned)((__ffs(mine) - 1) * 32 + lane) : 0xffffffffu;
            const unsigned lowest = __reduce_min_sync(0xffffffffu, first);
            pair[p] = (int)lowest;
            x[p] = reinterpret_cast<const uint4*>(xs);
            if (lowest == 0xffffffffu) continue;
            if (first == lowest) mine &= mine - 1;
            x[p] = reinterpret_cast<const uint4*>(xs + (size_t)(lowest / pairs_per_row) * ldx);
            ++np;
        }
        if (np == 0) break;
        float acc[4][MATVEC_PAIRS] = {};
        if (np == 1) matvec_rows<1>(w, x, pieces, lane, acc);
        else if (np == 2) matvec_rows<2>(w, x, pieces, lane, acc);
        else matvec_rows<4>(w, x, pieces, lane, acc);
#pragma unroll
        for (int p = 0; p < MATVEC_PAIRS; ++p) {
            if (p >= np) break;
            float v[4];
#pragma unroll
            for (int r = 0; r < 4; ++r) v[r] = warp_sum(acc[r][p]);
            if (input_weights) {
#pragma unroll
                for (int r = 0; r < 4; ++r) v[r] *= input_weights[pair[p]];
            }
            if (MODE == 0) {                                      // lanes 0 and 1 hold a hidden unit each
                float g = lane == 0 ? v[0] : v[2], u = lane == 0 ? v[1] : v[3], a;
                if (activation == 1) {
                    g = fminf(g, limit);
                    u = fminf(fmaxf(u, -limit), limit);
                    a = g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
                } else {
                    a = g / (1.0f + expf(-g)) * u;
                }
                if (lane < 2 && r0 + 2 * lane + 1 < rows) ((bf16*)out)[(size_t)pair[p] * (rows / 2) + r0 / 2 + lane] = __float2bfloat16_rn(a);
            } else {
                const float y = lane == 0 ? v[0] : lane == 1 ? v[1] : lane == 2 ? v[2] : v[3];
                if (lane < 4 && r0 + lane < rows) {
                    if (MODE == 1) ((bf16*)out)[(size_t)pair[p] * rows + r0 + lane] = __float2bfloat16_rn(gelu_erf(y));
                    else ((float*)out)[(size_t)pair[p] * rows + r0 + lane] = y;
                }
            }
        }
        if (np < MATVEC_PAIRS) break;
    }
}

// out[t] = sum_k weight[t, k] * (y[t, k] or h[t] for an identity choice) + gate[t] * shared[t], four columns a thread
__global__ void __launch_bounds__(256) moe_sum_kernel(const float* __restrict__ y, const int* __restrict__ ids, const float* __restrict__ weights,
                                                      const bf16* __restrict__ h, long long ld, const void* __restrict__ shared, int shared_dtype,
                                                      const float* __restrict__ gate, float* __restrict__ out, int width, int top, int experts) {
    const int t = blockIdx.x, j = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
    if (j >= width) return;
    float4 total = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int k = 0; k < top; ++k) {
        const float w = weights ? weights[(size_t)t * top + k] : 1.0f;
        float4 v;
        if (ids[(size_t)t * top + k] >= experts) {
            const uint2 raw = *reinterpret_cast<const uint2*>(h + (size_t)t * ld + j);
            const float2 a = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&raw)[0]), b = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&raw)[1]);
            v = make_float4(a.x, a.y, b.x, b.y);
        } else {
            v = *reinterpret_cast<const float4*>(y + ((size_t)t * top + k) * width + j);
        }
        total.x = fmaf(w, v.x, total.x);
        total.y = fmaf(w, v.y, total.y);
        total.z = fmaf(w, v.z, total.z);
        total.w = fmaf(w, v.w, total.w);
    }
    if (shared) {
        const float g = gate ? gate[t] : 1.0f;
        const size_t i = (size_t)t * width + j;
        float4 v;
        if (shared_dtype == EG_BF16) {
            const uint2 raw = *reinterpret_cast<const uint2*>((const bf16*)shared + i);
            const float2 a = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&raw)[0]), b = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&raw)[1]);
            v = make_float4(a.x, a.y, b.x, b.y);
        } else {
            v = *reinterpret_cast<const float4*>((const float*)shared + i);
        }
        total.x = fmaf(g, v.x, total.x);
        total.y = fmaf(g, v.y, total.y);
        total.z = fmaf(g, v.z, total.z);
        total.w = fmaf(g, v.w, total.w);
    }
    *reinterpret_cast<float4*>(out + (size_t)t * width + j) = total;
}
}  // namespace

// mode: see moe_matvec_kernel.  x bfloat16: row i / pairs_per_row belongs to pair i; W [experts, rows, K]; `activation` and `limit` as in
// eg_moe_hidden (mode 0).  Takes K % 8 == 0, 16-byte aligned rows, at most 512 pairs; anything else: cudaErrorInvalidValue.
EG_API int eg_moe_matvec(cudaStream_t stream, int mode, const void* x, long long ldx, int pairs_per_row, const void* W, const int* ids, const float* input_weights,
                         void* out, int pairs, int rows, int K, int experts, int activation, float limit) {
    if (pairs <= 0 || experts <= 0) return 0;
    if (mode < 0 || mode > 2 || K % 8 || ldx % 8 || pairs > MATVEC_MOST || pairs_per_row < 1 || rows < 1 || (mode == 0 && rows % 2) || (uintptr_t)x % 16 ||
        (uintptr_t)W % 16)
        return (int)cudaErrorInvalidValue;
    dim3 grid((rows + 31) / 32, experts);
#define EG_MATVEC(M) \
    moe_matvec_kernel<M><<<grid, 256, 0, stream>>>((const bf16*)x, ldx, pairs_per_row, (const bf16*)W, ids, input_weights, out, pairs, rows, K, activation, limit)
    if (mode == 0) EG_MATVEC(0);
    else if (mode == 1) EG_MATVEC(1);
    else EG_MATVEC(2);
#undef EG_MATVEC
    return eg_launch_status();
}

// out [T, width] float32 from y float32 [T, top, width]; width % 4 == 0
EG_API int eg_moe_sum(cudaStream_t stream, const float* y, const int* ids, const float* weights, const void* h, long long ld, const void* shared, int shared_dtype,
                      const float* gate, float* out, int tokens, int width, int top, int experts) {
    if (tokens <= 0) return 0;
    if (width % 4 || ld % 4) return (int)cudaErrorInvalidValue;
    moe_sum_kernel<<<dim3(tokens, (width / 4 + 255) / 256), 256, 0, stream>>>(y, ids, weights, (const bf16*)h, ld, shared, shared_dtype, gate, out, width, top,
                                                                             experts);
    return eg_launch_status();
}

namespace {
__global__ void moe_count_kernel(const int* __restrict__ ids, int* __restrict__ counts, int pairs, int experts) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < pairs && ids[i] < experts) atomicAdd(&counts[ids[i]], 1);
}
// one block: starts[e] = first row of expert e's run (runs padded to 128 rows), cursors to zero, tiles labelled
__global__ void moe_offsets_kernel(const int* __restrict__ counts, int* __restrict__ starts, int* __restrict__ cursors, int* __restrict__ tile_group,
                                   int experts, int max_tiles) {
    for (int i = threadIdx.x; i < max_tiles; i += blockDim.x) tile_group[i] = -1;
    if (threadIdx.x == 0) {
        int at = 0;
        for (int e = 0; e < experts; ++e) {
            starts[e] = at;
            at += (counts[e] + 127) / 128 * 128;
        }
        starts[experts] = at;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < experts; e += blockDim.x) {
        cursors[e] = 0;
        for (int tile = starts[e] / 128; tile < starts[e + 1] / 128 && tile < max_tiles; ++tile) tile_group[tile] = e;
    }
}
// a warp per (token, choice): takes the next row of the expert's run and copies the token's row there
__global__ void __launch_bounds__(256) moe_scatter_kernel(const bf16* __restrict__ h, long long ld, const int* __restrict__ ids, const int* __restrict__ starts,
                                                          int* __restrict__ cursors, int* __restrict__ row_of, bf16* __restrict__ rows,
                                                          const float* __restrict__ input_weights, int pairs, int width, int top, int experts, int max_rows) {
    const int pair = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (pair >= pairs) return;
    const int e = ids[pair];
    if (e >= experts) {
        if (lane == 0) row_of[pair] = -1;
        return;
    }
    int row = 0;
    if (lane == 0) {
        row = starts[e] + atomicAdd(&cursors[e], 1);
        if (row >= max_rows) row = -1;
        row_of[pair] = row;
    }
    row = __shfl_sync(0xffffffffu, row, 0);
    if (row < 0) return;
    const bf16* src = h + (size_t)(pair / top) * ld;
    bf16* dst = rows + (size_t)row * width;
    if (input_weights) {                                        // the expert's input is the row times the pair's weight
        const float wgt = input_weights[pair];
        for (int j = lane; j < width; j += 32) dst[j] = __float2bfloat16_rn(wgt * __bfloat162float(src[j]));
    } else if (width % 8 == 0 && ld % 8 == 0) {
        for (int j = lane; j < width / 8; j += 32) reinterpret_cast<uint4*>(dst)[j] = reinterpret_cast<const uint4*>(src)[j];
    } else {
        for (int j = lane; j < width; j += 32) dst[j] = src[j];
    }
}
// eight columns a thread (widths and strides that are multiples of eight): the rows are read and written 16 bytes at a time
__global__ void __launch_bounds__(256) moe_gather_vec_kernel(const bf16* __restrict__ y, const int* __restrict__ row_of, const int* __restrict__ ids,
                                                             const float* __restrict__ weights, const bf16* __restrict__ h, long long ld,
                                                             const void* __restrict__ shared, int shared_dtype, const float* __restrict__ gate,
                                                             float* __restrict__ out, int tokens, int width, int top, int experts) {
    const int groups = width / 8;
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * groups) return;
    const int t = (int)(i / groups), j = (int)(i % groups) * 8;
    float total[8] = {};
#pragma unroll 4
    for (int k = 0; k < top; ++k) {
        const size_t pair = (size_t)t * top + k;
        const float wgt = weights ? weights[pair] : 1.0f;
        const bf16* src = nullptr;
        if (ids[pair] >= experts) src = h + (size_t)t * ld + j;
        else if (row_of[pair] >= 0) src = y + (size_t)row_of[pair] * width + j;
        if (!src) continue;
        const uint4 raw = *reinterpret_cast<const uint4*>(src);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const float2 f = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&raw)[q]);
            total[2 * q] += wgt * f.x;
            total[2 * q + 1] += wgt * f.y;
        }
    }
    const size_t at = (size_t)t * width + j;
    if (shared) {
        const float g = gate ? gate[t] : 1.0f;
        if (shared_dtype == EG_BF16) {
            const uint4 raw = *reinterpret_cast<const uint4*>((const bf16*)shared + at);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float2 f = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&raw)[q]);
                total[2 * q] += g * f.x;
                total[2 * q + 1] += g * f.y;
            }
        } else {
            const float4 a = reinterpret_cast<const float4*>((const float*)shared + at)[0], b = reinterpret_cast<const float4*>((const float*)shared + at)[1];
            total[0] += g * a.x; total[1] += g * a.y; total[2] += g * a.z; total[3] += g * a.w;
            total[4] += g * b.x; total[5] += g * b.y; total[6] += g * b.z; total[7] += g * b.w;
        }
    }
    float4* dst = reinterpret_cast<float4*>(out + at);
    dst[0] = make_float4(total[0], total[1], total[2], total[3]);
    dst[1] = make_float4(total[4], total[5], total[6], total[7]);
}
__global__ void moe_gather_kernel(const bf16* __restrict__ y, const int* __restrict__ row_of, const int* __restrict__ ids, const float* __restrict__ weights,
                                  const bf16* __restrict__ h, long long ld, const void* __restrict__ shared, int shared_dtype, const float* __restrict__ gate,
                                  float* __restrict__ out, int tokens, int width, int top, int experts) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * width) return;
    const int t = (int)(i / width), j = (int)(i % width);
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
        const int e = ids[(size_t)t * top + k];
        const float wgt = weights ? weights[(size_t)t * top + k] : 1.0f;
        if (e >= experts) total += wgt * __bfloat162float(h[(size_t)t * ld + j]);
        else {
            const int row = row_of[(size_t)t * top + k];
            if (row >= 0) total += wgt * __bfloat162float(y[(size_t)row * width + j]);
        }
    }
    if (shared) total += (gate ? gate[t] : 1.0f) * (shared_dtype == EG_BF16 ? __bfloat162float(((const bf16*)shared)[i]) : ((const float*)shared)[i]);
    out[i] = total;
}
}  // namespace

// Sorts the step's (token, choice) pairs by expert (bfloat16 rows).  counts, cursors [experts] and starts [experts + 1] are
// scratch; tile_group [max_rows / 128] and row_of [tokens * top] are results, rows [max_rows, width] receives the copies.
// max_rows: a multiple of 128, at least tokens * top rounded up to 128 plus 128 per expert.
EG_API int eg_moe_dispatch(cudaStream_t stream, const void* h, long long ld, const int* ids, const float* input_weights, int* counts, int* starts, int* cursors,
                           int* tile_group, int* row_of, void* rows, int tokens, int width, int top, int experts, int max_rows) {
    const int pairs = tokens * top;
    if (pairs <= 0 || experts <= 0) return 0;
    if (max_rows % 128 || max_rows < (pairs + 127) / 128 * 128 + 128 * experts || experts > 2048) return (int)cudaErrorInvalidValue;
    cudaError_t e = cudaMemsetAsync(counts, 0, (size_t)experts * sizeof(int), stream);
    if (e != cudaSuccess) return (int)e;
    moe_count_kernel<<<(pairs + 255) / 256, 256, 0, stream>>>(ids, counts, pairs, experts);
    moe_offsets_kernel<<<1, 256, 0, stream>>>(counts, starts, cursors, tile_group, experts, max_rows / 128);
    moe_scatter_kernel<<<(pairs + 7) / 8, 256, 0, stream>>>((const bf16*)h, ld, ids, starts, cursors, row_of, (bf16*)rows, input_weights, pairs, width, top, experts, max_rows);
    return eg_launch_status();
}

// out [T, width] float32 from the experts' outputs y [max_rows, width] (bfloat16) in sorted order
EG_API int eg_moe_gather(cudaStream_t stream, const void* y, const int* row_of, const int* ids, const float* weights, const void* h, long long ld,
                         const void* shared, int shared_dtype, const float* gate, float* out, int tokens, int width, int top, int experts) {
    const long long n = (long long)tokens * width;
    if (n <= 0) return 0;
    if (width % 8 == 0 && ld % 8 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)h % 16 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)shared % 16 == 0) {
        moe_gather_vec_kernel<<<(unsigned)((n / 8 + 255) / 256), 256, 0, stream>>>((const bf16*)y, row_of, ids, weights, (const bf16*)h, ld, shared, shared_dtype,
                                                                                  gate, out, tokens, width, top, experts);
        return eg_launch_status();
    }
    moe_gather_kernel<<<(unsigned)((n + 255) / 256), 256, 0, stream>>>((const bf16*)y, row_of, ids, weights, (const bf16*)h, ld, shared, shared_dtype, gate, out,
                                                                      tokens, width, top, experts);
    return eg_launch_status();
}
