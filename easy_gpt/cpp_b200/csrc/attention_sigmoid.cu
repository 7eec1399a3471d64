// Grouped-query attention whose weights are a function of each score alone: the weight of a visible key is the sigmoid of its
// score, and weights are not normalised over the keys.  Over the paged cache; a key of KV head g lies at
// k[page * page_stride + g * head_stride + offset * row_stride], its value at the same place from v (keys and values in
// planes of their own with row_stride = dk = dv, or side by side in one row with row_stride = dk + dv).
//
//   q = (W_q h + b_q) / rms(W_q h + b_q) * gain_q * temp(p)      the norm over the WHOLE projection, before the split into heads
//   k = (W_k h + b_k) / rms(W_k h + b_k) * gain_k
//   temp(p) = 1 + coef * ln(floor((p + 1) / every) + 1)
//   s_h(i, j) = (q_h(i) . k_c(h)(j)) * scale + bias_h(i - j),  j <= i,   c(h) = h / (H / G)
//   out_h(i) = sigmoid(gate_h(i)) * sum_j sigmoid(s_h(i, j)) v_c(h)(j)
//
// bias_h(n) comes from a table [heads, reach]: entry min(n, reach - 1) (the caller folds whatever depends on head and distance
// into it: a learned bias by distance bucket, a number per head).  Scores, weights, norms and sums are float32.
//
// Since no weight depends on another key's score there is no running maximum, no rescaling and no final division, and partial
// sums of key ranges simply add up.
//
//   eg_sigmoid_attention_prepare  norms, temperature, cache write: a block per token
//   eg_sigmoid_attention          both precisions, any sizes (dv <= 256): a warp per (token, head), keys in ascending chunks of 32
//   eg_sigmoid_attention_tiles    bfloat16 prompt portions on the warp-level tensor cores, for sizes the tcgen05 kernel does not
//                                 take: a CTA takes 128 tokens of a listed tile and one head, a warp 32 (or 16) query rows; keys come
//                                 32 at a time through a three-stage cp.async ring
//   eg_sigmoid_attention_split    bfloat16 single tokens: a CTA takes one token, up to 16 query heads of one KV head (the rows of
//                                 the tensor-core tile) and one of `splits` ranges of the keys; each warp walks 16-key slices through
//                                 buffers of its own; the last CTA of a (token, KV head) to arrive adds the ranges' sums in order
//
// The tensor-core kernels work in base 2 on negated scores: weight = 1 / (1 + 2^x) with x = -log2(e) s; the caller hands
// -log2(e) scale and a table of -log2(e) bias.
#include "mma_utils.cuh"

namespace {
constexpr int MAX_PER_LANE = 8;        // value size <= 256 in the generic kernel
constexpr int LISTED_ROWS = 128;       // tokens of a listed tile
constexpr int BN = 32;                 // keys a step of the prompt kernel
constexpr int STAGES = 3;
constexpr int SMEM_LIMIT = 227 * 1024;
constexpr int TABLE_SMEM = 4096;       // entries of a head's bias table that are kept in shared memory

__device__ __forceinline__ float sigmoid_exact(float x) { return 1.0f / (1.0f + expf(-x)); }
// 1 / (1 + 2^x) by the hardware's approximations (relative error of a few 2^-23); 2^x = inf gives 0
__device__ __forceinline__ float weight_of(float x) {
    float e, w;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(w) : "f"(1.0f + e));
    return w;
}

// ---- preparation -----------------------------------------------------------------------------------------------------------
// VEC values a thread and pass (4: every row and every head starts on a 16-byte boundary)
template <int VEC> struct Pack { float v[VEC]; };
template <int VEC> __device__ __forceinline__ Pack<VEC> load_pack(const float* p) {
    Pack<VEC> r;
    if constexpr (VEC == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <typename T, int VEC> __device__ __forceinline__ void store_pack(T* p, const Pack<VEC>& r) {
    if constexpr (VEC == 4 && sizeof(T) == 2) {
        uint2 o;
        o.x = pack_bf16(r.v[0], r.v[1]);
        o.y = pack_bf16(r.v[2], r.v[3]);
        *reinterpret_cast<uint2*>(p) = o;
    } else if constexpr (VEC == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    } else {
        *p = from_f32<T>(r.v[0]);
    }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) sigmoid_prepare_kernel(const float* __restrict__ proj, long long ld, const float* __restrict__ bias,
                                                              const float* __restrict__ q_gain, const float* __restrict__ k_gain, float eps, float temp_coef,
                                                              int temp_every, const int* __restrict__ positions, const int* __restrict__ slot_map,
                                                              T* __restrict__ k_cache, T* __restrict__ v_cache, int row_stride, long long head_stride,
                                                              int page_size, long long page_stride, long long pool_slots, T* __restrict__ q_out, int nq, int nk,
                                                              int nv, int dk, int dv, int* status) {
    __shared__ float scratch[32];
    const int t = blockIdx.x;
    const float* row = proj + (size_t)t * ld;
    auto value = [&](int c) {
        Pack<VEC> x = load_pack<VEC>(row + c);
        if (bias) {
            const Pack<VEC> b = load_pack<VEC>(bias + c);
#pragma unroll
            for (int e = 0; e < VEC; ++e) x.v[e] += b.v[e];
        }
        return x;
    };
    float inv_q = 1.0f, inv_k = 1.0f;
    if (eps >= 0.f) {
        float sq = 0.f, sk = 0.f;
        for (int c = threadIdx.x * VEC; c < nq + nk; c += blockDim.x * VEC) {       // nq is a multiple of VEC: a pack lies on one side
            const Pack<VEC> x = value(c);
            float s = 0.f;
#pragma unroll
            for (int e = 0; e < VEC; ++e) s = fmaf(x.v[e], x.v[e], s);
            if (c < nq) sq += s; else sk += s;
        }
        inv_q = 1.0f / sqrtf(block_sum(sq, scratch) / (float)nq + eps);
        inv_k = 1.0f / sqrtf(block_sum(sk, scratch) / (float)nk + eps);
    }
    if (temp_every > 0) inv_q *= 1.0f + temp_coef * logf((float)((positions[t] + 1) / temp_every + 1));
    for (int c = threadIdx.x * VEC; c < nq; c += blockDim.x * VEC) {
        Pack<VEC> x = value(c);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x.v[e] *= inv_q;
        if (q_gain) {
            const Pack<VEC> g = load_pack<VEC>(q_gain + c);
#pragma unroll
            for (int e = 0; e < VEC; ++e) x.v[e] *= g.v[e];
        }
        store_pack<T, VEC>(q_out + (size_t)t * nq + c, x);
    }
    if (!k_cache) return;                               // the entry reads another entry's cache and stores nothing
    const long long slot = slot_map[t];
    if (slot < 0 || slot >= pool_slots) {
        if (threadIdx.x == 0) atomicOr(status, EG_STATUS_BAD_SLOT);
        return;
    }
    const long long at = (slot / page_size) * page_stride + (slot % page_size) * (long long)row_stride;
    for (int c = threadIdx.x * VEC; c < nk; c += blockDim.x * VEC) {
        Pack<VEC> x = value(nq + c);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x.v[e] *= inv_k;
        if (k_gain) {
            const Pack<VEC> g = load_pack<VEC>(k_gain + c);
#pragma unroll
            for (int e = 0; e < VEC; ++e) x.v[e] *= g.v[e];
        }
        store_pack<T, VEC>(k_cache + at + (c / dk) * head_stride + c % dk, x);
    }
    for (int c = threadIdx.x * VEC; c < nv; c += blockDim.x * VEC)
        store_pack<T, VEC>(v_cache + at + (c / dv) * head_stride + c % dv, value(nq + nk + c));
}

// ---- any sizes, both precisions -----------------------------------------------------------------------------------------------
constexpr int WARPS = 4;
template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
sigmoid_attention_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache, int row_stride, long long head_stride,
                         const int* __restrict__ block_table, int table_stride, const int* __restrict__ token_seq, const int* __restrict__ positions,
                         const float* __restrict__ bias_table, int reach, const float* __restrict__ gate, long long ld_gate, T* __restrict__ out, long long ldo,
                         int heads, int kv_heads, int dk, int dv, int page_size, long long page_stride, int num_pages, float scale, int* status) {
    extern __shared__ float q_shared[];                  // WARPS * dk
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x, h = blockIdx.y * WARPS + warp;
    if (h >= heads) return;                              // no block-wide barrier below
    const int g = h / (heads / kv_heads);
    const int pos = positions[t];
    const int* table = block_table + (size_t)token_seq[t] * table_stride;
    const float* bias = bias_table + (size_t)h * reach;
    float* qs = q_shared + warp * dk;
    const T* qrow = q + ((size_t)t * heads + h) * dk;
    for (int d = lane; d < dk; d += 32) qs[d] = to_f32<T>(qrow[d]);
    __syncwarp();
    float acc[MAX_PER_LANE];
#pragma unroll
    for (int i = 0; i < MAX_PER_LANE; ++i) acc[i] = 0.0f;
    for (int base = 0; base <= pos; base += 32) {
        const int kpos = base + lane;
        long long row_off = -1;
        if (kpos <= pos) {
            const int page = table[kpos / page_size];
            if (page < 0 || page >= num_pages) atomicOr(status, EG_STATUS_BAD_PAGE);
            else row_off = (long long)page * page_stride + g * head_stride + (long long)(kpos % page_size) * row_stride;
        }
        float w = 0.0f;
        if (row_off >= 0) {
            const T* krow = k_cache + row_off;
            float dot = 0.0f;
            for (int d = 0; d < dk; ++d) dot = fmaf(qs[d], to_f32<T>(krow[d]), dot);
            w = sigmoid_exact(dot * scale + bias[min(pos - kpos, reach - 1)]);
        }
        const int nkeys = min(32, pos + 1 - base);
        for (int j = 0; j < nkeys; ++j) {
            const float wj = __shfl_sync(0xffffffffu, w, j);
            const long long off_j = __shfl_sync(0xffffffffu, row_off, j);
            if (off_j < 0) continue;
            const T* vrow = v_cache + off_j;
#pragma unroll
            for (int i = 0; i < MAX_PER_LANE; ++i) {
                const int d = lane + 32 * i;
                if (d < dv) acc[i] = fmaf(wj, to_f32<T>(vrow[d]), acc[i]);
            }
        }
    }
    const float f = gate ? sigmoid_exact(gate[(size_t)t * ld_gate + h]) : 1.0f;
    T* orow = out + (size_t)t * ldo + (size_t)h * dv;
#pragma unroll
    for (int i = 0; i < MAX_PER_LANE; ++i) {
        const int d = lane + 32 * i;
        if (d < dv) orow[d] = from_f32<T>(acc[i] * f);
    }
}

// ---- what the two tensor-core kernels share -------------------------------------------------------------------------------------
struct MmaParams {
    const bf16 *q, *k_cache, *v_cache;
    int row_stride;
    long long head_stride, page_stride;
    const int* block_table;
    int table_stride;
    const int *token_seq, *positions, *list;      // list: the listed tiles (prompt), or the single tokens' indices (or null: all)
    int count;                                    // listed sub-tiles, or tokens
    const float* bias_table;                      // [heads, reach], times -log2(e)
    int reach;
    const float* gate;
    long long ld_gate;
    bf16* out;
    long long ldo;
    float* partial;                               // [token, head, split, dv]
    int* counters;                                // a ticket per (token, row block), zero before and after
    int heads, kv_heads, dk, dv, page_size, num_pages, splits;
    float neg_scale;                              // -log2(e) * scale
    int* status;
};
__host__ __device__ constexpr int pad16(int n) { return (n + 15) / 16 * 16; }

// S[16 MT x 8 NKT] = Q K^T over `wide` (a multiple of 16) columns; rows of q_rows qs apart, of k_rows ks apart in shared memory
template <int MT, int NKT>
__device__ __forceinline__ void score_tile(float (&s)[MT][NKT][4], const bf16* q_rows, int qs, const bf16* k_rows, int ks, int wide, int lane) {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < NKT; ++i) s[mt][i][0] = s[mt][i][1] = s[mt][i][2] = s[mt][i][3] = 0.f;
    const bf16* qa = q_rows + (lane & 15) * qs + (lane >> 4) * 8;
    const bf16* kb = k_rows + ((lane >> 4) * 8 + (lane & 7)) * ks + ((lane >> 3) & 1) * 8;
#pragma unroll 2
    for (int k0 = 0; k0 < wide; k0 += 16) {
        uint32_t a[MT][4];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) ldmatrix_x4(a[mt], qa + mt * 16 * qs + k0);
#pragma unroll
        for (int np = 0; np < NKT / 2; ++np) {
            uint32_t b[4];
            ldmatrix_x4(b, kb + np * 16 * ks + k0);
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                mma_bf16_16816(s[mt][2 * np], a[mt], b[0], b[1]);
                mma_bf16_16816(s[mt][2 * np + 1], a[mt], b[2], b[3]);
            }
        }
    }
}

// scores -> weights in place, for the rows lane / 4 (position lo) and lane / 4 + 8 (position hi); key column nt, pair e is key0 + 8 nt +
// 2 (lane % 4) + e; a key behind the row's position has weight 0 (position -1: no key).  `far`: every distance is at least
// reach - 1 and no key lies behind a row.
template <int NKT>
__device__ __forceinline__ void weigh_tile(float (&s)[NKT][4], int key0, int lo, int hi, const float* bias_lo, const float* bias_hi, int last, float neg_scale,
                                           bool far, int lane) {
    if (far) {
        const float b0 = bias_lo[last], b1 = bias_hi[last];
#pragma unroll
        for (int nt = 0; nt < NKT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[nt][e] = weight_of(fmaf(s[nt][e], neg_scale, e < 2 ? b0 : b1));
        return;
    }
#pragma unroll
    for (int nt = 0; nt < NKT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int n = (e < 2 ? lo : hi) - (key0 + nt * 8 + 2 * (lane & 3) + (e & 1));
            const float* bias = e < 2 ? bias_lo : bias_hi;
            s[nt][e] = n >= 0 ? weight_of(fmaf(s[nt][e], neg_scale, bias[min(n, last)])) : 0.f;
        }
}

// O[16 MT x dv] += A[16 MT x 16] V[16 keys x dv]
template <int MT, int NT>
__device__ __forceinline__ void value_step(float (&o)[MT][NT][4], const uint32_t (&a)[MT][4], const bf16* v_rows, int vs, int dv, int lane) {
    const bf16* vb = v_rows + (((lane >> 3) & 1) * 8 + (lane & 7)) * vs + (lane >> 4) * 8;
#pragma unroll
    for (int dp = 0; dp < NT / 2; ++dp) {
        if (dp * 16 < dv) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, vb + dp * 16);
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                mma_bf16_16816(o[mt][2 * dp], a[mt], b[0], b[1]);
                mma_bf16_16816(o[mt][2 * dp + 1], a[mt], b[2], b[3]);
            }
        }
    }
}
template <int NKT>
__device__ __forceinline__ void weights_fragment(uint32_t (&a)[4], const float (&s)[NKT][4], int ks) {
    a[0] = pack_bf16(s[2 * ks][0], s[2 * ks][1]);
    a[1] = pack_bf16(s[2 * ks][2], s[2 * ks][3]);
    a[2] = pack_bf16(s[2 * ks + 1][0], s[2 * ks + 1][1]);
    a[3] = pack_bf16(s[2 * ks + 1][2], s[2 * ks + 1][3]);
}

// ---- prompt portions -----------------------------------------------------------------------------------------------------------
template <int NT, int MT, int NWARPS>
__global__ void __launch_bounds__(NWARPS * 32) sigmoid_tiles_kernel(const MmaParams p) {
    constexpr int ROWS = 16 * MT * NWARPS, SUBS = LISTED_ROWS / ROWS, NTHREADS = NWARPS * 32;
    extern __shared__ __align__(16) unsigned char smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int dk = p.dk, dv = p.dv, wide = pad16(dk), qs = wide + 8, vs = pad16(dv) + 8;
    const int sub = p.count - 1 - (int)blockIdx.y;              // the last tiles of a prompt have the most keys: they start first, for all heads
    const int* tile = p.list + 3 * (sub / SUBS);
    const int first = tile[1] + ROWS * (sub % SUBS);
    const int count = min(ROWS, tile[2] - ROWS * (sub % SUBS));
    if (count <= 0) return;
    const int h = blockIdx.x, g = h / (p.heads / p.kv_heads);
    const int* table = p.block_table + (size_t)tile[0] * p.table_stride;

    bf16* q_s = (bf16*)smem;                                   // [ROWS][qs]
    bf16* k_s = q_s + ROWS * qs;                               // [STAGES][BN][qs]
    bf16* v_s = k_s + STAGES * BN * qs;                        // [STAGES][BN][vs]
    float* bias_s = (float*)(v_s + STAGES * BN * vs);          // [min(reach, TABLE_SMEM)]
    const int pos_first = p.positions[first], pos_last = pos_first + count - 1;       // positions in a tile are consecutive
    const int steps = pos_last / BN + 1, last = p.reach - 1;
    // the padding columns of every row hold zeros; the copies leave them alone
    for (int i = tid; i < (ROWS + STAGES * BN); i += NTHREADS)
        for (int d = dk; d < wide; ++d) q_s[i * qs + d] = __float2bfloat16_rn(0.f);
    for (int i = tid; i < STAGES * BN; i += NTHREADS)
        for (int d = dv; d < pad16(dv); ++d) v_s[i * vs + d] = __float2bfloat16_rn(0.f);
    const float* bias = p.bias_table + (size_t)h * p.reach;
    if (p.reach <= TABLE_SMEM) {
        for (int i = tid; i < p.reach; i += NTHREADS) bias_s[i] = bias[i];
        bias = bias_s;
    }
    auto fetch = [&](int step) {
        const int buf = step % STAGES;
        for (int j = warp; j < BN; j += NWARPS) {
            const int kpos = step * BN + j;
            bool valid = kpos <= pos_last;
            long long off = 0;
            if (valid) {
                const int page = __ldg(table + kpos / p.page_size);
                if (page < 0 || page >= p.num_pages) {
                    if (lane == 0) atomicOr(p.status, EG_STATUS_BAD_PAGE);
                    valid = false;
                } else {
                    off = (long long)page * p.page_stride + g * p.head_stride + (long long)(kpos % p.page_size) * p.row_stride;
                }
            }
            bf16* kd = k_s + (buf * BN + j) * qs;
            for (int c = lane; c < dk / 8; c += 32) cp_async_16(kd + c * 8, p.k_cache + off + c * 8, valid);
            bf16* vd = v_s + (buf * BN + j) * vs;
            for (int c = lane; c < dv / 8; c += 32) cp_async_16(vd + c * 8, p.v_cache + off + c * 8, valid);
        }
    };
    for (int i = tid; i < ROWS * (dk / 8); i += NTHREADS) {
        const int r = i / (dk / 8), c = i % (dk / 8);
        const bool valid = r < count;
        cp_async_16(q_s + r * qs + c * 8, p.q + (valid ? ((size_t)(first + r) * p.heads + h) * dk + c * 8 : 0), valid);
    }
    fetch(0);
    cp_async_commit();
    if (steps > 1) fetch(1);
    cp_async_commit();

    const int row0 = warp * MT * 16;
    int lim[MT][2];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int row = row0 + mt * 16 + (lane >> 2) + 8 * r;
            lim[mt][r] = row < count ? pos_first + row : -1;
        }
    const int warp_lo = pos_first + row0, warp_hi = row0 < count ? pos_first + min(count - 1, row0 + MT * 16 - 1) : -1;
    const bool whole = row0 + MT * 16 <= count;
    float o[MT][NT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < NT; ++i) o[mt][i][0] = o[mt][i][1] = o[mt][i][2] = o[mt][i][3] = 0.f;

    for (int step = 0; step < steps; ++step) {
        cp_async_wait<1>();
        __syncthreads();                                       // this step's keys have arrived; the buffer of the step before is free
        if (step + 2 < steps) fetch(step + 2);
        cp_async_commit();
        const int key0 = step * BN, buf = step % STAGES;
        if (key0 > warp_hi) continue;
        float s[MT][BN / 8][4];
        score_tile<MT, BN / 8>(s, q_s + row0 * qs, qs, k_s + buf * BN * qs, qs, wide, lane);
        const bool far = whole && warp_lo - (key0 + BN - 1) >= last;
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) weigh_tile<BN / 8>(s[mt], key0, lim[mt][0], lim[mt][1], bias, bias, last, p.neg_scale, far, lane);
#pragma unroll
        for (int ks = 0; ks < BN / 16; ++ks) {
            uint32_t a[MT][4];
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) weights_fragment<BN / 8>(a[mt], s[mt], ks);
            value_step<MT, NT>(o, a, v_s + (buf * BN + ks * 16) * vs, vs, dv, lane);
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int row = row0 + mt * 16 + (lane >> 2) + 8 * r;
            if (row >= count) continue;
            const size_t t = (size_t)(first + row);
            const float f = p.gate ? sigmoid_exact(p.gate[t * p.ld_gate + h]) : 1.0f;
            bf16* dst = p.out + t * p.ldo + (size_t)h * dv;
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) {
                const int d = nt * 8 + 2 * (lane & 3);
                if (d < dv) *(__nv_bfloat162*)(dst + d) = __floats2bfloat162_rn(o[mt][nt][2 * r] * f, o[mt][nt][2 * r + 1] * f);
            }
        }
}

size_t tiles_smem(int dk, int dv, int rows, int reach) {
    return (size_t)(rows + STAGES * BN) * (pad16(dk) + 8) * 2 + (size_t)STAGES * BN * (pad16(dv) + 8) * 2 + (reach <= TABLE_SMEM ? (size_t)reach * 4 : 0);
}

// ---- single tokens ---------------------------------------------------------------------------------------------------------------
constexpr int SPLIT_WARPS = 4, SLICE = 16, SLICE_STAGES = 3;

// keys of a range: whole slices for every warp, at least 64 keys
__host__ __device__ inline int range_keys(int keys, int splits) {
    const int per = (keys + splits - 1) / splits;
    return (per + 63) / 64 * 64;
}

template <int NT>
__global__ void __launch_bounds__(SPLIT_WARPS * 32) sigmoid_split_kernel(const MmaParams p) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ int last_here;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int dk = p.dk, dv = p.dv, wide = pad16(dk), qs = wide + 8, vs = pad16(dv) + 8, group = p.heads / p.kv_heads;
    const int listed = blockIdx.x, t = p.list ? p.list[listed] : listed;
    const int blocks_per_head = (group + 15) / 16, g = blockIdx.y / blocks_per_head, r0 = blockIdx.y % blocks_per_head * 16;
    const int rows = min(16, group - r0), h0 = g * group + r0, z = blockIdx.z;
    const int pos = p.positions[t];
    const int* table = p.block_table + (size_t)p.token_seq[t] * p.table_stride;
    const int chunk = range_keys(pos + 1, p.splits);
    const int k_begin = z * chunk, k_end = min(pos + 1, k_begin + chunk);

    bf16* q_s = (bf16*)smem;                                                       // [16][qs]
    bf16* ring = q_s + 16 * qs;                                                    // per warp: SLICE_STAGES x (SLICE keys [qs], SLICE values [vs])
    bf16* my_ring = ring + (size_t)warp * SLICE_STAGES * SLICE * (qs + vs);
    for (int i = tid; i < 16; i += SPLIT_WARPS * 32)
        for (int d = dk; d < wide; ++d) q_s[i * qs + d] = __float2bfloat16_rn(0.f);
    for (int i = lane; i < SLICE_STAGES * SLICE; i += 32) {
        bf16* base = my_ring + (size_t)(i / SLICE) * SLICE * (qs + vs);
        for (int d = dk; d < wide; ++d) base[(i % SLICE) * qs + d] = __float2bfloat16_rn(0.f);
        for (int d = dv; d < pad16(dv); ++d) base[SLICE * qs + (i % SLICE) * vs + d] = __float2bfloat16_rn(0.f);
    }
    for (int i = tid; i < 16 * (dk / 8); i += SPLIT_WARPS * 32) {
        const int r = i / (dk / 8), c = i % (dk / 8);
        const bool valid = r < rows;
        cp_async_16(q_s + r * qs + c * 8, p.q + (valid ? ((size_t)t * p.heads + h0 + r) * dk + c * 8 : 0), valid);
    }
    cp_async_commit();
    // warp w takes the slices w, w + 4, ... of the range
    const int slices = k_begin < k_end ? (k_end - k_begin + SLICE - 1) / SLICE : 0;
    const int mine = slices > warp ? (slices - warp + SPLIT_WARPS - 1) / SPLIT_WARPS : 0;
    const int pieces_k = dk / 8, pieces = pieces_k + dv / 8;
    auto fetch = [&](int i) {
        bf16* base = my_ring + (size_t)(i % SLICE_STAGES) * SLICE * (qs + vs);
        const int key0 = k_begin + (warp + i * SPLIT_WARPS) * SLICE;
        // lane j < 16 looks up key j's row
        const int kpos = key0 + (lane & 15);
        long long off = -1;
        if (kpos < k_end) {
            const int page = __ldg(table + kpos / p.page_size);
            if (page < 0 || page >= p.num_pages) atomicOr(p.status, EG_STATUS_BAD_PAGE);
            else off = (long long)page * p.page_stride + g * p.head_stride + (long long)(kpos % p.page_size) * p.row_stride;
        }
        for (int w = lane; w < (SLICE * pieces + 31) / 32 * 32; w += 32) {
            const int j = min(w / pieces, SLICE - 1), c = w % pieces;
            const long long row = __shfl_sync(0xffffffffu, off, j);
            if (w >= SLICE * pieces) continue;
            const bool valid = row >= 0;
            if (c < pieces_k) cp_async_16(base + j * qs + c * 8, p.k_cache + (valid ? row : 0) + c * 8, valid);
            else cp_async_16(base + SLICE * qs + j * vs + (c - pieces_k) * 8, p.v_cache + (valid ? row : 0) + (c - pieces_k) * 8, valid);
        }
    };
#pragma unroll
    for (int i = 0; i < SLICE_STAGES - 1; ++i) {
        if (i < mine) fetch(i);
        cp_async_commit();
    }
    cp_async_wait<SLICE_STAGES - 1>();                         // the queries
    __syncthreads();
    const int row_lo = lane >> 2, row_hi = row_lo + 8, last = p.reach - 1;
    const float* bias_lo = p.bias_table + (size_t)(h0 + min(row_lo, rows - 1)) * p.reach;
    const float* bias_hi = p.bias_table + (size_t)(h0 + min(row_hi, rows - 1)) * p.reach;
    float o[1][NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) o[0][i][0] = o[0][i][1] = o[0][i][2] = o[0][i][3] = 0.f;
    for (int i = 0; i < mine; ++i) {
        cp_async_wait<SLICE_STAGES - 2>();
        __syncwarp();                                          // the slice has arrived, and every lane is done with the one before
        if (i + SLICE_STAGES - 1 < mine) fetch(i + SLICE_STAGES - 1);
        cp_async_commit();
        const bf16* base = my_ring + (size_t)(i % SLICE_STAGES) * SLICE * (qs + vs);
        const int key0 = k_begin + (warp + i * SPLIT_WARPS) * SLICE;
        float s[1][2][4];
        score_tile<1, 2>(s, q_s, qs, base, qs, wide, lane);
        const int limit = k_end - 1;                            // every row of the tile is the same token; keys beyond the range are others'
        const bool far = key0 + SLICE <= k_end && pos - (key0 + SLICE - 1) >= last;
        if (far) {
            weigh_tile<2>(s[0], key0, pos, pos, bias_lo, bias_hi, last, p.neg_scale, true, lane);
        } else {
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int kpos = key0 + nt * 8 + 2 * (lane & 3) + (e & 1);
                    const float* bias = e < 2 ? bias_lo : bias_hi;
                    s[0][nt][e] = kpos <= limit ? weight_of(fmaf(s[0][nt][e], p.neg_scale, bias[min(pos - kpos, last)])) : 0.f;
                }
        }
        uint32_t a[1][4];
        weights_fragment<2>(a[0], s[0], 0);
        value_step<1, NT>(o, a, base + SLICE * qs, vs, dv, lane);
    }
    cp_async_wait<0>();
    __syncthreads();                                            // the rings are free: the warps' sums meet there, [warp][16][dv]
    float* sums = (float*)ring;
    const int dvp = pad16(dv);
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
        const int d = nt * 8 + 2 * (lane & 3);
        if (d < dvp) {
            *(float2*)(sums + (size_t)(warp * 16 + row_lo) * dvp + d) = make_float2(o[0][nt][0], o[0][nt][1]);
            *(float2*)(sums + (size_t)(warp * 16 + row_hi) * dvp + d) = make_float2(o[0][nt][2], o[0][nt][3]);
        }
    }
    __syncthreads();
    const size_t part0 = ((size_t)listed * p.heads + h0) * p.splits;
    auto finish = [&](int r, int d, float v) {
        const float f = p.gate ? sigmoid_exact(p.gate[(size_t)t * p.ld_gate + h0 + r]) : 1.0f;
        p.out[(size_t)t * p.ldo + (size_t)(h0 + r) * dv + d] = __float2bfloat16_rn(v * f);
    };
    for (int i = tid; i < rows * dv; i += SPLIT_WARPS * 32) {
        const int r = i / dv, d = i % dv;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < SPLIT_WARPS; ++w) v += sums[(size_t)(w * 16 + r) * dvp + d];
        if (p.splits == 1) finish(r, d, v);
        else __stcg(p.partial + (part0 + (size_t)r * p.splits + z) * dv + d, v);
    }
    if (p.splits == 1) return;
    __threadfence();
    __syncthreads();
    int* ticket = p.counters + (size_t)listed * gridDim.y + blockIdx.y;
    if (tid == 0) last_here = atomicAdd(ticket, 1) == p.splits - 1;
    __syncthreads();
    if (!last_here) return;
    __threadfence();
    for (int i = tid; i < rows * dv; i += SPLIT_WARPS * 32) {
        const int r = i / dv, d = i % dv;
        float v = 0.f;
        for (int s = 0; s < p.splits; ++s) v += __ldcg(p.partial + (part0 + (size_t)r * p.splits + s) * dv + d);
        finish(r, d, v);
    }
    if (tid == 0) *ticket = 0;
}

size_t split_smem(int dk, int dv) {
    const size_t qs = pad16(dk) + 8, vs = pad16(dv) + 8;
    const size_t ring = (size_t)SPLIT_WARPS * SLICE_STAGES * SLICE * (qs + vs) * 2, sums = (size_t)SPLIT_WARPS * 16 * pad16(dv) * 4;
    return 16 * qs * 2 + (ring > sums ? ring : sums);
}

template <typename K>
int allow_smem(K kernel, size_t bytes) {
    return bytes > 48 * 1024 ? (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) : 0;
}
}  // namespace

// proj float32 [tokens, ld]: queries (nq = heads * dk columns), keys (kv_heads * dk), values (kv_heads * dv) side by side; bias
// float32 over the same columns, or null; eps < 0: no norm; gains [nq] / [nk] or null; temp_every 0: no temperature.
// k_cache null: nothing is stored.  q_out [tokens, nq].
EG_API int eg_sigmoid_attention_prepare(cudaStream_t stream, int dtype, const float* proj, long long ld, const float* bias, const float* q_gain,
                                        const float* k_gain, float eps, float temp_coef, int temp_every, const int* positions, const int* slot_map,
                                        void* k_cache, void* v_cache, int row_stride, long long head_stride, int page_size, long long page_stride,
                                        long long pool_slots, void* q_out, int tokens, int heads, int kv_heads, int dk, int dv, int* status) {
    if (tokens <= 0) return 0;
    if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || dk <= 0 || dv <= 0 || temp_every < 0) return (int)cudaErrorInvalidValue;
    const int nq = heads * dk, nk = kv_heads * dk, nv = kv_heads * dv;
    const bool wide = dk % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && row_stride % 4 == 0 && head_stride % 4 == 0 && page_stride % 4 == 0 &&
                      (uintptr_t)proj % 16 == 0 && (uintptr_t)bias % 16 == 0 && (uintptr_t)q_gain % 16 == 0 && (uintptr_t)k_gain % 16 == 0 &&
                      (uintptr_t)k_cache % 16 == 0 && (uintptr_t)v_cache % (dtype == EG_BF16 ? 8 : 16) == 0 && (uintptr_t)q_out % 16 == 0;
#define EG_PREPARE(T, VEC)                                                                                                                                    \
    sigmoid_prepare_kernel<T, VEC><<<tokens, 256, 0, stream>>>(proj, ld, bias, q_gain, k_gain, eps, temp_coef, temp_every, positions, slot_map, (T*)k_cache,   \
                                                               (T*)v_cache, row_stride, head_stride, page_size, page_stride, pool_slots, (T*)q_out, nq, nk,    \
                                                               nv, dk, dv, status)
    if (dtype == EG_BF16) {
        if (wide) EG_PREPARE(bf16, 4);
        else EG_PREPARE(bf16, 1);
    } else {
        if (wide) EG_PREPARE(float, 4);
        else EG_PREPARE(float, 1);
    }
#undef EG_PREPARE
    return eg_launch_status();
}

// q [tokens, heads, dk]; bias_table float32 [heads, reach] (natural units); gate float32 [tokens, ld_gate] (head h at column h) or null;
// out [tokens, ldo], head h at column h * dv.
EG_API int eg_sigmoid_attention(cudaStream_t stream, int dtype, const void* q, const void* k_cache, const void* v_cache, int row_stride, long long head_stride,
                                const int* block_table, int table_stride, const int* token_seq, const int* positions, const float* bias_table, int reach,
                                const float* gate, long long ld_gate, void* out, long long ldo, int tokens, int heads, int kv_heads, int dk, int dv,
                                int page_size, long long page_stride, int num_pages, float scale, int* status) {
    if (tokens <= 0) return 0;
    if (dv > 32 * MAX_PER_LANE || dv <= 0 || dk <= 0 || dk > 2048 || kv_heads <= 0 || heads % kv_heads || reach < 1) return (int)cudaErrorInvalidValue;
    const dim3 grid(tokens, (heads + WARPS - 1) / WARPS);
    const size_t smem = (size_t)WARPS * dk * sizeof(float);
#define EG_GENERIC(T)                                                                                                                                          \
    sigmoid_attention_kernel<T><<<grid, WARPS * 32, smem, stream>>>((const T*)q, (const T*)k_cache, (const T*)v_cache, row_stride, head_stride, block_table,     \
                                                                    table_stride, token_seq, positions, bias_table, reach, gate, ld_gate, (T*)out, ldo, heads,   \
                                                                    kv_heads, dk, dv, page_size, page_stride, num_pages, scale, status)
    if (dtype == EG_BF16) EG_GENERIC(bf16);
    else EG_GENERIC(float);
#undef EG_GENERIC
    return eg_launch_status();
}

// whether the tensor-core kernels take these sizes (rows of keys and values in pieces of 16 bytes)
EG_API int eg_sigmoid_attention_mma_takes(int dk, int dv, int reach) {
    return dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 512 && dv <= 256 && reach >= 1 && tiles_smem(dk, dv, 64, reach) <= SMEM_LIMIT &&
           split_smem(dk, dv) <= SMEM_LIMIT;
}

// bfloat16; bias_table float32 [heads, reach] times -log2(e).  tiles: int32 [num_tiles, 3] = (entry, first token, tokens <= 128).
EG_API int eg_sigmoid_attention_tiles(cudaStream_t stream, const void* q, const void* k_cache, const void* v_cache, int row_stride, long long head_stride,
                                      const int* block_table, int table_stride, const int* positions, const int* tiles, int num_tiles, const float* bias_table,
                                      int reach, const float* gate, long long ld_gate, void* out, long long ldo, int heads, int kv_heads, int dk, int dv,
                                      int page_size, long long page_stride, int num_pages, float scale, int* status) {
    if (num_tiles <= 0) return 0;
    if (kv_heads <= 0 || heads % kv_heads || !eg_sigmoid_attention_mma_takes(dk, dv, reach) || row_stride % 8 || head_stride % 8 || page_stride % 8 || ldo % 2 ||
        (uintptr_t)q % 16 || (uintptr_t)k_cache % 16 || (uintptr_t)v_cache % 16)
        return (int)cudaErrorInvalidValue;
    MmaParams p{};
    p.q = (const bf16*)q;
    p.k_cache = (const bf16*)k_cache;
    p.v_cache = (const bf16*)v_cache;
    p.row_stride = row_stride;
    p.head_stride = head_stride;
    p.page_stride = page_stride;
    p.block_table = block_table;
    p.table_stride = table_stride;
    p.positions = positions;
    p.list = tiles;
    p.bias_table = bias_table;
    p.reach = reach;
    p.gate = gate;
    p.ld_gate = ld_gate;
    p.out = (bf16*)out;
    p.ldo = ldo;
    p.heads = heads;
    p.kv_heads = kv_heads;
    p.dk = dk;
    p.dv = dv;
    p.page_size = page_size;
    p.num_pages = num_pages;
    p.neg_scale = -1.4426950408889634f * scale;
    p.status = status;
#define EG_TILES(NT, MT)                                                                                                     \
    {                                                                                                                        \
        constexpr int rows = 16 * MT * 4;                                                                                    \
        const size_t smem = tiles_smem(dk, dv, rows, reach);                                                                 \
        const int rc = allow_smem(sigmoid_tiles_kernel<NT, MT, 4>, smem);                                                    \
        if (rc) return rc;                                                                                                   \
        p.count = num_tiles * (LISTED_ROWS / rows);                                                                          \
        sigmoid_tiles_kernel<NT, MT, 4><<<dim3(heads, p.count), 128, smem, stream>>>(p);                                     \
    }
    const bool tall = tiles_smem(dk, dv, 128, reach) <= SMEM_LIMIT;      // 128 rows of queries a CTA, else 64
    const int nt = pad16(dv) / 8;
    if (nt <= 4 && tall) EG_TILES(4, 2)
    else if (nt <= 8 && tall) EG_TILES(8, 2)
    else if (nt <= 12 && tall) EG_TILES(12, 2)
    else if (nt <= 16 && tall) EG_TILES(16, 2)
    else EG_TILES(32, 1)
#undef EG_TILES
    return eg_launch_status();
}

// bfloat16 single tokens (num_tokens of them, token_list their indices or null for 0 .. num_tokens - 1).  splits > 1: partial float32
// [num_tokens, heads, splits, dv] and a zeroed counter per (token, KV head, 16 query heads).
EG_API int eg_sigmoid_attention_split(cudaStream_t stream, const void* q, const void* k_cache, const void* v_cache, int row_stride, long long head_stride,
                                      const int* block_table, int table_stride, const int* token_seq, const int* positions, const int* token_list,
                                      int num_tokens, const float* bias_table, int reach, const float* gate, long long ld_gate, void* out, long long ldo,
                                      float* partial, int* counters, int splits, int heads, int kv_heads, int dk, int dv, int page_size,
                                      long long page_stride, int num_pages, float scale, int* status) {
    if (num_tokens <= 0) return 0;
    if (kv_heads <= 0 || heads % kv_heads || splits < 1 || (splits > 1 && (!partial || !counters)) || !eg_sigmoid_attention_mma_takes(dk, dv, reach) ||
        row_stride % 8 || head_stride % 8 || page_stride % 8 || (uintptr_t)q % 16 || (uintptr_t)k_cache % 16 || (uintptr_t)v_cache % 16)
        return (int)cudaErrorInvalidValue;
    MmaParams p{};
    p.q = (const bf16*)q;
    p.k_cache = (const bf16*)k_cache;
    p.v_cache = (const bf16*)v_cache;
    p.row_stride = row_stride;
    p.head_stride = head_stride;
    p.page_stride = page_stride;
    p.block_table = block_table;
    p.table_stride = table_stride;
    p.token_seq = token_seq;
    p.positions = positions;
    p.list = token_list;
    p.count = num_tokens;
    p.bias_table = bias_table;
    p.reach = reach;
    p.gate = gate;
    p.ld_gate = ld_gate;
    p.out = (bf16*)out;
    p.ldo = ldo;
    p.partial = partial;
    p.counters = counters;
    p.heads = heads;
    p.kv_heads = kv_heads;
    p.dk = dk;
    p.dv = dv;
    p.page_size = page_size;
    p.num_pages = num_pages;
    p.splits = splits;
    p.neg_scale = -1.4426950408889634f * scale;
    p.status = status;
    const int group = heads / kv_heads;
    const dim3 grid(num_tokens, kv_heads * ((group + 15) / 16), splits);
    const size_t smem = split_smem(dk, dv);
#define EG_SPLIT(NT)                                                                 \
    {                                                                                \
        const int rc = allow_smem(sigmoid_split_kernel<NT>, smem);                   \
        if (rc) return rc;                                                           \
        sigmoid_split_kernel<NT><<<grid, SPLIT_WARPS * 32, smem, stream>>>(p);       \
    }
    const int nt = pad16(dv) / 8;
    if (nt <= 4) EG_SPLIT(4)
    else if (nt <= 8) EG_SPLIT(8)
    else if (nt <= 12) EG_SPLIT(12)
    else if (nt <= 16) EG_SPLIT(16)
    else EG_SPLIT(32)
#undef EG_SPLIT
    return eg_launch_status();
}
