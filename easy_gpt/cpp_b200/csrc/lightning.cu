// Linear attention whose state fades by a constant of the head ("lightning attention"): per head a matrix S [dk, dv] (float32,
// in the request's state slot),
//
//   q, k, v <- silu(.);   S <- decay_h S + k v^T;   o = S^T q
//   out = o / sqrt(mean(o^2) + eps) * gain * sigmoid(g)                 (mean over all heads' values together)
//
// q, k, v and g are columns of one projection's float32 output.
//
// One block per (head, batch entry, slice of the head's columns).  COLS neighbouring columns of S belong to P neighbouring lanes,
// each with R of their rows in registers for the entry's whole run of tokens; nothing a step computes is waited for by the
// next one but the state itself.  The block walks the entry in tiles of 16 tokens: the next tile's rows are on their way into
// registers while this one's steps run, are activated there and put into the other buffer.  A kernel behind norms and gates.  The
// slot keeps S as [head, column, row].  The order of every sum depends on the sizes alone.
#include <algorithm>

#include "common.cuh"

namespace {
constexpr int TILE = 16, PAD = 4;
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }

template <int R, int P, int COLS>
__global__ void __launch_bounds__(512, 1) lightning_kernel(const float* __restrict__ proj, long long ldp, int q_col, int k_col, int v_col,
                                                         const float* __restrict__ decays, float* __restrict__ state, long long slot_floats,
                                                         long long state_offset, const int* __restrict__ seq_starts, const int* __restrict__ seq_slots,
                                                         float* __restrict__ o_raw, int cols, int heads, int dk, int dv) {
    extern __shared__ __align__(16) float smem[];
    constexpr int RS = R + PAD, DS = RS * P;
    const int stage_floats = TILE * (2 * DS + cols);
    float* s_o = smem + 2 * stage_floats;           // [TILE, cols]
    const int head = blockIdx.x, seq = blockIdx.y, j0 = blockIdx.z * cols;
    const int start = seq_starts[seq], count = seq_starts[seq + 1] - start;
    const int jl = threadIdx.x / P * COLS, part = threadIdx.x % P;
    const int width = min(cols, dv - j0);
    const float decay = decays[head];
    float* S = state + (size_t)seq_slots[seq] * slot_floats + state_offset + ((size_t)head * dv + j0 + jl) * dk + part * R;
    float s[COLS][R];
#pragma unroll
    for (int c = 0; c < COLS; ++c)
#pragma unroll
        for (int r = 0; r < R; ++r) s[c][r] = (jl + c < width && part * R + r < dk) ? S[(size_t)c * dk + r] : 0.f;
    for (int i = threadIdx.x; i < 2 * stage_floats; i += blockDim.x) smem[i] = 0.f;      // rows beyond dk stay zero
    __syncthreads();
    const int per = 2 * dk + width;                 // values a token brings: its query, its key, this block's values
    constexpr int AHEAD = 8;                        // values a thread holds on their way
    float held[AHEAD];
    auto source = [&](int t0, int i) {
        const int t = i / per, d = i % per;
        const float* row = proj + (size_t)(start + t0 + t) * ldp;
        return d < dk ? row + q_col + head * dk + d : d < 2 * dk ? row + k_col + head * dk + d - dk : row + v_col + head * dv + j0 + d - 2 * dk;
    };
    auto place = [&](int b, int i, float v) {
        const int t = i / per, d = i % per;
        float* base = smem + b * stage_floats;
        const int e = d < dk ? d : d - dk;
        float* dst = d < 2 * dk ? base + (d < dk ? 0 : TILE * DS) + t * DS + (e / R) * RS + e % R : base + 2 * TILE * DS + t * cols + d - 2 * dk;
        *dst = silu_f(v);
    };
    auto request = [&](int ti) {                    // the first AHEAD values of a thread's share of tile ti
        const int t0 = ti * TILE, n = min(TILE, count - t0);
#pragma unroll
        for (int a = 0; a < AHEAD; ++a) {
            const int i = threadIdx.x + a * blockDim.x;
            held[a] = i < n * per ? __ldg(source(t0, i)) : 0.f;
        }
    };
    auto deliver = [&](int ti, int b) {
        const int t0 = ti * TILE, n = min(TILE, count - t0);
#pragma unroll
        for (int a = 0; a < AHEAD; ++a) {
            const int i = threadIdx.x + a * blockDim.x;
            if (i < n * per) place(b, i, held[a]);
        }
        for (int i = threadIdx.x + AHEAD * blockDim.x; i < n * per; i += blockDim.x) place(b, i, __ldg(source(t0, i)));
    };
    const int tiles = (count + TILE - 1) / TILE;
    if (tiles > 0) {
        request(0);
        deliver(0, 0);
    }
    __syncthreads();
    for (int ti = 0; ti < tiles; ++ti) {
        const int t0 = ti * TILE, n = min(TILE, count - t0);
        if (ti + 1 < tiles) request(ti + 1);
        const float* s_q = smem + (ti & 1) * stage_floats;
        const float* s_k = s_q + TILE * DS;
        const float* s_v = s_k + TILE * DS;
        auto step = [&](int t) {
            const float* q = s_q + t * DS + part * RS;
            const float* k = s_k + t * DS + part * RS;
            float value[COLS], read[COLS][2] = {};
#pragma unroll
            for (int c = 0; c < COLS; ++c) value[c] = s_v[t * cols + jl + c];
#pragma unroll
            for (int r = 0; r < R; r += 4) {
                const float4 kk = *reinterpret_cast<const float4*>(k + r), qq = *reinterpret_cast<const float4*>(q + r);
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    s[c][r] = fmaf(kk.x, value[c], decay * s[c][r]);
                    s[c][r + 1] = fmaf(kk.y, value[c], decay * s[c][r + 1]);
                    s[c][r + 2] = fmaf(kk.z, value[c], decay * s[c][r + 2]);
                    s[c][r + 3] = fmaf(kk.w, value[c], decay * s[c][r + 3]);
                    read[c][0] = fmaf(s[c][r], qq.x, read[c][0]);
                    read[c][1] = fmaf(s[c][r + 1], qq.y, read[c][1]);
                    read[c][0] = fmaf(s[c][r + 2], qq.z, read[c][0]);
                    read[c][1] = fmaf(s[c][r + 3], qq.w, read[c][1]);
                }
            }
#pragma unroll
            for (int c = 0; c < COLS; ++c) {
                float o = read[c][0] + read[c][1];
#pragma unroll
                for (int x = 1; x < P; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
                if (part == 0 && jl + c < width) s_o[t * cols + jl + c] = o;
            }
        };
        if (n == TILE) {
#pragma unroll 4
            for (int t = 0; t < TILE; ++t) step(t);
        } else {
            for (int t = 0; t < n; ++t) step(t);
        }
        if (ti + 1 < tiles) deliver(ti + 1, (ti + 1) & 1);      // that buffer's last reader was the tile before, a barrier ago
        __syncthreads();                                         // the tile's outputs and the next tile's rows are complete
        for (int i = threadIdx.x; i < n * width; i += blockDim.x) {
            const int t = i / width, d = i % width;
            o_raw[(size_t)(start + t0 + t) * ((size_t)heads * dv) + head * dv + j0 + d] = s_o[t * cols + d];
        }
        __syncthreads();                                         // before the next tile writes s_o
    }
#pragma unroll
    for (int c = 0; c < COLS; ++c)
#pragma unroll
        for (int r = 0; r < R; ++r)
            if (jl + c < width && part * R + r < dk) S[(size_t)c * dk + r] = s[c][r];
}

// a block per token
template <typename TO>
__global__ void __launch_bounds__(256) lightning_output_kernel(const float* __restrict__ o_raw, const float* __restrict__ proj, long long ldp, int g_col,
                                                               const float* __restrict__ gain, TO* __restrict__ y, long long ldy, int n, float eps) {
    __shared__ float scratch[32];
    const int t = blockIdx.x;
    const float* o = o_raw + (size_t)t * n;
    const float* g = proj + (size_t)t * ldp + g_col;
    float ss = 0.f;
    for (int d = threadIdx.x; d < n; d += blockDim.x) ss = fmaf(o[d], o[d], ss);
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
    for (int d = threadIdx.x; d < n; d += blockDim.x) y[(size_t)t * ldy + d] = from_f32<TO>(o[d] * inv * gain[d] * sigmoid_f(g[d]));
}

template <int R, int P, int COLS>
int launch_lightning(cudaStream_t stream, const float* proj, long long ldp, int q_col, int k_col, int v_col, const float* decays, float* state,
                     long long slot_floats, long long state_offset, const int* seq_starts, const int* seq_slots, float* o_raw, int slices, int num_seqs,
                     int heads, int dk, int dv) {
    constexpr int per_warp = 32 / P * COLS;
    const int most = 512 / P * COLS / per_warp * per_warp;
    int cols = (dv + slices - 1) / slices;
    cols = std::min((cols + per_warp - 1) / per_warp * per_warp, most);
    slices = (dv + cols - 1) / cols;
    const int threads = cols / COLS * P;
    const size_t smem = ((size_t)2 * TILE * (2 * (R + PAD) * P + cols) + (size_t)TILE * cols) * sizeof(float);
    if (threads > 512 || smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    auto kernel = lightning_kernel<R, P, COLS>;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    kernel<<<dim3(heads, num_seqs, slices), threads, smem, stream>>>(proj, ldp, q_col, k_col, v_col, decays, state, slot_floats, state_offset, seq_starts,
                                                                     seq_slots, o_raw, cols, heads, dk, dv);
    return 0;
}
}  // namespace

// proj float32 [tokens, ldp] with q, k (heads x dk), v and g (heads x dv) at their columns; decays float32 [heads]; gain float32
// [heads * dv]; o_raw float32 [tokens, heads * dv] of scratch; S of a request lies state_offset floats into its slot.  y [tokens, ldy] in
// y_dtype.  slices: into how many blocks a head's columns are dealt.  dk up to 256.
EG_API int eg_lightning(cudaStream_t stream, const float* proj, long long ldp, int q_col, int k_col, int v_col, int g_col, const float* decays,
                        const float* gain, float* state, long long slot_floats, long long state_offset, const int* seq_starts, const int* seq_slots,
                        float* o_raw, void* y, int y_dtype, long long ldy, int slices, int tokens, int num_seqs, int heads, int dk, int dv, float eps) {
    if (num_seqs <= 0 || tokens <= 0) return 0;
    if (heads <= 0 || dk <= 0 || dk > 256 || dv <= 0 || slices < 1 || !o_raw) return (int)cudaErrorInvalidValue;
    int rc;
#define EG_LIGHTNING(R, P, COLS)                                                                                                                        \
    rc = launch_lightning<R, P, COLS>(stream, proj, ldp, q_col, k_col, v_col, decays, state, slot_floats, state_offset, seq_starts, seq_slots, o_raw,     \
                                      slices, num_seqs, heads, dk, dv)
    if (dk <= 16) EG_LIGHTNING(4, 4, 1);
    else if (dk <= 32) EG_LIGHTNING(8, 4, 1);
    else if (dk <= 64) EG_LIGHTNING(8, 8, 2);
    else if (dk <= 128) EG_LIGHTNING(8, 16, 2);
    else EG_LIGHTNING(8, 32, 2);
#undef EG_LIGHTNING
    if (rc) return rc;
    const int n = heads * dv;
    if (y_dtype == EG_BF16) lightning_output_kernel<bf16><<<tokens, 256, 0, stream>>>(o_raw, proj, ldp, g_col, gain, (bf16*)y, ldy, n, eps);
    else lightning_output_kernel<float><<<tokens, 256, 0, stream>>>(o_raw, proj, ldp, g_col, gain, (float*)y, ldy, n, eps);
    return eg_launch_status();
}
