// The generalised delta rule: per head a matrix S [dim, dim] (float32, in the request's state slot) whose rows decay each at a
// rate of its own, from which every token takes off what it holds along the token's unit key (at a rate per row), and into
// which it writes its value along its key; both terms read the old state:
//
//   u = k / sqrt(|k|^2 + unit_eps)                                                      (per head, float32)
//   w = exp(-decay_scale * sigmoid(x + w0)),   a = sigmoid(y + a0)                        (per head and key channel)
//   S <- diag(w) S - (a u)(u^T S) + k v^T;   o = S^T r                                    (o reads the new state)
//   out = o / sqrt(mean(o^2) + eps) * gain * sigmoid(g)                                  (mean per head, gain per head and channel)
//
// r, k, v, y and g are columns of one projection's float32 output, x comes from a second product.
//
// A kernel over all tokens first makes w, u and a u (a warp per token and head).  Then one block per (head, batch entry,
// slice of the head's columns: the columns of S do not depend on one another).  COLS neighbouring columns of S belong to P
// neighbouring lanes, each with R of their rows in registers for the entry's whole run of tokens.  Per token a lane reads its
// rows' pieces of five vectors (w, u, a u, k, r) from shared memory once for all its columns; the dot product with u over the
// old rows is the only thing the next step waits for, the one with r over the new rows is not.  The block walks the entry in
// tiles of tokens that arrive by asynchronous copies, the next tile's behind this one's steps.  Outputs are normed and gated by the
// block itself where it holds a whole head, else by a kernel behind.  The slot keeps S as [head, column, row].  The order of
// every sum depends on the sizes alone.
#include <algorithm>
#include <cstdlib>

#include "common.cuh"
#include "decay_exp.cuh"

namespace {

constexpr int PAD = 4;          // floats between the parts' pieces of a staged vector: the parts' 16-byte loads then hit different banks
constexpr int VECS = 5;         // staged vectors a token: w, u, a u, k, r

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ void copy_async_16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_async_4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

struct DeltaParams {
    const float* proj;          // [tokens, ldp]
    long long ldp;
    int r_col, k_col, v_col, g_col, a_col;
    const float* x;             // decays' logits [tokens, ldx], heads x dim
    long long ldx;
    const float *w0, *a0, *gain;
    float* vecs;                // [tokens, heads, 3, dim]: w, u, a u
    float* state;
    long long slot_floats, state_offset;
    const int *seq_starts, *seq_slots;
    void* y;
    long long ldy;
    float* o_raw;               // [tokens, heads * dim], or null: the block holds whole heads
    int tokens, heads, dim, cols, tile, wide;
    float unit_eps, eps, decay_scale;
};

// a warp per (token, head)
__global__ void __launch_bounds__(128) general_delta_prepare_kernel(const DeltaParams p) {
    const int lane = threadIdx.x & 31;
    const long long i = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (i >= (long long)p.tokens * p.heads) return;
    const int t = (int)(i / p.heads), h = (int)(i % p.heads), at = h * p.dim;
    const float* row = p.proj + (size_t)t * p.ldp;
    float kk = 0.f;
    for (int d = lane; d < p.dim; d += 32) {
        const float k = row[p.k_col + at + d];
        kk = fmaf(k, k, kk);
    }
    const float inv = 1.0f / sqrtf(warp_sum(kk) + p.unit_eps);
    float* out = p.vecs + (size_t)i * 3 * p.dim;
    for (int d = lane; d < p.dim; d += 32) {
        const float u = row[p.k_col + at + d] * inv;
        out[d] = decay_exp(-p.decay_scale * sigmoid_f(p.x[(size_t)t * p.ldx + at + d] + p.w0[at + d]));
        out[p.dim + d] = u;
        out[2 * p.dim + d] = sigmoid_f(row[p.a_col + at + d] + p.a0[at + d]) * u;
    }
}

// y = o / rms(o) * gain * sigmoid(g), o dim values in shared or global memory, a warp
template <typename TO>
__device__ __forceinline__ void norm_and_gate(const DeltaParams& p, const float* o, size_t t, int h, int lane) {
    float ss = 0.f;
    for (int d = lane; d < p.dim; d += 32) ss = fmaf(o[d], o[d], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
    const float* g = p.proj + t * p.ldp + p.g_col + h * p.dim;
    TO* out = (TO*)p.y + t * p.ldy + h * p.dim;
    for (int d = lane; d < p.dim; d += 32) out[d] = from_f32<TO>(o[d] * inv * p.gain[h * p.dim + d] * sigmoid_f(g[d]));
}

template <typename TO>
__global__ void __launch_bounds__(128) general_delta_output_kernel(const DeltaParams p) {
    const long long i = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (i >= (long long)p.tokens * p.heads) return;
    norm_and_gate<TO>(p, p.o_raw + (size_t)i * p.dim, (size_t)(i / p.heads), (int)(i % p.heads), threadIdx.x & 31);
}

template <typename TO, int R, int P, int COLS>
__global__ void __launch_bounds__(512, 1) general_delta_kernel(const DeltaParams p) {
    extern __shared__ __align__(16) float smem[];
    constexpr int RS = R + PAD, DS = RS * P;        // a part's stride, a staged vector's length (rows beyond dim hold zeros)
    const int dim = p.dim, cols = p.cols, vcols = (cols + 3) & ~3, TILE = p.tile;
    const int stage_floats = TILE * (VECS * DS + vcols);
    float* s_o = smem + 2 * stage_floats;           // [TILE, cols]
    const int head = blockIdx.x, seq = blockIdx.y, j0 = blockIdx.z * cols;
    const int start = p.seq_starts[seq], count = p.seq_starts[seq + 1] - start;
    const int jl = threadIdx.x / P * COLS, part = threadIdx.x % P;
    const int width = min(cols, dim - j0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    float* S = p.state + (size_t)p.seq_slots[seq] * p.slot_floats + p.state_offset + ((size_t)head * dim + j0 + jl) * dim + part * R;
    float s[COLS][R];
#pragma unroll
    for (int c = 0; c < COLS; ++c)
#pragma unroll
        for (int r = 0; r < R; ++r) s[c][r] = (jl + c < width && part * R + r < dim) ? S[(size_t)c * dim + r] : 0.f;
    for (int i = threadIdx.x; i < 2 * stage_floats; i += blockDim.x) smem[i] = 0.f;      // rows beyond dim stay zero
    __syncthreads();
    // vector v of a tile: [v][token][DS]; then the values [token][vcols]
    auto fetch = [&](int ti, int b) {
        const int t0 = ti * TILE, n = min(TILE, count - t0);
        float* base = smem + b * stage_floats;
        float* sv = base + VECS * TILE * DS;
        if (p.wide) {
            const int pieces = dim / 4;
            for (int i = threadIdx.x; i < n * pieces; i += blockDim.x) {
                const int t = i / pieces, d = (i % pieces) * 4;
                const size_t tok = (size_t)(start + t0 + t);
                const float* vec = p.vecs + (tok * p.heads + head) * 3 * dim + d;
                const float* row = p.proj + tok * p.ldp + head * dim + d;
                float* dst = base + t * DS + (d / R) * RS + d % R;
                copy_async_16(dst, vec);
                copy_async_16(dst + TILE * DS, vec + dim);
                copy_async_16(dst + 2 * TILE * DS, vec + 2 * dim);
                copy_async_16(dst + 3 * TILE * DS, row + p.k_col);
                copy_async_16(dst + 4 * TILE * DS, row + p.r_col);
            }
            const int vp = width / 4;
            for (int i = threadIdx.x; i < n * vp; i += blockDim.x) {
                const int t = i / vp, d = (i % vp) * 4;
                copy_async_16(sv + t * vcols + d, p.proj + (size_t)(start + t0 + t) * p.ldp + p.v_col + head * dim + j0 + d);
            }
        } else {
            for (int i = threadIdx.x; i < n * dim; i += blockDim.x) {
                const int t = i / dim, d = i % dim;
                const size_t tok = (size_t)(start + t0 + t);
                const float* vec = p.vecs + (tok * p.heads + head) * 3 * dim + d;
                const float* row = p.proj + tok * p.ldp + head * dim + d;
                float* dst = base + t * DS + (d / R) * RS + d % R;
                copy_async_4(dst, vec);
                copy_async_4(dst + TILE * DS, vec + dim);
                copy_async_4(dst + 2 * TILE * DS, vec + 2 * dim);
                copy_async_4(dst + 3 * TILE * DS, row + p.k_col);
                copy_async_4(dst + 4 * TILE * DS, row + p.r_col);
            }
            for (int i = threadIdx.x; i < n * width; i += blockDim.x) {
                const int t = i / width, d = i % width;
                copy_async_4(sv + t * vcols + d, p.proj + (size_t)(start + t0 + t) * p.ldp + p.v_col + head * dim + j0 + d);
            }
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    const int tiles = (count + TILE - 1) / TILE;
    if (tiles > 0) fetch(0, 0);
    for (int ti = 0; ti < tiles; ++ti) {
        const int t0 = ti * TILE, n = min(TILE, count - t0);
        if (ti + 1 < tiles) {
            fetch(ti + 1, (ti + 1) & 1);
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();                            // this tile has arrived; the tile before is done with s_o
        const float* base = smem + (ti & 1) * stage_floats;
        const float* s_v = base + VECS * TILE * DS;
        auto step = [&](int t) {
            const float* at = base + t * DS + part * RS;
            auto piece = [&](int v, int r) { return *reinterpret_cast<const float4*>(at + v * TILE * DS + r); };
            // what the old state holds along the unit key
            float held[COLS][2] = {};
#pragma unroll
            for (int r = 0; r < R; r += 4) {
                const float4 u = piece(1, r);
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    held[c][0] = fmaf(s[c][r], u.x, held[c][0]);
                    held[c][1] = fmaf(s[c][r + 1], u.y, held[c][1]);
                    held[c][0] = fmaf(s[c][r + 2], u.z, held[c][0]);
                    held[c][1] = fmaf(s[c][r + 3], u.w, held[c][1]);
                }
            }
            float off[COLS], value[COLS], read[COLS][2] = {};
#pragma unroll
            for (int c = 0; c < COLS; ++c) {
                off[c] = held[c][0] + held[c][1];
                value[c] = s_v[t * vcols + jl + c];
            }
            // meanwhile the rows decay and take in the value
#pragma unroll
            for (int r = 0; r < R; r += 4) {
                const float4 w = piece(0, r), k = piece(3, r);
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    s[c][r] = fmaf(k.x, value[c], w.x * s[c][r]);
                    s[c][r + 1] = fmaf(k.y, value[c], w.y * s[c][r + 1]);
                    s[c][r + 2] = fmaf(k.z, value[c], w.z * s[c][r + 2]);
                    s[c][r + 3] = fmaf(k.w, value[c], w.w * s[c][r + 3]);
                }
            }
#pragma unroll
            for (int o = 1; o < P; o <<= 1)
#pragma unroll
                for (int c = 0; c < COLS; ++c) off[c] += __shfl_xor_sync(0xffffffffu, off[c], o);
#pragma unroll
            for (int r = 0; r < R; r += 4) {
                const float4 a = piece(2, r), q = piece(4, r);
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    s[c][r] = fmaf(-a.x, off[c], s[c][r]);
                    s[c][r + 1] = fmaf(-a.y, off[c], s[c][r + 1]);
                    s[c][r + 2] = fmaf(-a.z, off[c], s[c][r + 2]);
                    s[c][r + 3] = fmaf(-a.w, off[c], s[c][r + 3]);
                    read[c][0] = fmaf(s[c][r], q.x, read[c][0]);
                    read[c][1] = fmaf(s[c][r + 1], q.y, read[c][1]);
                    read[c][0] = fmaf(s[c][r + 2], q.z, read[c][0]);
                    read[c][1] = fmaf(s[c][r + 3], q.w, read[c][1]);
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
        if (n == TILE && TILE == 16) {              // a whole tile: unrolled, so that the loads of the next tokens go out ahead of their steps
#pragma unroll 4
            for (int t = 0; t < 16; ++t) step(t);
        } else {
            for (int t = 0; t < n; ++t) step(t);
        }
        __syncthreads();                            // the tile's outputs are complete; its buffer may be filled again
        if (p.o_raw) {
            for (int i = threadIdx.x; i < n * width; i += blockDim.x) {
                const int t = i / width, d = i % width;
                p.o_raw[(size_t)(start + t0 + t) * ((size_t)p.heads * dim) + head * dim + j0 + d] = s_o[t * cols + d];
            }
        } else {
            for (int t = warp; t < n; t += warps) norm_and_gate<TO>(p, s_o + t * cols, (size_t)(start + t0 + t), head, lane);
        }
    }
#pragma unroll
    for (int c = 0; c < COLS; ++c)
#pragma unroll
        for (int r = 0; r < R; ++r)
            if (jl + c < width && part * R + r < dim) S[(size_t)c * dim + r] = s[c][r];
}

template <typename TO, int R, int P, int COLS>
int launch_general_delta(cudaStream_t stream, DeltaParams p, int slices, int num_seqs) {
    // columns a block: whole warps of them, a multiple of four (the slices' values start on 16-byte boundaries)
    constexpr int per_warp = 32 / P * COLS < 4 ? 4 : 32 / P * COLS;
    const int most = 512 / P * COLS / per_warp * per_warp;
    if (!p.o_raw) slices = 1;
    int cols = (p.dim + slices - 1) / slices;
    cols = std::min((cols + per_warp - 1) / per_warp * per_warp, most);
    slices = (p.dim + cols - 1) / cols;
    if (slices > 1 && !p.o_raw) return (int)cudaErrorInvalidValue;
    if (slices == 1) p.o_raw = nullptr;
    p.cols = cols;
    const int threads = cols / COLS * P, vcols = (cols + 3) & ~3;
    auto bytes = [&](int tile) { return ((size_t)2 * tile * (VECS * (R + PAD) * P + vcols) + (size_t)tile * cols) * sizeof(float); };
    p.tile = 16;
    while (p.tile > 2 && bytes(p.tile) > 200 * 1024) p.tile /= 2;
    const size_t smem = bytes(p.tile);
    if (threads > 512 || smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    auto kernel = general_delta_kernel<TO, R, P, COLS>;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    p.wide = p.dim % 4 == 0 && p.ldp % 4 == 0 && p.r_col % 4 == 0 && p.k_col % 4 == 0 && p.v_col % 4 == 0 && (uintptr_t)p.proj % 16 == 0 && (uintptr_t)p.vecs % 16 == 0;
    const long long warps = (long long)p.tokens * p.heads;
    general_delta_prepare_kernel<<<(unsigned)((warps + 3) / 4), 128, 0, stream>>>(p);
    kernel<<<dim3(p.heads, num_seqs, slices), threads, smem, stream>>>(p);
    if (p.o_raw) general_delta_output_kernel<TO><<<(unsigned)((warps + 3) / 4), 128, 0, stream>>>(p);
    return eg_launch_status();
}

template <typename TO>
int dispatch_general_delta(cudaStream_t stream, const DeltaParams& p, int slices, int num_seqs) {
    if (p.dim <= 16) return launch_general_delta<TO, 4, 4, 1>(stream, p, slices, num_seqs);
    if (p.dim <= 32) return launch_general_delta<TO, 8, 4, 1>(stream, p, slices, num_seqs);
    if (p.dim <= 64) return launch_general_delta<TO, 8, 8, 2>(stream, p, slices, num_seqs);
    if (p.dim <= 128) return launch_general_delta<TO, 8, 16, 2>(stream, p, slices, num_seqs);
    return launch_general_delta<TO, 8, 32, 2>(stream, p, slices, num_seqs);
}

template <typename T>
__global__ void tanh_columns_kernel(const float* __restrict__ src, long long lds, T* __restrict__ dst, long long ldd, int rows, int cols, int padded) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)rows * padded) return;
    const int t = (int)(i / padded), c = (int)(i % padded);
    dst[(size_t)t * ldd + c] = from_f32<T>(c < cols ? tanhf(src[(size_t)t * lds + c]) : 0.f);
}
}  // namespace

// proj float32 [tokens, ldp] with r, k, v, g (the output gate) and a (the removal rates' logits, bias a0 still to be added), heads x dim
// each, at their columns; x float32 [tokens, ldx]: the decays' logits (w0 still to be added); a0, w0, gain float32 [heads * dim].
// vecs float32 [tokens, heads, 3, dim] of scratch.  state: the requests' slots; S of a request lies state_offset floats into its
// slot.  y [tokens, ldy] in y_dtype.  slices > 1 (with o_raw float32 [tokens, heads * dim]): a head's columns are dealt to that many
// blocks, and the outputs are normed by a kernel behind.  dim up to 256.
EG_API int eg_general_delta(cudaStream_t stream, const float* proj, long long ldp, int r_col, int k_col, int v_col, int g_col, int a_col, const float* x,
                            long long ldx, const float* w0, const float* a0, const float* gain, float* vecs, float* state, long long slot_floats,
                            long long state_offset, const int* seq_starts, const int* seq_slots, void* y, int y_dtype, long long ldy, float* o_raw, int slices,
                            int tokens, int num_seqs, int heads, int dim, float unit_eps, float eps, float decay_scale) {
    if (num_seqs <= 0 || tokens <= 0) return 0;
    if (heads <= 0 || dim <= 0 || dim > 256 || slices < 1 || !vecs) return (int)cudaErrorInvalidValue;
    DeltaParams p{};
    p.proj = proj;
    p.ldp = ldp;
    p.r_col = r_col;
    p.k_col = k_col;
    p.v_col = v_col;
    p.g_col = g_col;
    p.a_col = a_col;
    p.x = x;
    p.ldx = ldx;
    p.w0 = w0;
    p.a0 = a0;
    p.gain = gain;
    p.vecs = vecs;
    p.state = state;
    p.slot_floats = slot_floats;
    p.state_offset = state_offset;
    p.seq_starts = seq_starts;
    p.seq_slots = seq_slots;
    p.y = y;
    p.ldy = ldy;
    p.o_raw = o_raw;
    p.tokens = tokens;
    p.heads = heads;
    p.dim = dim;
    p.unit_eps = unit_eps;
    p.eps = eps;
    p.decay_scale = decay_scale;
    return y_dtype == EG_BF16 ? dispatch_general_delta<bf16>(stream, p, slices, num_seqs) : dispatch_general_delta<float>(stream, p, slices, num_seqs);
}

// dst [rows, ldd] in dst_dtype: column c < cols holds tanh(src[., c]), columns up to `padded` hold zeros
EG_API int eg_tanh_columns(cudaStream_t stream, const float* src, long long lds, void* dst, int dst_dtype, long long ldd, int rows, int cols, int padded) {
    if (rows <= 0 || padded <= 0) return 0;
    const unsigned blocks = (unsigned)(((long long)rows * padded + 255) / 256);
    if (dst_dtype == EG_BF16) tanh_columns_kernel<bf16><<<blocks, 256, 0, stream>>>(src, lds, (bf16*)dst, ldd, rows, cols, padded);
    else tanh_columns_kernel<float><<<blocks, 256, 0, stream>>>(src, lds, (float*)dst, ldd, rows, cols, padded);
    return eg_launch_status();
}
