// Linear attention whose state fades by a constant of the head ("lightning attention"): per head a matrix S [dk, dv] (float32,
// in the request's state slot),
//
//   q, k, v <- silu(.);   S <- lambda_h S + k v^T;   o = S^T q
//   out = o / sqrt(mean(o^2) + eps) * gain * sigmoid(g)                 (mean over all heads' values together)
//
// q, k, v and g are columns of one projection's float32 output.  All sums are float32 in both precisions.
//
// Two forms of the recurrence.
//
// Steps of short entries (decoding): one block per (head, batch entry, slice of the head's columns).  A column of S belongs to P
// neighbouring lanes, each with R of its rows in registers (lane p has rows 4 (i P + p) .. + 3), token after token.
//
// Longer entries: the entry is cut into chunks of C = 64 tokens.  With i, j counting inside a chunk and S the state in front of it,
//   o_i = lambda^(i+1) S^T q_i + sum_{j <= i} lambda^(i-j) (q_i . k_j) v_j,      S' = lambda^n S + sum_j lambda^(n-1-j) k_j v_j^T
// so that three kernels do it: the chunks' own contributions to the state (all chunks at once), a pass over the entry's chunks that turns
// them into the states in front of every chunk (element by element, in order), and the chunks' outputs (all at once).  In float32
// the products are multiply-adds on pairs, out of tiles of 64 x 64 in shared memory.  In bfloat16 they run on the warp-level tensor
// cores with float32 sums: q, k and v (activated projections) are rounded to bfloat16, but what belongs to the state is not: the keys
// with their decay, and the states that the queries read, go in as the sum of two bfloat16 numbers each (16 bits of mantissa), two
// products instead of one; the states themselves stay float32.  A portion's end may cut a chunk: the sums then group
// differently, which is a difference of rounding.
//
// A kernel behind norms and gates.  The slot keeps S as [head, column, row].
#include <algorithm>

#include "mma_utils.cuh"

namespace {
constexpr int TILE = 16;                            // tokens a step of the short form
constexpr int C = 64, LD = C + 4;                   // a chunk's tokens and the tiles' edge; a staged row's stride
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ float sum_of(uint64_t v) {
    float lo, hi;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
    return lo + hi;
}

struct LightningParams {
    const float* proj;          // [tokens, ldp]
    long long ldp;
    int q_col, k_col, v_col, g_col;
    const float* powers;        // [heads, C + 1]: lambda^0 .. lambda^C
    const float* gain;
    float* state;
    long long slot_floats, state_offset;
    const int *seq_starts, *seq_slots;
    float* o_raw;               // [tokens, heads * dv]
    float* chunks;              // [chunk, heads, dv, dk]: contributions, then the states in front of the chunks
    int tokens, num_seqs, heads, dk, dv, cols;
};

// ---- short entries -------------------------------------------------------------------------------------------------------------
template <int R, int P>
__global__ void __launch_bounds__(512, 1) lightning_short_kernel(const LightningParams p) {
    extern __shared__ __align__(16) float smem[];
    constexpr int DS = R * P;
    const int cols = p.cols, dk = p.dk, dv = p.dv;
    float* s_q = smem;                              // [TILE][DS]
    float* s_k = s_q + TILE * DS;
    float* s_v = s_k + TILE * DS;                   // [TILE][cols]
    const int head = blockIdx.x, seq = blockIdx.y, j0 = blockIdx.z * cols;
    const int start = p.seq_starts[seq], count = p.seq_starts[seq + 1] - start;
    const int jl = threadIdx.x / P, part = threadIdx.x % P;
    const int width = min(cols, dv - j0);
    const bool mine = jl < width;
    const float decay = p.powers[head * (C + 1) + 1];
    float* S = p.state + (size_t)p.seq_slots[seq] * p.slot_floats + p.state_offset + ((size_t)head * dv + j0 + jl) * dk;
    float s[R];
    const bool vec = dk % 4 == 0;
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        const int row = (i * P + part) * 4;
        if (vec) {
            const float4 f = mine && row < dk ? *reinterpret_cast<const float4*>(S + row) : make_float4(0.f, 0.f, 0.f, 0.f);
            s[4 * i] = f.x; s[4 * i + 1] = f.y; s[4 * i + 2] = f.z; s[4 * i + 3] = f.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) s[4 * i + e] = mine && row + e < dk ? S[row + e] : 0.f;
        }
    }
    for (int t0 = 0; t0 < count; t0 += TILE) {
        const int n = min(TILE, count - t0);
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float* row = p.proj + (size_t)(start + t0 + t) * p.ldp;
            for (int d = threadIdx.x; d < DS; d += blockDim.x) {
                s_q[t * DS + d] = d < dk ? silu_f(row[p.q_col + head * dk + d]) : 0.f;
                s_k[t * DS + d] = d < dk ? silu_f(row[p.k_col + head * dk + d]) : 0.f;
            }
            for (int d = threadIdx.x; d < width; d += blockDim.x) s_v[t * cols + d] = silu_f(row[p.v_col + head * dv + j0 + d]);
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float value = mine ? s_v[t * cols + jl] : 0.f;
            float read = 0.f;
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const int row = (i * P + part) * 4;
                const float4 k = *reinterpret_cast<const float4*>(s_k + t * DS + row), q = *reinterpret_cast<const float4*>(s_q + t * DS + row);
                s[4 * i] = fmaf(k.x, value, decay * s[4 * i]);
                s[4 * i + 1] = fmaf(k.y, value, decay * s[4 * i + 1]);
                s[4 * i + 2] = fmaf(k.z, value, decay * s[4 * i + 2]);
                s[4 * i + 3] = fmaf(k.w, value, decay * s[4 * i + 3]);
                read = fmaf(s[4 * i], q.x, read);
                read = fmaf(s[4 * i + 1], q.y, read);
                read = fmaf(s[4 * i + 2], q.z, read);
                read = fmaf(s[4 * i + 3], q.w, read);
            }
#pragma unroll
            for (int x = 1; x < P; x <<= 1) read += __shfl_xor_sync(0xffffffffu, read, x);
            if (part == 0 && mine) p.o_raw[(size_t)(start + t0 + t) * ((size_t)p.heads * dv) + head * dv + j0 + jl] = read;
        }
    }
    if (!mine) return;
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        const int row = (i * P + part) * 4;
        if (vec) {
            if (row < dk) *reinterpret_cast<float4*>(S + row) = make_float4(s[4 * i], s[4 * i + 1], s[4 * i + 2], s[4 * i + 3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (row + e < dk) S[row + e] = s[4 * i + e];
        }
    }
}

// ---- chunks --------------------------------------------------------------------------------------------------------------------
// which entry and which of its tokens chunk number `index` (over all entries, in order) covers; count 0: there is no such chunk
__device__ __forceinline__ void find_chunk(const LightningParams& p, int index, int* seq, int* first, int* count) {
    *count = 0;
    for (int s = 0; s < p.num_seqs; ++s) {
        const int lo = p.seq_starts[s], n = p.seq_starts[s + 1] - lo, chunks = (n + C - 1) / C;
        if (index < chunks) {
            *seq = s;
            *first = lo + index * C;
            *count = min(C, n - index * C);
            return;
        }
        index -= chunks;
    }
}

// acc[r][c] += sum over 64 of X[ty + 16 r][.] Y[tx + 16 c][.], rows LD floats apart, pairs of partial sums
__device__ __forceinline__ void product_64(uint64_t (&acc)[4][4], const float* X, const float* Y, int ty, int tx) {
#pragma unroll 4
    for (int d = 0; d < C; d += 4) {
        ulonglong2 x[4], y[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            x[r] = *reinterpret_cast<const ulonglong2*>(X + (ty + 16 * r) * LD + d);
            y[r] = *reinterpret_cast<const ulonglong2*>(Y + (tx + 16 * r) * LD + d);
        }
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[r][c] = fma2(x[r].y, y[c].y, fma2(x[r].x, y[c].x, acc[r][c]));
    }
}
__device__ __forceinline__ void clear(uint64_t (&acc)[4][4]) {
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[r][c] = 0ull;
}
// a block of 64 tokens x 64 columns of the projection, activated: tile[token][column] (or, TURNED, tile[column][token]); zeros outside
template <bool TURNED>
__device__ __forceinline__ void stage(float* tile, const LightningParams& p, int first, int count, int col, int cols, const float* scale) {
    for (int i = threadIdx.x; i < C * C; i += 256) {
        const int t = i / C, d = i % C;
        float v = 0.f;
        if (t < count && d < cols) {
            v = silu_f(p.proj[(size_t)(first + t) * p.ldp + col + d]);
            if (scale) v *= scale[count - 1 - t];
        }
        tile[TURNED ? d * LD + t : t * LD + d] = v;
    }
}

// grid (chunks, heads, blocks of 64 rows x 64 columns of S): the chunk's own contribution to the state behind it
__global__ void __launch_bounds__(256) lightning_chunk_state_kernel(const LightningParams p) {
    extern __shared__ __align__(16) float smem[];
    float *s_v = smem, *s_k = smem + C * LD;        // [column][token], [row][token]
    int seq, first, count;
    find_chunk(p, blockIdx.x, &seq, &first, &count);
    if (count == 0) return;
    const int head = blockIdx.y, row_blocks = (p.dk + C - 1) / C, d0 = blockIdx.z % row_blocks * C, v0 = blockIdx.z / row_blocks * C;
    const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    stage<true>(s_k, p, first, count, p.k_col + head * p.dk + d0, min(C, p.dk - d0), p.powers + head * (C + 1));
    stage<true>(s_v, p, first, count, p.v_col + head * p.dv + v0, min(C, p.dv - v0), nullptr);
    __syncthreads();
    uint64_t acc[4][4];
    clear(acc);
    product_64(acc, s_v, s_k, ty, tx);
    float* out = p.chunks + ((size_t)blockIdx.x * p.heads + head) * p.dv * p.dk;
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int v = v0 + ty + 16 * r, d = d0 + tx + 16 * c;
            if (v < p.dv && d < p.dk) out[(size_t)v * p.dk + d] = sum_of(acc[r][c]);
        }
}

// grid (elements of a head's S / 256 / VEC, heads, entries): contributions -> states in front of the chunks; the slot takes the last state
template <int VEC>
__global__ void __launch_bounds__(256) lightning_chunk_scan_kernel(const LightningParams p) {
    struct alignas(VEC * 4) Part { float v[VEC]; };
    const int e = (blockIdx.x * blockDim.x + threadIdx.x) * VEC, head = blockIdx.y, seq = blockIdx.z, size = p.dk * p.dv;
    if (e >= size) return;
    int index = 0;
    for (int s = 0; s < seq; ++s) index += (p.seq_starts[s + 1] - p.seq_starts[s] + C - 1) / C;
    const int n = p.seq_starts[seq + 1] - p.seq_starts[seq], chunks = (n + C - 1) / C;
    Part* slot = reinterpret_cast<Part*>(p.state + (size_t)p.seq_slots[seq] * p.slot_floats + p.state_offset + (size_t)head * size + e);
    Part* at = reinterpret_cast<Part*>(p.chunks + ((size_t)index * p.heads + head) * size + e);
    const size_t stride = (size_t)p.heads * size / VEC;
    const float whole = p.powers[head * (C + 1) + C], rest = p.powers[head * (C + 1) + (n - 1) % C + 1];
    Part S = *slot;
    auto take = [&](int c, Part own) {
        at[(size_t)c * stride] = S;
        const float f = c + 1 < chunks ? whole : rest;
#pragma unroll
        for (int i = 0; i < VEC; ++i) S.v[i] = fmaf(f, S.v[i], own.v[i]);
    };
    int c = 0;
    for (; c + 8 <= chunks; c += 8) {               // eight loads on their way at a time
        Part own[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) own[i] = at[(size_t)(c + i) * stride];
#pragma unroll
        for (int i = 0; i < 8; ++i) take(c + i, own[i]);
    }
    for (; c < chunks; ++c) take(c, at[(size_t)c * stride]);
    *slot = S;
}

// grid (chunks, heads, blocks of 64 columns): the chunk's outputs
__global__ void __launch_bounds__(256) lightning_chunk_out_kernel(const LightningParams p) {
    extern __shared__ __align__(16) float smem[];
    float *s_q = smem, *s_k = s_q + C * LD, *s_s = s_k + C * LD, *s_pow = s_s + C * LD;     // s_pow [C + 1]
    int seq, first, count;
    find_chunk(p, blockIdx.x, &seq, &first, &count);
    if (count == 0) return;
    const int head = blockIdx.y, v0 = blockIdx.z * C;
    const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    if (threadIdx.x <= C) s_pow[threadIdx.x] = p.powers[head * (C + 1) + threadIdx.x];
    const float* S = p.chunks + ((size_t)blockIdx.x * p.heads + head) * p.dv * p.dk;
    uint64_t own[4][4], old[4][4];
    clear(own);
    clear(old);
    for (int d0 = 0; d0 < p.dk; d0 += C) {
        __syncthreads();
        stage<false>(s_q, p, first, count, p.q_col + head * p.dk + d0, min(C, p.dk - d0), nullptr);
        stage<false>(s_k, p, first, count, p.k_col + head * p.dk + d0, min(C, p.dk - d0), nullptr);
        for (int i = threadIdx.x; i < C * C; i += 256) {
            const int v = i / C, d = i % C;
            s_s[v * LD + d] = v0 + v < p.dv && d0 + d < p.dk ? S[(size_t)(v0 + v) * p.dk + d0 + d] : 0.f;
        }
        __syncthreads();
        product_64(own, s_q, s_k, ty, tx);          // q_i . k_j
        product_64(old, s_q, s_s, ty, tx);          // S^T q_i
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int i = ty + 16 * r, j = tx + 16 * c;
            s_q[i * LD + j] = j <= i ? s_pow[i - j] * sum_of(own[r][c]) : 0.f;
        }
    stage<true>(s_k, p, first, count, p.v_col + head * p.dv + v0, min(C, p.dv - v0), nullptr);      // [column][token]
    __syncthreads();
    clear(own);
    product_64(own, s_q, s_k, ty, tx);
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int i = ty + 16 * r, v = tx + 16 * c;
            if (i < count && v0 + v < p.dv)
                p.o_raw[(size_t)(first + i) * ((size_t)p.heads * p.dv) + head * p.dv + v0 + v] = fmaf(s_pow[i + 1], sum_of(old[r][c]), sum_of(own[r][c]));
        }
}

// ---- chunks on the tensor cores --------------------------------------------------------------------------------------------------
constexpr int VB = 128, DB = 128;                   // columns and rows of S a block works on
__device__ __forceinline__ void split_bf16(float x, bf16& hi, bf16& lo) {
    hi = __float2bfloat16_rn(x);
    lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}
// a chunk's columns of the projection, activated, in bfloat16: tile[token][column] (rows `ld` apart), zeros outside; with `scale` (the
// decay's powers) times scale[count - 1 - t] and, into `low`, what the rounding lost
template <int COLS, bool SPLIT>
__device__ __forceinline__ void stage_bf16(bf16* tile, bf16* low, int ld, const LightningParams& p, int first, int count, int col, int cols, bool wide,
                                           const float* scale) {
    for (int i = threadIdx.x; i < C * (COLS / 4); i += 256) {
        const int t = i / (COLS / 4), d = i % (COLS / 4) * 4;
        float v[4] = {0.f, 0.f, 0.f, 0.f};
        if (t < count && d < cols) {
            const float* src = p.proj + (size_t)(first + t) * p.ldp + col + d;
            if (wide) {
                const float4 f = *reinterpret_cast<const float4*>(src);
                v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) v[e] = d + e < cols ? src[e] : 0.f;
            }
            const float f = SPLIT ? scale[count - 1 - t] : 1.f;
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] = __fdividef(v[e], 1.0f + __expf(-v[e])) * f;
        }
        if (SPLIT) {
            __align__(8) bf16 hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) split_bf16(v[e], hi[e], lo[e]);
            *reinterpret_cast<uint2*>(tile + t * ld + d) = *reinterpret_cast<uint2*>(hi);
            *reinterpret_cast<uint2*>(low + t * ld + d) = *reinterpret_cast<uint2*>(lo);
        } else {
            *reinterpret_cast<uint2*>(tile + t * ld + d) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
        }
    }
}

// grid (chunks, heads, blocks of DB rows x VB columns of S): warp w takes columns 16 w .. 16 w + 15 of the block
__global__ void __launch_bounds__(256, 2) lightning_state_mma_kernel(const LightningParams p, int wide) {
    extern __shared__ __align__(16) unsigned char raw[];
    constexpr int KL = DB + 8, VL = VB + 8;
    bf16 *s_hi = (bf16*)raw, *s_lo = s_hi + C * KL, *s_v = s_lo + C * KL;      // keys [token][row] twice, values [token][column]
    int seq, first, count;
    find_chunk(p, blockIdx.x, &seq, &first, &count);
    if (count == 0) return;
    const int head = blockIdx.y, row_blocks = (p.dk + DB - 1) / DB, d0 = blockIdx.z % row_blocks * DB, v0 = blockIdx.z / row_blocks * VB;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, m0 = warp * 16;
    stage_bf16<DB, true>(s_hi, s_lo, KL, p, first, count, p.k_col + head * p.dk + d0, min(DB, p.dk - d0), wide, p.powers + head * (C + 1));
    stage_bf16<VB, false>(s_v, nullptr, VL, p, first, count, p.v_col + head * p.dv + v0, min(VB, p.dv - v0), wide, nullptr);
    __syncthreads();
    if (v0 + m0 >= p.dv) return;
    float acc[DB / 8][4] = {};
#pragma unroll
    for (int k0 = 0; k0 < C; k0 += 16) {
        uint32_t a[4];                              // values turned: rows of the product are columns of S
        ldmatrix_x4_trans(a, s_v + (k0 + (lane & 7) + ((lane >> 4) & 1) * 8) * VL + m0 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int np = 0; np < DB / 16; ++np) {
            if (d0 + np * 16 >= p.dk) break;
            const int at = (k0 + ((lane >> 3) & 1) * 8 + (lane & 7)) * KL + np * 16 + (lane >> 4) * 8;
            uint32_t b[4];
            ldmatrix_x4_trans(b, s_hi + at);
            mma_bf16_16816(acc[2 * np], a, b[0], b[1]);
            mma_bf16_16816(acc[2 * np + 1], a, b[2], b[3]);
            ldmatrix_x4_trans(b, s_lo + at);
            mma_bf16_16816(acc[2 * np], a, b[0], b[1]);
            mma_bf16_16816(acc[2 * np + 1], a, b[2], b[3]);
        }
    }
    float* out = p.chunks + ((size_t)blockIdx.x * p.heads + head) * p.dv * p.dk;
#pragma unroll
    for (int nt = 0; nt < DB / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int v = v0 + m0 + (lane >> 2) + (e ? 8 : 0), d = d0 + nt * 8 + 2 * (lane & 3);
            if (v >= p.dv || d >= p.dk) continue;
            float* at = out + (size_t)v * p.dk + d;
            if (p.dk % 2 == 0) {
                *reinterpret_cast<float2*>(at) = make_float2(acc[nt][e], acc[nt][e + 1]);
            } else {
                at[0] = acc[nt][e];
                if (d + 1 < p.dk) at[1] = acc[nt][e + 1];
            }
        }
}

// grid (chunks, heads, blocks of VB columns): warp w takes tokens 16 (w % 4) .. + 15 and half w / 4 of the block's columns
__global__ void __launch_bounds__(256, 2) lightning_out_mma_kernel(const LightningParams p, int wide) {
    extern __shared__ __align__(16) unsigned char raw[];
    constexpr int QL = C + 8, VL = VB + 8;
    bf16 *s_q = (bf16*)raw, *s_k = s_q + C * QL, *s_hi = s_k + C * QL, *s_lo = s_hi + VB * QL, *s_v = s_lo + VB * QL;
    float* s_pow = (float*)(s_v + C * VL);
    int seq, first, count;
    find_chunk(p, blockIdx.x, &seq, &first, &count);
    if (count == 0) return;
    const int head = blockIdx.y, v0 = blockIdx.z * VB;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, m0 = (warp & 3) * 16, half = (warp >> 2) * (VB / 2);
    if (threadIdx.x <= C) s_pow[threadIdx.x] = p.powers[head * (C + 1) + threadIdx.x];
    const float* S = p.chunks + ((size_t)blockIdx.x * p.heads + head) * p.dv * p.dk;
    stage_bf16<VB, false>(s_v, nullptr, VL, p, first, count, p.v_col + head * p.dv + v0, min(VB, p.dv - v0), wide, nullptr);
    float own[C / 8][4] = {}, o[VB / 16][4] = {};   // q . k of the chunk's tokens; S^T q, then the outputs
    for (int d0 = 0; d0 < p.dk; d0 += C) {
        if (d0) __syncthreads();
        const int cols = min(C, p.dk - d0);
        stage_bf16<C, false>(s_q, nullptr, QL, p, first, count, p.q_col + head * p.dk + d0, cols, wide, nullptr);
        stage_bf16<C, false>(s_k, nullptr, QL, p, first, count, p.k_col + head * p.dk + d0, cols, wide, nullptr);
        for (int i = threadIdx.x; i < VB * (C / 4); i += 256) {
            const int v = i / (C / 4), d = i % (C / 4) * 4;
            float x[4] = {0.f, 0.f, 0.f, 0.f};
            if (v0 + v < p.dv && d < cols) {
                const float* src = S + (size_t)(v0 + v) * p.dk + d0 + d;
                if (p.dk % 4 == 0) {
                    const float4 f = *reinterpret_cast<const float4*>(src);
                    x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w;
                } else {
#pragma unroll
                    for (int e = 0; e < 4; ++e) x[e] = d + e < cols ? src[e] : 0.f;
                }
            }
            __align__(8) bf16 hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) split_bf16(x[e], hi[e], lo[e]);
            *reinterpret_cast<uint2*>(s_hi + v * QL + d) = *reinterpret_cast<uint2*>(hi);
            *reinterpret_cast<uint2*>(s_lo + v * QL + d) = *reinterpret_cast<uint2*>(lo);
        }
        __syncthreads();
#pragma unroll
        for (int k0 = 0; k0 < C; k0 += 16) {
            uint32_t a[4], b[4];
            ldmatrix_x4(a, s_q + (m0 + (lane & 15)) * QL + k0 + (lane >> 4) * 8);
            const int row = (lane >> 4) * 8 + (lane & 7), at = k0 + ((lane >> 3) & 1) * 8;
#pragma unroll
            for (int np = 0; np < C / 16; ++np) {
                if (np * 16 > m0 + 15) break;       // keys behind every token of the warp
                ldmatrix_x4(b, s_k + (np * 16 + row) * QL + at);
                mma_bf16_16816(own[2 * np], a, b[0], b[1]);
                mma_bf16_16816(own[2 * np + 1], a, b[2], b[3]);
            }
#pragma unroll
            for (int np = 0; np < VB / 32; ++np) {
                ldmatrix_x4(b, s_hi + (half + np * 16 + row) * QL + at);
                mma_bf16_16816(o[2 * np], a, b[0], b[1]);
                mma_bf16_16816(o[2 * np + 1], a, b[2], b[3]);
                ldmatrix_x4(b, s_lo + (half + np * 16 + row) * QL + at);
                mma_bf16_16816(o[2 * np], a, b[0], b[1]);
                mma_bf16_16816(o[2 * np + 1], a, b[2], b[3]);
            }
        }
    }
    const int lo_row = m0 + (lane >> 2), hi_row = lo_row + 8;
    const float f_lo = s_pow[lo_row + 1], f_hi = s_pow[hi_row + 1];
#pragma unroll
    for (int nt = 0; nt < VB / 16; ++nt) {
        o[nt][0] *= f_lo;
        o[nt][1] *= f_lo;
        o[nt][2] *= f_hi;
        o[nt][3] *= f_hi;
    }
#pragma unroll
    for (int nt = 0; nt < C / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int back = (e < 2 ? lo_row : hi_row) - (nt * 8 + 2 * (lane & 3) + (e & 1));
            own[nt][e] = back >= 0 ? own[nt][e] * s_pow[back] : 0.f;
        }
#pragma unroll
    for (int ks = 0; ks < C / 16; ++ks) {
        if (ks * 16 > m0 + 15) break;
        const uint32_t a[4] = {pack_bf16(own[2 * ks][0], own[2 * ks][1]), pack_bf16(own[2 * ks][2], own[2 * ks][3]),
                               pack_bf16(own[2 * ks + 1][0], own[2 * ks + 1][1]), pack_bf16(own[2 * ks + 1][2], own[2 * ks + 1][3])};
#pragma unroll
        for (int np = 0; np < VB / 32; ++np) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, s_v + (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * VL + half + np * 16 + (lane >> 4) * 8);
            mma_bf16_16816(o[2 * np], a, b[0], b[1]);
            mma_bf16_16816(o[2 * np + 1], a, b[2], b[3]);
        }
    }
    const size_t n = (size_t)p.heads * p.dv;
#pragma unroll
    for (int nt = 0; nt < VB / 16; ++nt)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int i = e ? hi_row : lo_row, v = v0 + half + nt * 8 + 2 * (lane & 3);
            if (i >= count || v >= p.dv) continue;
            float* at = p.o_raw + (size_t)(first + i) * n + head * p.dv + v;
            if (p.dv % 2 == 0) {
                *reinterpret_cast<float2*>(at) = make_float2(o[nt][e], o[nt][e + 1]);
            } else {
                at[0] = o[nt][e];
                if (v + 1 < p.dv) at[1] = o[nt][e + 1];
            }
        }
}

// a block per token
template <typename TO, int VEC>
__global__ void __launch_bounds__(256) lightning_output_kernel(const float* __restrict__ o_raw, const float* __restrict__ proj, long long ldp, int g_col,
                                                               const float* __restrict__ gain, TO* __restrict__ y, long long ldy, int n, float eps) {
    __shared__ float scratch[32];
    const int t = blockIdx.x;
    const float* o = o_raw + (size_t)t * n;
    const float* g = proj + (size_t)t * ldp + g_col;
    TO* out = y + (size_t)t * ldy;
    float ss = 0.f;
    if (VEC == 4) {
        for (int d = threadIdx.x * 4; d < n; d += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(o + d);
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        for (int d = threadIdx.x; d < n; d += blockDim.x) ss = fmaf(o[d], o[d], ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
    if (VEC == 4) {
        for (int d = threadIdx.x * 4; d < n; d += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(o + d), z = *reinterpret_cast<const float4*>(g + d), w = *reinterpret_cast<const float4*>(gain + d);
            const float r0 = v.x * inv * w.x * sigmoid_f(z.x), r1 = v.y * inv * w.y * sigmoid_f(z.y), r2 = v.z * inv * w.z * sigmoid_f(z.z),
                        r3 = v.w * inv * w.w * sigmoid_f(z.w);
            if (sizeof(TO) == 2) {
                __nv_bfloat162 lo = __floats2bfloat162_rn(r0, r1), hi = __floats2bfloat162_rn(r2, r3);
                *reinterpret_cast<uint2*>(out + d) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
            } else {
                *reinterpret_cast<float4*>(out + d) = make_float4(r0, r1, r2, r3);
            }
        }
    } else {
        for (int d = threadIdx.x; d < n; d += blockDim.x) out[d] = from_f32<TO>(o[d] * inv * gain[d] * sigmoid_f(g[d]));
    }
}

template <int R, int P>
int launch_short(cudaStream_t stream, LightningParams p, int slices) {
    constexpr int per_warp = 32 / P;
    const int most = 512 / P / per_warp * per_warp;
    int cols = (p.dv + slices - 1) / slices;
    cols = std::min((cols + per_warp - 1) / per_warp * per_warp, most);
    slices = (p.dv + cols - 1) / cols;
    p.cols = cols;
    const size_t smem = (size_t)TILE * (2 * R * P + cols) * sizeof(float);
    lightning_short_kernel<R, P><<<dim3(p.heads, p.num_seqs, slices), cols * P, smem, stream>>>(p);
    return 0;
}
}  // namespace

// float32 values of scratch that a step of these sizes needs for its chunks, and whether it is run in chunks at all (0: no): entries
// of more than 16 tokens, and not so many short ones beside them that their chunks would be mostly empty
EG_API long long eg_lightning_chunk_floats(int tokens, int num_seqs, int longest_entry, int heads, int dk, int dv) {
    if (longest_entry <= TILE || num_seqs > tokens / 32 + 1) return 0;
    return (long long)(tokens / C + num_seqs) * heads * dk * dv;
}

// proj float32 [tokens, ldp] with q, k (heads x dk), v and g (heads x dv) at their columns; powers float32 [heads, 65]: the decay's powers
// from 0 to 64; gain float32 [heads * dv]; o_raw float32 [tokens, heads * dv] of scratch; chunks: scratch of eg_lightning_chunk_floats values, or
// null: token after token; S of a request lies state_offset floats into its slot.  y [tokens, ldy] in y_dtype.  slices: into how
// many blocks a head's columns are dealt (token after token).  dk up to 256.
EG_API int eg_lightning(cudaStream_t stream, const float* proj, long long ldp, int q_col, int k_col, int v_col, int g_col, const float* powers,
                        const float* gain, float* state, long long slot_floats, long long state_offset, const int* seq_starts, const int* seq_slots,
                        float* o_raw, float* chunks, void* y, int y_dtype, long long ldy, int slices, int tokens, int num_seqs, int heads, int dk, int dv,
                        float eps) {
    if (num_seqs <= 0 || tokens <= 0) return 0;
    if (heads <= 0 || dk <= 0 || dk > 256 || dv <= 0 || slices < 1 || !o_raw) return (int)cudaErrorInvalidValue;
    if (dk % 4 == 0 && (slot_floats % 4 || state_offset % 4 || (uintptr_t)state % 16)) return (int)cudaErrorInvalidValue;
    LightningParams p{proj, ldp, q_col, k_col, v_col, g_col, powers, gain, state, slot_floats, state_offset, seq_starts, seq_slots, o_raw, chunks, tokens, num_seqs,
                      heads, dk, dv, 0};
    if (chunks) {
        const int count = tokens / C + num_seqs;
        auto scan = [&] {
            if (dk * dv % 4 == 0 && slot_floats % 4 == 0 && state_offset % 4 == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)chunks % 16 == 0)
                lightning_chunk_scan_kernel<4><<<dim3((dk * dv / 4 + 255) / 256, heads, num_seqs), 256, 0, stream>>>(p);
            else
                lightning_chunk_scan_kernel<1><<<dim3((dk * dv + 255) / 256, heads, num_seqs), 256, 0, stream>>>(p);
        };
        cudaError_t e;
        if (y_dtype == EG_BF16) {
            const int col_blocks = (dv + VB - 1) / VB, row_blocks = (dk + DB - 1) / DB;
            const int wide = dk % 4 == 0 && dv % 4 == 0 && ldp % 4 == 0 && q_col % 4 == 0 && k_col % 4 == 0 && v_col % 4 == 0 && (uintptr_t)proj % 16 == 0;
            const size_t sums = (size_t)C * (2 * (DB + 8) + VB + 8) * 2, outs = (size_t)(2 * C * (C + 8) + 2 * VB * (C + 8) + C * (VB + 8)) * 2 + (C + 1) * 4;
            e = cudaFuncSetAttribute(lightning_state_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sums);
            if (e == cudaSuccess) e = cudaFuncSetAttribute(lightning_out_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)outs);
            if (e != cudaSuccess) return (int)e;
            lightning_state_mma_kernel<<<dim3(count, heads, row_blocks * col_blocks), 256, sums, stream>>>(p, wide);
            scan();
            lightning_out_mma_kernel<<<dim3(count, heads, col_blocks), 256, outs, stream>>>(p, wide);
        } else {
            const int row_blocks = (dk + C - 1) / C, col_blocks = (dv + C - 1) / C;
            const size_t two = (size_t)2 * C * LD * sizeof(float), three = ((size_t)3 * C * LD + C + 1) * sizeof(float);
            e = cudaFuncSetAttribute(lightning_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)three);
            if (e != cudaSuccess) return (int)e;
            lightning_chunk_state_kernel<<<dim3(count, heads, row_blocks * col_blocks), 256, two, stream>>>(p);
            scan();
            lightning_chunk_out_kernel<<<dim3(count, heads, col_blocks), 256, three, stream>>>(p);
        }
    } else {
        const int rc = dk <= 16    ? launch_short<4, 4>(stream, p, slices)
                       : dk <= 32  ? launch_short<8, 4>(stream, p, slices)
                       : dk <= 64  ? launch_short<8, 8>(stream, p, slices)
                       : dk <= 128 ? launch_short<8, 16>(stream, p, slices)
                                   : launch_short<8, 32>(stream, p, slices);
        if (rc) return rc;
    }
    const int n = heads * dv;
    const bool wide = n % 4 == 0 && ldp % 4 == 0 && g_col % 4 == 0 && ldy % 4 == 0 && (uintptr_t)proj % 16 == 0 && (uintptr_t)o_raw % 16 == 0 &&
                      (uintptr_t)gain % 16 == 0 && (uintptr_t)y % 16 == 0;
#define EG_OUTPUT(TO, VEC) lightning_output_kernel<TO, VEC><<<tokens, 256, 0, stream>>>(o_raw, proj, ldp, g_col, gain, (TO*)y, ldy, n, eps)
    if (y_dtype == EG_BF16) {
        if (wide) EG_OUTPUT(bf16, 4);
        else EG_OUTPUT(bf16, 1);
    } else {
        if (wide) EG_OUTPUT(float, 4);
        else EG_OUTPUT(float, 1);
    }
#undef EG_OUTPUT
    return eg_launch_status();
}
