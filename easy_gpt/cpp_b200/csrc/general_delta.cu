// The generalised delta rule: per head a matrix S [dim, dim] (float32, in the request's state slot) whose rows decay each at a
// rate of its own, from which every token takes off what it holds along the token's unit key (at a rate per row), and into
// which it writes its value along its key; both terms read the old state:
//
//   u = k / sqrt(|k|^2 + unit_eps)                                                      (per head, float32)
//   w = exp(-decay_scale * sigmoid(x + w0)),   a = sigmoid(y + a0)                        (per head and key channel)
//   S <- diag(w) S - (a u)(u^T S) + k v^T;   o = S^T r                                    (o reads the new state)
//   out = o / sqrt(mean(o^2) + eps) * gain * sigmoid(g)                                  (mean per head, gain per head and channel)
//
// r, k, v, y and g are columns of one projection's float32 output; x = W_2 tanh(the projection's last columns).
//
// The recurrence reads a *record* per token and head: the six vectors w, u, a u, k, r, v, each filled up with zeros to DS = R * P
// values, and eight numbers.  Records of a head lie one behind the other, so that a tile of tokens is ONE bulk copy; a kernel over
// all tokens makes them.  In steps whose entries are a few tokens each (decoding) the recurrence's own blocks make them in shared
// memory, and work out x as well (W_2 is small), which saves two kernels and a product.
//
// Recurrence: one block per (head, batch entry, slice of the head's columns: the columns of S do not depend on one another).  COLS
// neighbouring columns of S belong to P neighbouring lanes, each with R of their rows in registers for the entry's whole run of
// tokens (lane p has rows 4 (i P + p) .. + 3: eight neighbouring lanes read 128 neighbouring bytes, what shared memory hands out at a
// time).  All arithmetic on the rows is on pairs of float32.
//
// A token waits for the token before it through what the state holds along its key, h = S^T u: a dot product over the rows and log2 P
// shuffles.  So tokens go in blocks of four (counted from the entry's first token of the step), whose h all come from the state in
// front of the block: with w_i, u_i, ... the block's vectors and W_ij = w_(j+1) .. w_(i-1) channel by channel,
//   h_i = (u_i w_0 .. w_(i-1)) . S - sum_{j<i} (u_i . W_ij a_j u_j) h_j + sum_{j<i} (u_i . W_ij k_j) v_j
// (nothing is divided by a decay).  The record of a block's token i holds u_i w_0 .. w_(i-1) in place of u_i, and the dot products of the
// two sums; four dot products over the rows share their shuffle rounds, and the block's sums are a handful of multiply-adds.  The
// up to three tokens behind the last whole block go one by one.  (Measured on B200, 32 heads of 64, cycles a token: one column a
// thread and P = 4, 516: every warp reads all five vectors for its columns, and shared memory hands out four times the bytes that
// differ; two columns and P = 8, 445; with the outputs of four tokens summed over the lanes together, so that the loads of a token
// do not wait for the stores of the token before, 345; one column a thread, so twice the warps, 302.)
//
// Tiles arrive three stages ahead.  Outputs are normed and gated by the block where it holds a whole head, else by a kernel behind.
// The slot keeps S as [head, column, row].  The order of every sum depends on the sizes and on a token's place in its block.
#include <algorithm>
#include <cstdlib>

#include "common.cuh"
#include "decay_exp.cuh"
#include "mbarrier.cuh"

namespace {

constexpr int VECS = 6, STAGES = 3;
constexpr int BLOCK = 4, NUMBERS = 8;       // tokens of a block; a record's numbers behind its vectors: the factors of h_0..h_2, 0, of v_0..v_2, 0
constexpr unsigned WAIT_LIMIT = 1u << 24;

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint64_t pair_of(float lo, float hi) {
    uint64_t d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float sum_of(uint64_t v) {
    float lo, hi;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
    return lo + hi;
}
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n"
                 ::"r"(smem_addr(dst)), "l"(src), "r"(bytes), "r"(smem_addr(bar)) : "memory");
}

struct DeltaParams {
    const float* proj;          // [tokens, ldp]
    long long ldp;
    int r_col, k_col, v_col, g_col, a_col, inner_col;
    const float* x;             // decays' logits [tokens, ldx], heads x dim; null: worked out from w2 by the recurrence's blocks
    long long ldx;
    const void* w2;             // [heads * dim, ld2] in w2's dtype
    int ld2, rank;
    const float *w0, *a0, *gain;
    float* records;             // [heads, tokens, VECS * DS + NUMBERS]
    float* state;
    long long slot_floats, state_offset;
    const int *seq_starts, *seq_slots;
    void* y;
    long long ldy;
    float* o_raw;               // [tokens, heads * dim], or null: the block holds whole heads
    int tokens, heads, dim, cols, tile, lanes;      // lanes: of the group that makes a record
    float unit_eps, eps, decay_scale;
    int* status;
};

// one channel's six values, into rec[v * DS + d]
__device__ __forceinline__ void put_channel(const DeltaParams& p, const float* row, int at, int d, float x, float inv, float* rec, int DS) {
    const float k = row[p.k_col + at + d], u = k * inv;
    rec[d] = decay_exp(-p.decay_scale * sigmoid_f(x + p.w0[at + d]));
    rec[DS + d] = u;
    rec[2 * DS + d] = sigmoid_f(row[p.a_col + at + d] + p.a0[at + d]) * u;
    rec[3 * DS + d] = k;
    rec[4 * DS + d] = row[p.r_col + at + d];
    rec[5 * DS + d] = row[p.v_col + at + d];
}

// The records of N tokens from token t on (a whole block, or one token of an incomplete one) of the head whose channels start at
// `at`, by a group of lanes (`mask` in the warp), each with CH runs of four channels; WIDE: by 16-byte loads.
template <int N, int CH, bool WIDE>
__device__ __forceinline__ void make_records(const DeltaParams& p, int DS, int t, int h, int lane, int group, unsigned mask) {
    const int at = h * p.dim, REC = VECS * DS + NUMBERS;
    auto over_group = [&](float v) {
        for (int o = group >> 1; o > 0; o >>= 1) v += __shfl_xor_sync(mask, v, o);
        return v;
    };
    auto load = [&](const float* src, int c, float (&v)[4]) {                 // the run's channels of the head
        const int d = (c * group + lane) * 4;
        if (WIDE) {
            const float4 f = d < p.dim ? *reinterpret_cast<const float4*>(src + at + d) : make_float4(0.f, 0.f, 0.f, 0.f);
            v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] = d + e < p.dim ? src[at + d + e] : 0.f;
        }
    };
    float w[N][CH][4], au[N][CH][4], k[N][CH][4], kk[N];
#pragma unroll
    for (int b = 0; b < N; ++b) {
        const float* row = p.proj + (size_t)(t + b) * p.ldp;
        kk[b] = 0.f;
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            load(row + p.k_col, c, k[b][c]);
            load(p.x + (size_t)(t + b) * p.ldx, c, w[b][c]);
            load(row + p.a_col, c, au[b][c]);
        }
    }
    float w0[CH][4], a0[CH][4];
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        load(p.w0, c, w0[c]);
        load(p.a0, c, a0[c]);
    }
#pragma unroll
    for (int b = 0; b < N; ++b)
#pragma unroll
        for (int c = 0; c < CH; ++c)
#pragma unroll
            for (int e = 0; e < 4; ++e) kk[b] = fmaf(k[b][c][e], k[b][c][e], kk[b]);
#pragma unroll
    for (int b = 0; b < N; ++b) kk[b] = over_group(kk[b]);
#pragma unroll
    for (int b = 0; b < N; ++b) {
        const float* row = p.proj + (size_t)(t + b) * p.ldp;
        float* rec = p.records + ((size_t)h * p.tokens + t + b) * REC;
        auto store = [&](int v, int c, const float (&f)[4]) {
            const int d = (c * group + lane) * 4;
            if (d < DS) *reinterpret_cast<float4*>(rec + v * DS + d) = make_float4(f[0], f[1], f[2], f[3]);
        };
        const float inv = 1.0f / sqrtf(kk[b] + p.unit_eps);
        float u[CH][4];
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            float f[4];
            load(row + p.r_col, c, f);
            store(4, c, f);
            load(row + p.v_col, c, f);
            store(5, c, f);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                w[b][c][e] = decay_exp(-p.decay_scale * sigmoid_f(w[b][c][e] + w0[c][e]));
                u[c][e] = k[b][c][e] * inv;
                au[b][c][e] = sigmoid_f(au[b][c][e] + a0[c][e]) * u[c][e];
            }
            store(0, c, w[b][c]);
            store(2, c, au[b][c]);
            store(3, c, k[b][c]);
        }
        // from the token in front backwards: the products with its vectors, then its decay joins u
        float numbers[NUMBERS] = {};
#pragma unroll
        for (int j = b - 1; j >= 0; --j) {
            float along_a = 0.f, along_k = 0.f;
#pragma unroll
            for (int c = 0; c < CH; ++c)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    along_a = fmaf(u[c][e], au[j][c][e], along_a);
                    along_k = fmaf(u[c][e], k[j][c][e], along_k);
                    u[c][e] *= w[j][c][e];
                }
            numbers[j] = over_group(along_a);
            numbers[4 + j] = over_group(along_k);
        }
#pragma unroll
        for (int c = 0; c < CH; ++c) store(1, c, u[c]);
        if (lane < 2) *reinterpret_cast<float4*>(rec + VECS * DS + lane * 4) = lane ? make_float4(numbers[4], numbers[5], numbers[6], numbers[7])
                                                                                       : make_float4(numbers[0], numbers[1], numbers[2], numbers[3]);
    }
}

// a group of p.lanes lanes (a power of two up to 32) per (block of tokens, head)
template <int CH, bool WIDE>
__global__ void __launch_bounds__(128) general_delta_records_kernel(const DeltaParams p, int DS, int num_seqs) {
    const int group = p.lanes, lane = threadIdx.x % group;
    const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / group;
    // neighbouring groups take neighbouring heads of a block: the projection's rows are read in order
    int index = (int)(i / p.heads), t = -1, n = 0;
    for (int s = 0; s < num_seqs; ++s) {
        const int lo = p.seq_starts[s], count = p.seq_starts[s + 1] - lo, blocks = (count + BLOCK - 1) / BLOCK;
        if (index < blocks) {
            t = lo + index * BLOCK;
            n = min(BLOCK, count - index * BLOCK);
            break;
        }
        index -= blocks;
    }
    if (t < 0) return;
    const int h = (int)(i % p.heads);
    const unsigned mask = group == 32 ? 0xffffffffu : ((1u << group) - 1u) << (threadIdx.x % 32 / group * group);
    if (n == BLOCK) make_records<BLOCK, CH, WIDE>(p, DS, t, h, lane, group, mask);
    else
        for (int b = 0; b < n; ++b) make_records<1, CH, WIDE>(p, DS, t + b, h, lane, group, mask);
}

// y = o / rms(o) * gain * sigmoid(g), a warp per (token, head)
template <typename TO>
__device__ __forceinline__ void norm_and_gate(const DeltaParams& p, const float* o, size_t t, int h, int lane) {
    float ss = 0.f;
    for (int d = lane; d < p.dim; d += 32) ss = fmaf(o[d], o[d], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
    const float* g = p.proj + t * p.ldp + p.g_col + h * p.dim;
    TO* out = (TO*)p.y + t * p.ldy + h * p.dim;
    for (int d = lane; d < p.dim; d += 32) out[d] = from_f32<TO>(o[d] * inv * p.gain[h * p.dim + d] * sigmoid_f(g[d]));
}

// behind a recurrence whose blocks held slices of a head: `lanes` lanes per (token, head), four channels a lane and pass (WIDE)
template <typename TO, bool WIDE>
__global__ void __launch_bounds__(256) general_delta_output_kernel(const DeltaParams p) {
    if (!WIDE) {
        const long long i = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
        if (i >= (long long)p.tokens * p.heads) return;
        norm_and_gate<TO>(p, p.o_raw + (size_t)i * p.dim, (size_t)(i / p.heads), (int)(i % p.heads), threadIdx.x & 31);
        return;
    }
    const int group = p.lanes, lane = threadIdx.x % group;
    const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / group;
    const bool live = i < (long long)p.tokens * p.heads;
    const size_t t = live ? (size_t)(i / p.heads) : 0;
    const int at = live ? (int)(i % p.heads) * p.dim : 0;
    const float* o = p.o_raw + t * p.heads * p.dim + at;
    const float* g = p.proj + t * p.ldp + p.g_col + at;
    TO* out = (TO*)p.y + t * p.ldy + at;
    float ss = 0.f;
    for (int d = lane * 4; d < p.dim; d += group * 4) {
        const float4 v = *reinterpret_cast<const float4*>(o + d);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    for (int x = group >> 1; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    if (!live) return;
    const float inv = 1.0f / sqrtf(ss / (float)p.dim + p.eps);
    for (int d = lane * 4; d < p.dim; d += group * 4) {
        const float4 v = *reinterpret_cast<const float4*>(o + d), z = *reinterpret_cast<const float4*>(g + d), w = *reinterpret_cast<const float4*>(p.gain + at + d);
        const float r0 = v.x * inv * w.x * sigmoid_f(z.x), r1 = v.y * inv * w.y * sigmoid_f(z.y), r2 = v.z * inv * w.z * sigmoid_f(z.z),
                    r3 = v.w * inv * w.w * sigmoid_f(z.w);
        if (sizeof(TO) == 2) {
            __nv_bfloat162 lo = __floats2bfloat162_rn(r0, r1), hi = __floats2bfloat162_rn(r2, r3);
            *reinterpret_cast<uint2*>(out + d) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
        } else {
            *reinterpret_cast<float4*>(out + d) = make_float4(r0, r1, r2, r3);
        }
    }
}

// INLINE: the block makes its entry's records itself (entries of up to p.tile tokens)
template <typename TO, int R, int P, int COLS, bool INLINE>
__global__ void __launch_bounds__(INLINE ? 512 : 256, 1) general_delta_kernel(const DeltaParams p) {
    extern __shared__ __align__(128) float smem[];
    __shared__ __align__(8) uint64_t full[STAGES];
    __shared__ int abort_flag;
    constexpr int DS = R * P, REC = VECS * DS + NUMBERS, NSTAGES = INLINE ? 1 : STAGES;
    const int dim = p.dim, cols = p.cols, TILE = p.tile;
    float* s_o = smem + NSTAGES * TILE * REC;       // [2][TILE][cols]
    const int head = blockIdx.x, seq = blockIdx.y, j0 = blockIdx.z * cols;
    const int start = p.seq_starts[seq], count = p.seq_starts[seq + 1] - start;
    const int jl = threadIdx.x / P * COLS, part = threadIdx.x % P;
    const int width = min(cols, dim - j0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int tiles = (count + TILE - 1) / TILE;
    const float* source = p.records + ((size_t)head * p.tokens + start) * REC;
    auto fill = [&](int ti) {                       // one thread
        const uint32_t bytes = (uint32_t)(min(TILE, count - ti * TILE) * REC * 4);
        mbar_expect_tx(&full[ti % STAGES], bytes);
        bulk_load(smem + (ti % STAGES) * TILE * REC, source + (size_t)ti * TILE * REC, bytes, &full[ti % STAGES]);
    };
    if (!INLINE && threadIdx.x == 0) {
        for (int s = 0; s < STAGES; ++s) mbar_init(&full[s], 1);
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
        for (int ti = 0; ti < min(STAGES - 1, tiles); ++ti) fill(ti);
    }
    float* S = p.state + (size_t)p.seq_slots[seq] * p.slot_floats + p.state_offset + ((size_t)head * dim + j0 + jl) * dim;
    uint64_t s[COLS][R / 2];
#pragma unroll
    for (int c = 0; c < COLS; ++c)
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const int row = (i * P + part) * 4;
            const float* at = S + (size_t)c * dim + row;
            const bool mine = jl + c < width;
            float v[4];
            if (dim % 4 == 0) {
                const float4 f = mine && row < dim ? *reinterpret_cast<const float4*>(at) : make_float4(0.f, 0.f, 0.f, 0.f);
                v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) v[e] = mine && row + e < dim ? at[e] : 0.f;
            }
            s[c][2 * i] = pair_of(v[0], v[1]);
            s[c][2 * i + 1] = pair_of(v[2], v[3]);
        }
    if (INLINE && count > TILE) {                   // the host hands no such step here
        if (threadIdx.x == 0) atomicOr(p.status, EG_STATUS_BAD_SLOT);
        return;
    }
    if (INLINE) {
        float* inner = s_o + 2 * TILE * cols;       // [TILE][rank]
        for (int i = threadIdx.x; i < count * p.rank; i += blockDim.x)
            inner[i] = tanhf(p.proj[(size_t)(start + i / p.rank) * p.ldp + p.inner_col + i % p.rank]);
        __syncthreads();
        // a warp per (token, 32 channels); every warp sums the whole key's squares
        const int blocks = (DS + 31) / 32;
        for (int it = warp; it < count * blocks; it += warps) {
            const int t = it / blocks, d = it % blocks * 32 + lane, at = head * dim;
            const float* row = p.proj + (size_t)(start + t) * p.ldp;
            float kk = 0.f;
            for (int c = lane; c < dim; c += 32) {
                const float k = row[p.k_col + at + c];
                kk = fmaf(k, k, kk);
            }
            const float inv = 1.0f / sqrtf(warp_sum(kk) + p.unit_eps);
            float* rec = smem + (size_t)t * REC;
            if (d < dim) {
                const TO* w2 = (const TO*)p.w2 + (size_t)(at + d) * p.ld2;
                const float* in = inner + t * p.rank;
                float x0 = 0.f, x1 = 0.f;
                int r = 0;
                if (sizeof(TO) == 2) {              // rows of w2 start on 16-byte boundaries (ld2 a multiple of 8)
                    for (; r + 8 <= p.rank; r += 8) {
                        const uint4 q = *reinterpret_cast<const uint4*>(w2 + r);
                        const uint32_t m[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            x0 = fmaf(__uint_as_float(m[e] << 16), in[r + 2 * e], x0);
                            x1 = fmaf(__uint_as_float(m[e] & 0xffff0000u), in[r + 2 * e + 1], x1);
                        }
                    }
                }
                for (; r < p.rank; ++r) x0 = fmaf(to_f32<TO>(w2[r]), in[r], x0);
                put_channel(p, row, at, d, x0 + x1, inv, rec, DS);
            } else if (d < DS) {
                for (int q = 0; q < VECS; ++q) rec[q * DS + d] = 0.f;
            }
        }
    }
    __syncthreads();
    auto write_out = [&](int ti) {                  // the outputs of tile ti, complete in s_o
        const int t0 = ti * TILE, n = min(TILE, count - t0);
        const float* o = s_o + (ti & 1) * TILE * cols;
        if (p.o_raw) {
            for (int i = threadIdx.x; i < n * width; i += blockDim.x) {
                const int t = i / width, d = i % width;
                p.o_raw[(size_t)(start + t0 + t) * ((size_t)p.heads * dim) + head * dim + j0 + d] = o[t * cols + d];
            }
        } else {
            for (int t = warp; t < n; t += warps) norm_and_gate<TO>(p, o + t * cols, (size_t)(start + t0 + t), head, lane);
        }
    };
    bool ok = true;
    int done = 0;
    for (int ti = 0; ti < tiles; ++ti) {
        if (!INLINE) {
            ok = mbar_wait_bounded(&full[ti % STAGES], (ti / STAGES) & 1, &abort_flag, p.status, WAIT_LIMIT);
            ok = __syncthreads_and(ok);             // every warp is done with the tile before: its stage may be filled again, its outputs read
            if (!ok) break;
            if (threadIdx.x == 0 && ti + STAGES - 1 < tiles) fill(ti + STAGES - 1);
        } else if (ti > 0) {
            break;                                  // entries that make their records here are one tile
        }
        if (ti > 0) write_out(ti - 1);
        const int n = min(TILE, count - ti * TILE);
        const float* base = smem + (INLINE ? 0 : ti % STAGES) * TILE * REC;
        float* out = s_o + (ti & 1) * TILE * cols + jl;
        // one token: the rows move on; o: this lane's share of the columns' outputs
        auto step = [&](int t, float (&o)[COLS]) {
            const float* rec = base + t * REC + part * 4;
            auto piece = [&](int v, int i) { return *reinterpret_cast<const ulonglong2*>(rec + v * DS + i * P * 4); };
            // what the old state holds along the unit key
            uint64_t held[COLS][2] = {};
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const ulonglong2 u = piece(1, i);
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    held[c][0] = fma2(s[c][2 * i], u.x, held[c][0]);
                    held[c][1] = fma2(s[c][2 * i + 1], u.y, held[c][1]);
                }
            }
            float off[COLS];
            uint64_t value2[COLS];
#pragma unroll
            for (int c = 0; c < COLS; ++c) {
                off[c] = sum_of(held[c][0]) + sum_of(held[c][1]);
                const float value = base[t * REC + 5 * DS + j0 + jl + c];
                value2[c] = pair_of(value, value);
            }
            // meanwhile the rows decay and take in the value
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const ulonglong2 w = piece(0, i), k = piece(3, i);
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    s[c][2 * i] = fma2(w.x, s[c][2 * i], mul2(k.x, value2[c]));
                    s[c][2 * i + 1] = fma2(w.y, s[c][2 * i + 1], mul2(k.y, value2[c]));
                }
            }
#pragma unroll
            for (int o = 1; o < P; o <<= 1)
#pragma unroll
                for (int c = 0; c < COLS; ++c) off[c] += __shfl_xor_sync(0xffffffffu, off[c], o);
            uint64_t off2[COLS], read[COLS][2] = {};
#pragma unroll
            for (int c = 0; c < COLS; ++c) off2[c] = pair_of(-off[c], -off[c]);
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const ulonglong2 a = piece(2, i), q = piece(4, i);
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    s[c][2 * i] = fma2(a.x, off2[c], s[c][2 * i]);
                    s[c][2 * i + 1] = fma2(a.y, off2[c], s[c][2 * i + 1]);
                    read[c][0] = fma2(s[c][2 * i], q.x, read[c][0]);
                    read[c][1] = fma2(s[c][2 * i + 1], q.y, read[c][1]);
                }
            }
#pragma unroll
            for (int c = 0; c < COLS; ++c) o[c] = sum_of(read[c][0]) + sum_of(read[c][1]);
        };
        int t = 0;
        for (; !INLINE && t + BLOCK <= n; t += BLOCK) {
            const float* rec = base + t * REC + part * 4;
            auto piece = [&](int b, int v, int i) { return *reinterpret_cast<const ulonglong2*>(rec + b * REC + v * DS + i * P * 4); };
            float held[BLOCK][COLS], value[BLOCK][COLS];
#pragma unroll
            for (int b = 0; b < BLOCK; ++b) {
                uint64_t sum[COLS][2] = {};
#pragma unroll
                for (int i = 0; i < R / 4; ++i) {
                    const ulonglong2 u = piece(b, 1, i);
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        sum[c][0] = fma2(s[c][2 * i], u.x, sum[c][0]);
                        sum[c][1] = fma2(s[c][2 * i + 1], u.y, sum[c][1]);
                    }
                }
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    held[b][c] = sum_of(sum[c][0]) + sum_of(sum[c][1]);
                    value[b][c] = base[(t + b) * REC + 5 * DS + j0 + jl + c];
                }
            }
#pragma unroll
            for (int x = 1; x < P; x <<= 1)
#pragma unroll
                for (int b = 0; b < BLOCK; ++b)
#pragma unroll
                    for (int c = 0; c < COLS; ++c) held[b][c] += __shfl_xor_sync(0xffffffffu, held[b][c], x);
#pragma unroll
            for (int b = 1; b < BLOCK; ++b) {
                const float4 fa = *reinterpret_cast<const float4*>(base + (t + b) * REC + VECS * DS), fk = *reinterpret_cast<const float4*>(base + (t + b) * REC + VECS * DS + 4);
                const float A[3] = {fa.x, fa.y, fa.z}, K[3] = {fk.x, fk.y, fk.z};
#pragma unroll
                for (int c = 0; c < COLS; ++c)
#pragma unroll
                    for (int j = 0; j < b; ++j) held[b][c] = fmaf(-A[j], held[j][c], fmaf(K[j], value[j][c], held[b][c]));
            }
            float o[BLOCK * COLS];
#pragma unroll
            for (int b = 0; b < BLOCK; ++b) {
                uint64_t off2[COLS], value2[COLS], read[COLS][2] = {};
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    off2[c] = pair_of(-held[b][c], -held[b][c]);
                    value2[c] = pair_of(value[b][c], value[b][c]);
                }
#pragma unroll
                for (int i = 0; i < R / 4; ++i) {
                    const ulonglong2 w = piece(b, 0, i), a = piece(b, 2, i), k = piece(b, 3, i), q = piece(b, 4, i);
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        s[c][2 * i] = fma2(w.x, s[c][2 * i], fma2(a.x, off2[c], mul2(k.x, value2[c])));
                        s[c][2 * i + 1] = fma2(w.y, s[c][2 * i + 1], fma2(a.y, off2[c], mul2(k.y, value2[c])));
                        read[c][0] = fma2(s[c][2 * i], q.x, read[c][0]);
                        read[c][1] = fma2(s[c][2 * i + 1], q.y, read[c][1]);
                    }
                }
#pragma unroll
                for (int c = 0; c < COLS; ++c) o[b * COLS + c] = sum_of(read[c][0]) + sum_of(read[c][1]);
            }
            // the block's sums over the lanes: while a lane has several it gives half of them away for the other half of a neighbour's
            int which = 0;
#pragma unroll
            for (int x = 1, have = BLOCK * COLS; x < P; x <<= 1) {
                if (have > 1) {
                    have >>= 1;
                    const bool upper = part & x;
#pragma unroll
                    for (int i = 0; i < have; ++i) {
                        const float give = upper ? o[i] : o[have + i], keep = upper ? o[have + i] : o[i];
                        o[i] = keep + __shfl_xor_sync(0xffffffffu, give, x);
                    }
                    which += upper ? have : 0;
                } else {
                    o[0] += __shfl_xor_sync(0xffffffffu, o[0], x);
                }
            }
            static_assert(BLOCK * COLS <= P, "a lane ends with one sum");
            if (part < BLOCK * COLS && jl + which % COLS < width) out[(t + which / COLS) * cols + which % COLS] = o[0];
        }
        for (; t < n; ++t) {
            float o[COLS];
            step(t, o);
#pragma unroll
            for (int c = 0; c < COLS; ++c) {
#pragma unroll
                for (int x = 1; x < P; x <<= 1) o[c] += __shfl_xor_sync(0xffffffffu, o[c], x);
                if (part == 0 && jl + c < width) out[t * cols + c] = o[c];
            }
        }
        done = ti + 1;
    }
    if (!INLINE && !ok) {                           // every copy has to land before the block gives up its shared memory
        if (threadIdx.x == 0)
            for (int ti = done; ti < min(done + STAGES - 1, tiles); ++ti)
                for (unsigned i = 0; i < WAIT_LIMIT && !mbar_try_wait(&full[ti % STAGES], (ti / STAGES) & 1); ++i) {}
        return;
    }
    __syncthreads();
    if (tiles > 0) write_out(INLINE ? 0 : tiles - 1);
#pragma unroll
    for (int c = 0; c < COLS; ++c)
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const int row = (i * P + part) * 4;
            float* at = S + (size_t)c * dim + row;
            float v[4];
            asm("mov.b64 {%0, %1}, %2;" : "=f"(v[0]), "=f"(v[1]) : "l"(s[c][2 * i]));
            asm("mov.b64 {%0, %1}, %2;" : "=f"(v[2]), "=f"(v[3]) : "l"(s[c][2 * i + 1]));
            if (jl + c >= width) continue;
            if (dim % 4 == 0) {
                if (row < dim) *reinterpret_cast<float4*>(at) = make_float4(v[0], v[1], v[2], v[3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (row + e < dim) at[e] = v[e];
            }
        }
}

int power_of_two_lanes(int items) {                 // the least power of two that is at least `items`, up to 32
    int n = 1;
    while (n < items && n < 32) n <<= 1;
    return n;
}

template <typename TO, int R, int P, int COLS, bool INLINE>
int launch_general_delta(cudaStream_t stream, DeltaParams p, int slices, int num_seqs, bool float4_rows) {
    constexpr int DS = R * P, REC = VECS * DS + NUMBERS, per_warp = 32 / P * COLS;
    const int most = (INLINE ? 512 : 256) / P * COLS / per_warp * per_warp;
    if (!p.o_raw) slices = 1;
    int cols = (p.dim + slices - 1) / slices;
    cols = std::min((cols + per_warp - 1) / per_warp * per_warp, most);
    slices = (p.dim + cols - 1) / cols;
    if (slices > 1 && !p.o_raw) return (int)cudaErrorInvalidValue;
    if (slices == 1) p.o_raw = nullptr;
    p.cols = cols;
    p.tile = DS <= 128 ? 16 : 8;
    const size_t smem = ((size_t)(INLINE ? 1 : STAGES) * p.tile * REC + (size_t)2 * p.tile * cols + (INLINE ? (size_t)p.tile * p.rank : 0)) * sizeof(float);
    if (smem > 220 * 1024) return (int)cudaErrorInvalidValue;
    auto kernel = general_delta_kernel<TO, R, P, COLS, INLINE>;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    const bool wide = float4_rows && p.dim % 4 == 0;
    if (!INLINE) {
        constexpr int CH = DS <= 128 ? 1 : 2;
        p.lanes = DS / 4 / CH;
        const unsigned blocks = (unsigned)(((long long)(p.tokens / BLOCK + num_seqs) * p.heads * p.lanes + 127) / 128);
        if (wide) general_delta_records_kernel<CH, true><<<blocks, 128, 0, stream>>>(p, DS, num_seqs);
        else general_delta_records_kernel<CH, false><<<blocks, 128, 0, stream>>>(p, DS, num_seqs);
    }
    kernel<<<dim3(p.heads, num_seqs, slices), cols / COLS * P, smem, stream>>>(p);
    if (p.o_raw) {
        if (wide) {
            p.lanes = power_of_two_lanes((p.dim + 3) / 4);
            general_delta_output_kernel<TO, true><<<(unsigned)(((long long)p.tokens * p.heads * p.lanes + 255) / 256), 256, 0, stream>>>(p);
        } else {
            general_delta_output_kernel<TO, false><<<(unsigned)(((long long)p.tokens * p.heads + 7) / 8), 256, 0, stream>>>(p);
        }
    }
    return eg_launch_status();
}

template <typename TO, bool INLINE>
int dispatch_general_delta(cudaStream_t stream, const DeltaParams& p, int slices, int num_seqs, bool wide) {
    if (p.dim <= 16) return launch_general_delta<TO, 4, 4, 1, INLINE>(stream, p, slices, num_seqs, wide);
    if (p.dim <= 32) return launch_general_delta<TO, 4, 8, 2, INLINE>(stream, p, slices, num_seqs, wide);
    if (p.dim <= 64) {
        // (prompts: half the rows a lane of what steps of short entries have, whose blocks hold whole heads)
        if (INLINE) return launch_general_delta<TO, 8, 8, 2, INLINE>(stream, p, slices, num_seqs, wide);
        return launch_general_delta<TO, 4, 16, 2, INLINE>(stream, p, slices, num_seqs, wide);
    }
    if (p.dim <= 128) return launch_general_delta<TO, 8, 16, 2, INLINE>(stream, p, slices, num_seqs, wide);
    return launch_general_delta<TO, 8, 32, 2, INLINE>(stream, p, slices, num_seqs, wide);
}

template <typename T>
__global__ void tanh_columns_kernel(const float* __restrict__ src, long long lds, T* __restrict__ dst, long long ldd, int rows, int cols, int padded) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)rows * padded) return;
    const int t = (int)(i / padded), c = (int)(i % padded);
    dst[(size_t)t * ldd + c] = from_f32<T>(c < cols ? tanhf(src[(size_t)t * lds + c]) : 0.f);
}
}  // namespace

// float32 values of a record of a head of `dim` channels (scratch: heads * tokens of them)
EG_API int eg_general_delta_record(int dim) { return VECS * (dim <= 16 ? 16 : dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256) + NUMBERS; }

// up to how many tokens an entry may have, and how large the inner size may be, for eg_general_delta with x null
EG_API int eg_general_delta_inline_takes(int entry_tokens, int rank) { return entry_tokens <= 8 && rank <= 512; }

// proj float32 [tokens, ldp] with r, k, v, g (the output gate) and a (the removal rates' logits, bias a0 still to be added), heads x dim
// each, and the inner values of the decays' map (before tanh, `rank`) at their columns; x float32 [tokens, ldx]: the decays' logits
// (w0 still to be added), or null in steps whose entries eg_general_delta_inline_takes: then w2 [heads * dim, ld2] in y_dtype (ld2 a
// multiple of 8).  a0, w0, gain float32 [heads * dim].  records: scratch, not read with x null.  state: the requests' slots; S of
// a request lies state_offset floats into its slot.  y [tokens, ldy] in y_dtype.  slices > 1 (with o_raw float32 [tokens, heads * dim]): a
// head's columns are dealt to that many blocks, and the outputs are normed by a kernel behind.  dim up to 256.
EG_API int eg_general_delta(cudaStream_t stream, const float* proj, long long ldp, int r_col, int k_col, int v_col, int g_col, int a_col, int inner_col,
                            const float* x, long long ldx, const void* w2, int ld2, int rank, const float* w0, const float* a0, const float* gain,
                            float* records, float* state, long long slot_floats, long long state_offset, const int* seq_starts, const int* seq_slots,
                            void* y, int y_dtype, long long ldy, float* o_raw, int slices, int tokens, int num_seqs, int heads, int dim, float unit_eps,
                            float eps, float decay_scale, int* status) {
    if (num_seqs <= 0 || tokens <= 0) return 0;
    if (heads <= 0 || dim <= 0 || dim > 256 || slices < 1 || (x && !records) || (!x && (!w2 || ld2 % 8 || (uintptr_t)w2 % 16))) return (int)cudaErrorInvalidValue;
    if (slot_floats % 4 || state_offset % 4 || (uintptr_t)state % 16 || (uintptr_t)records % 16) {
        if (dim % 4 == 0 || (uintptr_t)records % 16) return (int)cudaErrorInvalidValue;     // heads of a multiple of four rows are read in 16-byte pieces
    }
    DeltaParams p{};
    p.proj = proj;
    p.ldp = ldp;
    p.r_col = r_col;
    p.k_col = k_col;
    p.v_col = v_col;
    p.g_col = g_col;
    p.a_col = a_col;
    p.inner_col = inner_col;
    p.x = x;
    p.ldx = ldx;
    p.w2 = w2;
    p.ld2 = ld2;
    p.rank = rank;
    p.w0 = w0;
    p.a0 = a0;
    p.gain = gain;
    p.records = records;
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
    p.status = status;
    auto aligned = [](const void* q) { return (uintptr_t)q % 16 == 0; };
    const bool wide = ldp % 4 == 0 && ldx % 4 == 0 && r_col % 4 == 0 && k_col % 4 == 0 && v_col % 4 == 0 && g_col % 4 == 0 && a_col % 4 == 0 && aligned(proj) &&
                      aligned(x) && aligned(w0) && aligned(a0) && aligned(gain) && aligned(o_raw) && aligned(y) && ldy % 4 == 0;
    if (y_dtype == EG_BF16)
        return x ? dispatch_general_delta<bf16, false>(stream, p, slices, num_seqs, wide) : dispatch_general_delta<bf16, true>(stream, p, slices, num_seqs, wide);
    return x ? dispatch_general_delta<float, false>(stream, p, slices, num_seqs, wide) : dispatch_general_delta<float, true>(stream, p, slices, num_seqs, wide);
}

// dst [rows, ldd] in dst_dtype: column c < cols holds tanh(src[., c]), columns up to `padded` hold zeros
EG_API int eg_tanh_columns(cudaStream_t stream, const float* src, long long lds, void* dst, int dst_dtype, long long ldd, int rows, int cols, int padded) {
    if (rows <= 0 || padded <= 0) return 0;
    const unsigned blocks = (unsigned)(((long long)rows * padded + 255) / 256);
    if (dst_dtype == EG_BF16) tanh_columns_kernel<bf16><<<blocks, 256, 0, stream>>>(src, lds, (bf16*)dst, ldd, rows, cols, padded);
    else tanh_columns_kernel<float><<<blocks, 256, 0, stream>>>(src, lds, (float*)dst, ldd, rows, cols, padded);
    return eg_launch_status();
}
