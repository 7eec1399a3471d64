// Attention over cached latent rows on the warp-level tensor cores (bfloat16): the heads of a token are the rows of the
// product.
//
// All heads of a token attend the same cached rows (rank + rot values each, see attention_latent.cu), so 16 heads of one
// token against a tile of 64 keys is a 16 x 64 x (rank + rot) product, and the weighted sum a 16 x rank x 64 one: shapes
// that mma.sync m16n8k16 takes as they are, for a prompt's tokens and for single decoded tokens alike.  A CTA of four
// warps takes (token, group of 16 heads, part of the keys):
//   the queries qa [16, D] and, tile by tile, 64 cached rows [64, D] go to shared memory: one bulk copy (cp.async.bulk,
//     counted on an mbarrier) per cached row, issued by the lanes of the first warp, rows beyond the token's position
//     zeroed; the cached rows are read once for scores and values; the wait on the mbarrier is bounded;
//   scores: warp w computes the tile's keys 16 w .. 16 w + 15 for all 16 heads; row maxima and sums meet in shared memory;
//   the weights go to shared memory as bfloat16 and every warp adds its share of the value columns (columns 16 (w + 4 i)..)
//     from the same key tile, read transposed by ldmatrix;
//   at the end the sink joins the denominator (one part) or the part's (o, m, l) goes to scratch and a second kernel
//     merges the parts and the sink.
// That form reads every key tile once per token: it is for single tokens and entries of a few.  Prompt portions go to a second kernel
// (attention_latent_tiles_kernel), whose CTA takes several consecutive tokens of a request, 64 rows of (token, head) in all, against
// the same key tile; see there.
// Scores, maxima, sums and the accumulators are float32.  Takes D = rank + rot a multiple of 8, rank a multiple of 8 up
// to 512; anything else: cudaErrorInvalidValue, and the caller uses the generic kernel.
#include "mbarrier.cuh"
#include "mma_utils.cuh"

namespace {
constexpr int KT = 64, WARPS = 4, PAIRS = 8;        // keys per tile; warps; pairs of 8-column value tiles per warp

__device__ __forceinline__ float quad_max(float v) {
    v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
    return fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
}
__device__ __forceinline__ float quad_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    return v + __shfl_xor_sync(0xffffffffu, v, 2);
}

__global__ void __launch_bounds__(WARPS * 32) attention_latent_mma_kernel(const bf16* __restrict__ qa, const bf16* __restrict__ cache,
                                                                          const int* __restrict__ block_table, int table_stride,
                                                                          const int* __restrict__ token_seq, const int* __restrict__ positions,
                                                                          const int* __restrict__ token_list, const float* __restrict__ sink,
                                                                          bf16* __restrict__ out, float* __restrict__ part_o, float* __restrict__ part_ml, int heads, int rank, int rot, int page_size,
                                                                          long long page_stride, int num_pages, int splits, int* __restrict__ status) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ __align__(8) uint64_t bar;
    __shared__ int abort_flag;
    const int D = rank + rot, D16 = (D + 15) / 16 * 16, DS = D16 + 8;           // row stride in elements: 16 bytes past a multiple of 32
    bf16* Qs = reinterpret_cast<bf16*>(smem);
    bf16* Ks = Qs + 16 * DS;
    bf16* Ps = Ks + KT * DS;
    float* red_max = reinterpret_cast<float*>(Ps + 16 * (KT + 8));
    float* red_sum = red_max + WARPS * 16;
    const int t = token_list ? token_list[blockIdx.x] : blockIdx.x, head0 = blockIdx.y * 16, part = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int last = positions[t];
    const int tiles = last / KT + 1, per = (tiles + splits - 1) / splits;
    const int tile0 = part * per, tile1 = min(tiles, tile0 + per);
    const int* table = block_table + (size_t)token_seq[t] * table_stride;

    // queries (zero rows for heads past the last one, zero columns past D), and the key tile's padding columns
    for (int i = threadIdx.x; i < 16 * (D / 8); i += blockDim.x) {          // 16 bytes a load
        const int h = i / (D / 8), c = i % (D / 8);
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (head0 + h < heads) v = *reinterpret_cast<const uint4*>(qa + ((size_t)t * heads + head0 + h) * D + c * 8);
        *reinterpret_cast<uint4*>(Qs + h * DS + c * 8) = v;
    }
    for (int i = threadIdx.x; i < 16 * (DS - D); i += blockDim.x) Qs[(i / (DS - D)) * DS + D + i % (DS - D)] = __float2bfloat16(0.f);
    for (int i = threadIdx.x; i < KT * (DS - D); i += blockDim.x) Ks[(i / (DS - D)) * DS + D + i % (DS - D)] = __float2bfloat16(0.f);

    float o[PAIRS][2][4];
#pragma unroll
    for (int i = 0; i < PAIRS; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int k = 0; k < 4; ++k) o[i][j][k] = 0.f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};      // rows lane / 4 and lane / 4 + 8
    const int chunks = D / 8;                                               // 16-byte pieces of a cached row
    const uint32_t row_bytes = (uint32_t)D * 2;
    if (threadIdx.x == 0) {
        mbar_init(&bar, 1);
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    __syncthreads();

    for (int tile = tile0; tile < tile1; ++tile) {
        const int j0 = tile * KT;
        const int valid_rows = min(KT, last - j0 + 1);
        if (warp == 0) {
            // the buffer was last touched by ldmatrix and plain stores: order them before the copies that overwrite it
            asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
            if (lane == 0) mbar_expect_tx(&bar, (uint32_t)valid_rows * row_bytes);
            __syncwarp();
            for (int r = lane; r < valid_rows; r += 32) {
                const int j = j0 + r, page = table[j / page_size];
                if (page < 0 || page >= num_pages) {             // a complaint, and the row's bytes from a page that exists
                    atomicOr(status, EG_STATUS_BAD_PAGE);
                }
                const int safe = (page < 0 || page >= num_pages) ? 0 : page;
                const bf16* src = cache + (size_t)safe * page_stride + (size_t)(j % page_size) * D;
                asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n" ::"r"(smem_addr(Ks + r * DS)),
                             "l"(src), "r"(row_bytes), "r"(smem_addr(&bar))
                             : "memory");
            }
        } else {
            for (int i = threadIdx.x - 32; i < (KT - valid_rows) * chunks; i += blockDim.x - 32)      // rows past the token's position: zeros
                *reinterpret_cast<uint4*>(Ks + (valid_rows + i / chunks) * DS + (i % chunks) * 8) = make_uint4(0u, 0u, 0u, 0u);
        }
        if (!mbar_wait_bounded(&bar, (uint32_t)((tile - tile0) & 1), &abort_flag, status, 1u << 24)) break;
        __syncthreads();

        // scores of this warp's 16 keys for the 16 heads
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        const bf16* a_at = Qs + (lane % 16) * DS + (lane / 16) * 8;
        const bf16* b_at = Ks + (warp * 16 + (lane % 8) + (lane / 16) * 8) * DS + ((lane / 8) % 2) * 8;
        for (int k0 = 0; k0 < D16; k0 += 16) {
            uint32_t a[4], b[4];
            ldmatrix_x4(a, a_at + k0);
            ldmatrix_x4(b, b_at + k0);
            mma_bf16_16816(s[0], a, b[0], b[1]);
            mma_bf16_16816(s[1], a, b[2], b[3]);
        }
        float tile_max[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int j = j0 + warp * 16 + i * 8 + 2 * (lane % 4) + (e & 1);
                if (j > last) s[i][e] = -INFINITY;
                tile_max[e >> 1] = fmaxf(tile_max[e >> 1], s[i][e]);
            }
        tile_max[0] = quad_max(tile_max[0]);
        tile_max[1] = quad_max(tile_max[1]);
        if (lane % 4 == 0) {
            red_max[warp * 16 + lane / 4] = tile_max[0];
            red_max[warp * 16 + lane / 4 + 8] = tile_max[1];
        }
        __syncthreads();
        float m_new[2], alpha[2], row_sum[2] = {0.f, 0.f};
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float m = m_run[r];
#pragma unroll
            for (int w = 0; w < WARPS; ++w) m = fmaxf(m, red_max[w * 16 + lane / 4 + 8 * r]);
            m_new[r] = m;
            alpha[r] = m == -INFINITY ? 1.f : expf(m_run[r] - m);          // exp(-inf) = 0 at the first keys
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = e >> 1;
                const float p = m_new[r] == -INFINITY ? 0.f : expf(s[i][e] - m_new[r]);
                s[i][e] = p;
                row_sum[r] += p;
            }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int col = warp * 16 + i * 8 + 2 * (lane % 4);
            *reinterpret_cast<uint32_t*>(Ps + (lane / 4) * (KT + 8) + col) = pack_bf16(s[i][0], s[i][1]);
            *reinterpret_cast<uint32_t*>(Ps + (lane / 4 + 8) * (KT + 8) + col) = pack_bf16(s[i][2], s[i][3]);
        }
        row_sum[0] = quad_sum(row_sum[0]);
        row_sum[1] = quad_sum(row_sum[1]);
        if (lane % 4 == 0) {
            red_sum[warp * 16 + lane / 4] = row_sum[0];
            red_sum[warp * 16 + lane / 4 + 8] = row_sum[1];
        }
        __syncthreads();
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float sum = 0.f;
#pragma unroll
            for (int w = 0; w < WARPS; ++w) sum += red_sum[w * 16 + lane / 4 + 8 * r];
            l_run[r] = l_run[r] * alpha[r] + sum;
            m_run[r] = m_new[r];
        }
        // weighted sums: this warp's value columns 16 (warp + 4 i) .. + 15 over the tile's 64 keys
#pragma unroll
        for (int i = 0; i < PAIRS; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                o[i][j][0] *= alpha[0];
                o[i][j][1] *= alpha[0];
                o[i][j][2] *= alpha[1];
                o[i][j][3] *= alpha[1];
            }
        const bf16* p_at = Ps + (lane % 16) * (KT + 8) + (lane / 16) * 8;
        const bf16* v_at = Ks + ((lane % 8) + ((lane / 8) % 2) * 8) * DS + (lane / 16) * 8;
#pragma unroll
        for (int kk = 0; kk < KT / 16; ++kk) {
            uint32_t a[4];
            ldmatrix_x4(a, p_at + kk * 16);
#pragma unroll
            for (int i = 0; i < PAIRS; ++i) {
                const int col = 16 * (warp + WARPS * i);
                if (col < rank) {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, v_at + (size_t)kk * 16 * DS + col);
                    mma_bf16_16816(o[i][0], a, b[0], b[1]);
                    mma_bf16_16816(o[i][1], a, b[2], b[3]);
                }
            }
        }
        __syncthreads();                                                    // the next tile overwrites the keys and the weights
    }

    if (abort_flag) return;                                                 // a wait gave up: the status word says so, nothing is written
    // a thread holds, per pair of column tiles, rows lane / 4 (values 0, 1) and lane / 4 + 8 (values 2, 3), columns 2 (lane % 4) + {0, 1}
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int head = head0 + lane / 4 + 8 * r;
        if (head >= heads) continue;
        const size_t row = (size_t)t * heads + head, part_row = (size_t)blockIdx.x * heads + head;
        float scale;
        if (splits == 1) {
            const float sk = sink ? sink[head] : -INFINITY;
            const float top = fmaxf(m_run[r], sk);
            const float f = m_run[r] == -INFINITY ? 0.f : expf(m_run[r] - top);
            const float denom = l_run[r] * f + (sink ? expf(sk - top) : 0.f);
            scale = f / denom;
        } else {
            scale = 1.f;
            if (lane % 4 == 0) {
                part_ml[(part_row * splits + part) * 2] = m_run[r];
                part_ml[(part_row * splits + part) * 2 + 1] = l_run[r];
            }
        }
#pragma unroll
        for (int i = 0; i < PAIRS; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int col = 16 * (warp + WARPS * i) + 8 * j + 2 * (lane % 4);
                if (col >= rank) continue;
                const float v0 = o[i][j][2 * r] * scale, v1 = o[i][j][2 * r + 1] * scale;
                if (splits == 1) *reinterpret_cast<uint32_t*>(out + row * rank + col) = pack_bf16(v0, v1);
                else *reinterpret_cast<float2*>(part_o + (part_row * splits + part) * rank + col) = make_float2(v0, v1);
            }
    }
}

// one block per (token, head): the parts' maxima, sums and weighted sums and the sink become the output row.  The parts'
// factors are worked out once, side by side (a thread per part), before the row is summed, four columns a thread with several parts'
// loads in flight.  The parts' rows are numbered by a token's place: with `tiles` its place in its tile (tile_stride places a tile), else
// in token_list, or the token itself.
__global__ void __launch_bounds__(128) attention_latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                                     const int* __restrict__ token_list, const int* __restrict__ tiles,
                                                                     int tile_stride, const float* __restrict__ sink, bf16* __restrict__ out, int heads, int rank,
                                                                     int splits) {
    __shared__ float factor[64];
    __shared__ float inv_denom;
    const int place = blockIdx.x / heads, head = blockIdx.x % heads;
    int t = token_list ? token_list[place] : place;
    if (tiles) {
        const int* tile = tiles + place / tile_stride * 3;
        if (place % tile_stride >= tile[2]) return;
        t = tile[1] + place % tile_stride;
    }
    const size_t row = (size_t)place * heads + head, out_row = (size_t)t * heads + head;
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        float m[2], l[2];
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            const int s = lane + 32 * q;
            m[q] = s < splits ? part_ml[(row * splits + s) * 2] : -INFINITY;
            l[q] = s < splits ? part_ml[(row * splits + s) * 2 + 1] : 0.f;
        }
        const float sk = sink ? sink[head] : -INFINITY;
        const float top = fmaxf(sk, warp_max(fmaxf(m[0], m[1])));
        float sum = 0.f;
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            const float f = m[q] == -INFINITY ? 0.f : expf(m[q] - top);
            factor[lane + 32 * q] = f;
            sum += l[q] * f;
        }
        sum = warp_sum(sum) + (sink ? expf(sk - top) : 0.f);
        if (lane == 0) inv_denom = 1.0f / sum;
    }
    const int columns = rank / 4;                                           // rank is a multiple of eight
    const float4* src = reinterpret_cast<const float4*>(part_o + row * splits * rank);
    for (int d0 = 0; d0 < columns; d0 += blockDim.x) {
        const int d = d0 + threadIdx.x;
        const bool mine = d < columns;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f), next[8];
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (mine && i < splits) next[i] = __ldcg(src + (size_t)i * columns + d);
        if (d0 == 0) __syncthreads();
        for (int s0 = 0; s0 < splits; s0 += 8) {
            float4 here[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) here[i] = next[i];
#pragma unroll
            for (int i = 0; i < 8; ++i)
                if (mine && s0 + 8 + i < splits) next[i] = __ldcg(src + (size_t)(s0 + 8 + i) * columns + d);
#pragma unroll
            for (int i = 0; i < 8; ++i)
                if (mine && s0 + i < splits) {
                    const float f = factor[s0 + i];
                    v.x = fmaf(here[i].x, f, v.x);
                    v.y = fmaf(here[i].y, f, v.y);
                    v.z = fmaf(here[i].z, f, v.z);
                    v.w = fmaf(here[i].w, f, v.w);
                }
        }
        if (mine)
            *reinterpret_cast<uint2*>(out + out_row * rank + 4 * d) = make_uint2(pack_bf16(v.x * inv_denom, v.y * inv_denom), pack_bf16(v.z * inv_denom, v.w * inv_denom));
    }
}

// ---- prompt portions ------------------------------------------------------------------------------------------------------------
// A CTA of eight warps takes `per_cta` consecutive tokens of a listed tile times a group of `group` heads, row = token * group + head,
// at most 64 rows, against key tiles of 64 (a part of them, where a step has few CTAs):
//   the queries [64, D] stay in shared memory; the cached rows come in halves of a tile (32 rows, one bulk copy a row, a lane of the
//     first warp each) into a ring of three, so that while a tile is worked on half of the next one is on its way, and the other half
//     starts when the first half of this one has been used up;
//   scores: warp (rows 32 (w / 4) .., keys 16 (w % 4) ..) computes 32 x 16 of them; the four warps of a row half exchange row maxima
//     and sums through shared memory (a named barrier of their own);
//   the weights go to shared memory as bfloat16, and a warp adds up its rows' share of the value columns, 16 (w % 4 + 4 i) .. + 15.
// A row's keys end at its token's position; rows past the tokens or heads see nothing and are not written.
constexpr int ROWS = 64, SUB = 32, RING = 3, TILE_WARPS = 8;

__device__ __forceinline__ void half_barrier(int half) { asm volatile("bar.sync %0, 128;\n" ::"r"(1 + half) : "memory"); }

template <int COLS>                                                         // 16-column value blocks per warp: rank <= 64 * COLS
__global__ void __launch_bounds__(TILE_WARPS * 32, 1)
attention_latent_tiles_kernel(const bf16* __restrict__ qa, const bf16* __restrict__ cache, const int* __restrict__ block_table, int table_stride,
                              const int* __restrict__ tiles, const int* __restrict__ positions, const float* __restrict__ sink, bf16* __restrict__ out,
                              float* __restrict__ part_o, float* __restrict__ part_ml, int heads, int group, int per_cta, int rank, int rot, int page_size,
                              long long page_stride, int num_pages, int splits, int tile_stride, int* __restrict__ status) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ __align__(8) uint64_t full[RING];
    __shared__ int abort_flag;
    const int D = rank + rot, D16 = (D + 15) / 16 * 16, DS = D16 + 8;
    bf16* Qs = reinterpret_cast<bf16*>(smem);
    bf16* Ks = Qs + ROWS * DS;
    bf16* Ps = Ks + RING * SUB * DS;
    float* red_max = reinterpret_cast<float*>(Ps + ROWS * (KT + 8));        // [4][ROWS]
    float* red_sum = red_max + 4 * ROWS;
    // later tokens see more keys: start them first
    const int per_tile = (128 + per_cta - 1) / per_cta, item = gridDim.x - 1 - blockIdx.x;
    const int tile = item / per_tile, first = item % per_tile * per_cta;
    const int count = min(per_cta, tiles[tile * 3 + 2] - first);
    if (count <= 0) return;
    const int t0 = tiles[tile * 3 + 1] + first, head0 = blockIdx.y * group, live_heads = min(group, heads - head0), part = blockIdx.z;
    const int* table = block_table + (size_t)tiles[tile * 3] * table_stride;
    const int pos0 = positions[t0], last = pos0 + count - 1;                // positions of a tile's tokens are consecutive
    const int key_tiles = last / KT + 1, per = (key_tiles + splits - 1) / splits;
    const int tile0 = part * per, my_tiles = max(0, min(key_tiles, tile0 + per) - tile0), subs = 2 * my_tiles;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = warp >> 2, quarter = warp & 3;
    const int chunks = D / 8;

    for (int i = threadIdx.x; i < ROWS * chunks; i += blockDim.x) {
        const int r = i / chunks, c = i % chunks, token = r / group, head = r % group;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (token < count && head < live_heads) v = *reinterpret_cast<const uint4*>(qa + ((size_t)(t0 + token) * heads + head0 + head) * D + c * 8);
        *reinterpret_cast<uint4*>(Qs + r * DS + c * 8) = v;
    }
    for (int i = threadIdx.x; i < (ROWS + RING * SUB) * (DS - D); i += blockDim.x) Qs[(i / (DS - D)) * DS + D + i % (DS - D)] = __float2bfloat16(0.f);     // Q and K rows lie behind one another
    if (threadIdx.x == 0) {
        for (int b = 0; b < RING; ++b) mbar_init(&full[b], 1);
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    __syncthreads();

    // half tile n of this CTA's part into ring place n % RING (the first warp, all lanes)
    auto load = [&](int n) {
        const int j = tile0 * KT + n * SUB + lane, b = n % RING;
        bf16* dst = Ks + (b * SUB + lane) * DS;
        const bool there = j <= last;
        if (!there)                                                         // rows past the last token's position: zeros
            for (int c = 0; c < chunks; ++c) *reinterpret_cast<uint4*>(dst + c * 8) = make_uint4(0u, 0u, 0u, 0u);
        // the place was last touched by ldmatrix and plain stores: order them before the copies that overwrite it
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
        const int rows = __popc(__ballot_sync(0xffffffffu, there));
        if (lane == 0) mbar_expect_tx(&full[b], (uint32_t)rows * (uint32_t)D * 2u);
        __syncwarp();
        if (there) {
            int page = table[j / page_size];
            if (page < 0 || page >= num_pages) {                            // a complaint, and the row's bytes from a page that exists
                atomicOr(status, EG_STATUS_BAD_PAGE);
                page = 0;
            }
            asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n" ::"r"(smem_addr(dst)),
                         "l"(cache + (size_t)page * page_stride + (size_t)(j % page_size) * D), "r"((uint32_t)D * 2u), "r"(smem_addr(&full[b]))
                         : "memory");
        }
    };
    int issued = 0;                                                         // half tiles asked for (the first warp's count)
    if (warp == 0)
        for (; issued < min(subs, RING); ++issued) load(issued);

    // this thread's rows: block mt, rows lane / 4 and lane / 4 + 8 of its 16; the last key each sees (-1: no such row)
    int limit[2][2];
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int row = half * 32 + mt * 16 + lane / 4 + 8 * r, token = row / group;
            limit[mt][r] = token < count && row % group < live_heads ? pos0 + token : -1;
        }
    float o[COLS][2][2][4];
#pragma unroll
    for (int i = 0; i < COLS; ++i)
#pragma unroll
        for (int e = 0; e < 16; ++e) o[i][e >> 3][(e >> 2) & 1][e & 3] = 0.f;
    float m_run[2][2] = {{-INFINITY, -INFINITY}, {-INFINITY, -INFINITY}}, l_run[2][2] = {{0.f, 0.f}, {0.f, 0.f}};

    for (int i = 0; i < my_tiles; ++i) {
        const int n0 = 2 * i, b0 = n0 % RING, b1 = (n0 + 1) % RING;
        const bool ok = mbar_wait_bounded(&full[b0], (uint32_t)(n0 / RING) & 1u, &abort_flag, status, 1u << 24) &&
                        mbar_wait_bounded(&full[b1], (uint32_t)((n0 + 1) / RING) & 1u, &abort_flag, status, 1u << 24);
        // everybody is past the tile before this one: its second half's place is free
        if (!__syncthreads_and(ok)) break;
        if (warp == 0 && issued < subs && issued < n0 + RING) load(issued++);
        const int j0 = (tile0 + i) * KT;
        float s[2][2][4] = {};
        {
            const bf16* a_at = Qs + (half * 32 + lane % 16) * DS + (lane / 16) * 8;
            const bf16* b_at = Ks + ((quarter < 2 ? b0 : b1) * SUB + (quarter & 1) * 16 + (lane % 8) + (lane / 16) * 8) * DS + ((lane / 8) % 2) * 8;
            // the fragments of the next step are on their way while a step's products run (a warp has one neighbour on its scheduler)
            uint32_t a0[2][4], a1[2][4], b[2][4];
            auto fetch = [&](int buf, int k0) {
                ldmatrix_x4(b[buf], b_at + k0);
                ldmatrix_x4(a0[buf], a_at + k0);
                ldmatrix_x4(a1[buf], a_at + 16 * DS + k0);
            };
            auto multiply = [&](int buf) {
                mma_bf16_16816(s[0][0], a0[buf], b[buf][0], b[buf][1]);
                mma_bf16_16816(s[0][1], a0[buf], b[buf][2], b[buf][3]);
                mma_bf16_16816(s[1][0], a1[buf], b[buf][0], b[buf][1]);
                mma_bf16_16816(s[1][1], a1[buf], b[buf][2], b[buf][3]);
            };
            fetch(0, 0);
            int k0 = 0;
            for (; k0 + 32 <= D16; k0 += 32) {
                fetch(1, k0 + 16);
                multiply(0);
                if (k0 + 32 < D16) fetch(0, k0 + 32);
                multiply(1);
            }
            if (k0 < D16) multiply(0);
        }
#pragma unroll
        for (int mt = 0; mt < 2; ++mt) {
            float top[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int q = 0; q < 2; ++q)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int j = j0 + quarter * 16 + q * 8 + 2 * (lane % 4) + (e & 1);
                    if (j > limit[mt][e >> 1]) s[mt][q][e] = -INFINITY;
                    top[e >> 1] = fmaxf(top[e >> 1], s[mt][q][e]);
                }
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                top[r] = quad_max(top[r]);
                if (lane % 4 == 0) red_max[quarter * ROWS + half * 32 + mt * 16 + lane / 4 + 8 * r] = top[r];
            }
        }
        half_barrier(half);
        bool moved = false;
        float alpha[2][2];
#pragma unroll
        for (int mt = 0; mt < 2; ++mt) {
            float sum[2] = {0.f, 0.f};
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int row = half * 32 + mt * 16 + lane / 4 + 8 * r;
                float m = m_run[mt][r];
#pragma unroll
                for (int w = 0; w < 4; ++w) m = fmaxf(m, red_max[w * ROWS + row]);
                alpha[mt][r] = m == -INFINITY ? 1.f : expf(m_run[mt][r] - m);        // exp(-inf) = 0 at the first keys
                moved |= alpha[mt][r] != 1.f;
                m_run[mt][r] = m;
            }
#pragma unroll
            for (int q = 0; q < 2; ++q) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float m = m_run[mt][e >> 1], p = m == -INFINITY ? 0.f : expf(s[mt][q][e] - m);
                    s[mt][q][e] = p;
                    sum[e >> 1] += p;
                }
                bf16* at = Ps + (half * 32 + mt * 16 + lane / 4) * (KT + 8) + quarter * 16 + q * 8 + 2 * (lane % 4);
                *reinterpret_cast<uint32_t*>(at) = pack_bf16(s[mt][q][0], s[mt][q][1]);
                *reinterpret_cast<uint32_t*>(at + 8 * (KT + 8)) = pack_bf16(s[mt][q][2], s[mt][q][3]);
            }
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                sum[r] = quad_sum(sum[r]);
                if (lane % 4 == 0) red_sum[quarter * ROWS + half * 32 + mt * 16 + lane / 4 + 8 * r] = sum[r];
            }
        }
        half_barrier(half);
#pragma unroll
        for (int mt = 0; mt < 2; ++mt)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                float sum = 0.f;
#pragma unroll
                for (int w = 0; w < 4; ++w) sum += red_sum[w * ROWS + half * 32 + mt * 16 + lane / 4 + 8 * r];
                l_run[mt][r] = l_run[mt][r] * alpha[mt][r] + sum;
            }
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
            for (int c = 0; c < COLS; ++c)
#pragma unroll
                for (int e = 0; e < 16; ++e) o[c][e >> 3][(e >> 2) & 1][e & 3] *= alpha[e >> 3][(e >> 1) & 1];
        }
        const bf16* p_at = Ps + (half * 32 + lane % 16) * (KT + 8) + (lane / 16) * 8;
        const bf16* v_at = Ks + ((lane % 8) + ((lane / 8) % 2) * 8) * DS + (lane / 16) * 8;
#pragma unroll
        for (int kk = 0; kk < KT / 16; ++kk) {
            if (kk == 2) {                                                  // the tile's first half is used up
                __syncthreads();
                if (warp == 0 && issued < subs) load(issued++);
            }
            uint32_t a0[4], a1[4], b[2][4];
            const bf16* rows = v_at + (size_t)((kk < 2 ? b0 : b1) * SUB + (kk & 1) * 16) * DS;
            // (a block past the rank reads the row's last columns and its products go nowhere)
            auto column = [&](int c) { return min(16 * (quarter + 4 * c), D16 - 16); };
            ldmatrix_x4_trans(b[0], rows + column(0));
            ldmatrix_x4(a0, p_at + kk * 16);
            ldmatrix_x4(a1, p_at + 16 * (KT + 8) + kk * 16);
#pragma unroll
            for (int c = 0; c < COLS; ++c) {
                if (c + 1 < COLS) ldmatrix_x4_trans(b[(c + 1) & 1], rows + column(c + 1));
                mma_bf16_16816(o[c][0][0], a0, b[c & 1][0], b[c & 1][1]);
                mma_bf16_16816(o[c][0][1], a0, b[c & 1][2], b[c & 1][3]);
                mma_bf16_16816(o[c][1][0], a1, b[c & 1][0], b[c & 1][1]);
                mma_bf16_16816(o[c][1][1], a1, b[c & 1][2], b[c & 1][3]);
            }
        }
    }
    if (abort_flag) {                                                       // a wait gave up: the copies in flight have to land, nothing is written
        if (warp == 0)
            for (int n = max(0, issued - RING); n < issued; ++n)
                for (unsigned k = 0; k < (1u << 24); ++k)
                    if (mbar_try_wait(&full[n % RING], (uint32_t)(n / RING) & 1u)) break;
        return;
    }
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            if (limit[mt][r] < 0) continue;
            const int in_cta = half * 32 + mt * 16 + lane / 4 + 8 * r, head = head0 + in_cta % group;
            const size_t row = (size_t)(t0 + in_cta / group) * heads + head;
            const size_t part_row = ((size_t)tile * tile_stride + first + in_cta / group) * heads + head;
            float scale = 1.f;
            if (splits == 1) {
                const float sk = sink ? sink[head] : -INFINITY, top = fmaxf(m_run[mt][r], sk), f = expf(m_run[mt][r] - top);
                scale = f / (l_run[mt][r] * f + (sink ? expf(sk - top) : 0.f));
            } else if (quarter == 0 && lane % 4 == 0) {
                part_ml[(part_row * splits + part) * 2] = m_run[mt][r];
                part_ml[(part_row * splits + part) * 2 + 1] = l_run[mt][r];
            }
#pragma unroll
            for (int c = 0; c < COLS; ++c)
#pragma unroll
                for (int q = 0; q < 2; ++q) {
                    const int col = 16 * (quarter + 4 * c) + 8 * q + 2 * (lane % 4);
                    if (col >= rank) continue;
                    const float v0 = o[c][mt][q][2 * r] * scale, v1 = o[c][mt][q][2 * r + 1] * scale;
                    if (splits == 1) *reinterpret_cast<uint32_t*>(out + row * rank + col) = pack_bf16(v0, v1);
                    else *reinterpret_cast<float2*>(part_o + (part_row * splits + part) * rank + col) = make_float2(v0, v1);
                }
        }
}

size_t tiles_smem(int rank, int rot) {
    const int DS = (rank + rot + 15) / 16 * 16 + 8;
    return (size_t)(ROWS + RING * SUB) * DS * 2 + ROWS * (KT + 8) * 2 + 8 * ROWS * 4;
}

// one thread per (token, head, pair): the rotated part of the query, scaled, into qa [T, heads, rank + rot]
__global__ void latent_rotate_query_kernel(const bf16* __restrict__ q, long long ldq, const int* __restrict__ positions, const float* __restrict__ inv_freq,
                                           int rot_dims, int rot_half, float scale, bf16* __restrict__ qa, int tokens, int heads, int dim, int rot, int rank) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const int half = (rot + 1) / 2;
    if (i >= (long long)tokens * heads * half) return;
    const int pair = (int)(i % half), h = (int)((i / half) % heads), t = (int)(i / ((long long)half * heads));
    const bf16* src = q + (size_t)t * ldq + (size_t)h * (dim + rot) + dim;
    bf16* dst = qa + ((size_t)t * heads + h) * (rank + rot) + rank;
    const int d = 2 * pair;
    if (d < rot_dims) {                             // as many pairs are turned as rot_dims has, neighbours or half of rot_dims apart
        float sn, cs;
        sincosf((float)positions[t] * inv_freq[pair], &sn, &cs);
        const int d0 = rot_half ? pair : d, d1 = rot_half ? pair + rot_dims / 2 : d + 1;
        const float a = __bfloat162float(src[d0]), b = __bfloat162float(src[d1]);
        dst[d0] = __float2bfloat16_rn((a * cs - b * sn) * scale);
        dst[d1] = __float2bfloat16_rn((b * cs + a * sn) * scale);
    } else {
        dst[d] = __float2bfloat16_rn(__bfloat162float(src[d]) * scale);
        if (d + 1 < rot) dst[d + 1] = __float2bfloat16_rn(__bfloat162float(src[d + 1]) * scale);
    }
}
}  // namespace

// whether eg_attention_latent_mma takes these sizes
EG_API int eg_attention_latent_mma_takes(int rank, int rot) {
    const int D = rank + rot, DS = (D + 15) / 16 * 16 + 8;
    const size_t smem = (size_t)(16 + KT) * DS * 2 + 16 * (KT + 8) * 2 + 2 * WARPS * 16 * 4;
    return D % 8 == 0 && rank % 8 == 0 && rank > 0 && rank <= 16 * WARPS * PAIRS && smem <= 200 * 1024;
}

// qa [T, heads, rank + rot] bfloat16 (scaled, rotated); cache rows bfloat16; out [T, heads, rank] bfloat16.  splits > 1:
// part_o [tokens, heads, splits, rank] and part_ml [tokens, heads, splits, 2] float32 scratch.  token_list: the `tokens` tokens to work
// on, or null for all.  sink [heads] float32 or null.
EG_API int eg_attention_latent_mma(cudaStream_t stream, const void* qa, const void* cache, const int* block_table, int table_stride, const int* token_seq,
                                   const int* positions, const int* token_list, const float* sink, void* out, float* part_o, float* part_ml, int tokens, int heads, int rank, int rot,
                                   int page_size, long long page_stride, int num_pages, int splits, int* status) {
    if (tokens <= 0) return 0;
    if (!eg_attention_latent_mma_takes(rank, rot) || splits < 1 || splits > 64 || (splits > 1 && (!part_o || !part_ml)) || page_stride % 8 || (uintptr_t)cache % 16 || (uintptr_t)qa % 16)
        return (int)cudaErrorInvalidValue;
    const int D = rank + rot, DS = (D + 15) / 16 * 16 + 8;
    const size_t smem = (size_t)(16 + KT) * DS * 2 + 16 * (KT + 8) * 2 + 2 * WARPS * 16 * 4;
    static size_t configured = 0;
    if (smem > configured) {
        const cudaError_t e = cudaFuncSetAttribute(attention_latent_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = smem;
    }
    dim3 grid(tokens, (heads + 15) / 16, splits);
    attention_latent_mma_kernel<<<grid, WARPS * 32, smem, stream>>>((const bf16*)qa, (const bf16*)cache, block_table, table_stride, token_seq, positions,
                                                                     token_list, sink, (bf16*)out, part_o, part_ml, heads, rank, rot, page_size, page_stride, num_pages, splits, status);
    if (splits > 1)
        attention_latent_merge_kernel<<<tokens * heads, 128, 0, stream>>>(part_o, part_ml, token_list, nullptr, 1, sink, (bf16*)out, heads, rank, splits);
    return eg_launch_status();
}

// whether eg_attention_latent_tiles takes these sizes, and how many tokens a CTA takes (0: it does not)
EG_API int eg_attention_latent_tiles_tokens(int heads, int rank, int rot) {
    if (heads <= 0 || !eg_attention_latent_mma_takes(rank, rot) || tiles_smem(rank, rot) > 227 * 1024 - 1024) return 0;
    const int groups = (heads + 15) / 16, group = (heads + groups - 1) / groups;
    return ROWS / group < 128 ? ROWS / group : 128;
}

// Prompt portions: tiles [num_tiles][3] = (block table row, first token, tokens <= 128), consecutive positions of one request each.
// Other arguments as eg_attention_latent_mma, except part_o [num_tiles * tile_stride, heads, splits, rank] and part_ml alike, with
// tile_stride at least the most tokens of a tile.
EG_API int eg_attention_latent_tiles(cudaStream_t stream, const void* qa, const void* cache, const int* block_table, int table_stride, const int* tiles,
                                     int num_tiles, const int* positions, const float* sink, void* out, float* part_o, float* part_ml, int heads, int rank, int rot,
                                     int page_size, long long page_stride, int num_pages, int splits, int tile_stride, int* status) {
    if (num_tiles <= 0) return 0;
    const int per_cta = eg_attention_latent_tiles_tokens(heads, rank, rot);
    if (!per_cta || splits < 1 || splits > 64 || (splits > 1 && (!part_o || !part_ml)) || page_stride % 8 || (uintptr_t)cache % 16 || (uintptr_t)qa % 16 || tile_stride < 1)
        return (int)cudaErrorInvalidValue;
    const int groups = (heads + 15) / 16, group = (heads + groups - 1) / groups;
    const size_t smem = tiles_smem(rank, rot);
    dim3 grid(num_tiles * ((128 + per_cta - 1) / per_cta), groups, splits);
#define EG_TILES(COLS)                                                                                                                                        \
    {                                                                                                                                                         \
        static size_t configured = 0;                                                                                                                         \
        if (smem > configured) {                                                                                                                              \
            const cudaError_t e = cudaFuncSetAttribute(attention_latent_tiles_kernel<COLS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);          \
            if (e != cudaSuccess) return (int)e;                                                                                                              \
            configured = smem;                                                                                                                                \
        }                                                                                                                                                     \
        attention_latent_tiles_kernel<COLS><<<grid, TILE_WARPS * 32, smem, stream>>>((const bf16*)qa, (const bf16*)cache, block_table, table_stride, tiles,    \
                                                                                     positions, sink, (bf16*)out, part_o, part_ml, heads, group, per_cta, rank, \
                                                                                     rot, page_size, page_stride, num_pages, splits, tile_stride, status);     \
    }
    if (rank <= 64) EG_TILES(1) else if (rank <= 128) EG_TILES(2) else if (rank <= 256) EG_TILES(4) else EG_TILES(8)
#undef EG_TILES
    if (splits > 1)
        attention_latent_merge_kernel<<<num_tiles * tile_stride * heads, 128, 0, stream>>>(part_o, part_ml, nullptr, tiles, tile_stride, sink, (bf16*)out, heads, rank, splits);
    return eg_launch_status();
}

// the rotated, scaled part of the queries: qa[t, h, rank:] from q [T, ldq] (head by head: dim plain values, rot rotated ones)
EG_API int eg_latent_rotate_query(cudaStream_t stream, const void* q, long long ldq, const int* positions, const float* inv_freq, int rot_dims, int rot_half,
                                  float scale, void* qa, int tokens, int heads, int dim, int rot, int rank) {
    const long long n = (long long)tokens * heads * ((rot + 1) / 2);
    if (n <= 0) return 0;
    if (rot_dims % 2 || rot_dims > rot) return (int)cudaErrorInvalidValue;
    latent_rotate_query_kernel<<<(unsigned)((n + 255) / 256), 256, 0, stream>>>((const bf16*)q, ldq, positions, inv_freq, rot_dims, rot_half, scale, (bf16*)qa, tokens, heads,
                                                                               dim, rot, rank);
    return eg_launch_status();
}
