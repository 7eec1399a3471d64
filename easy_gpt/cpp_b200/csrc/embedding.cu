// Token embedding: residual[t, :] = table[id[t], :] widened to float32.
// The reference gathers rows on the CPU with a range check that throws
// (src/models/embedding.cpp:54-76); here a bad id sets a status bit and the row
// becomes zero, so that the kernel never reads outside the table.
#include "common.cuh"

template <typename T>
__global__ void embedding_gather_kernel(const int* __restrict__ ids, const T* __restrict__ table,
                                        float* __restrict__ residual, int hidden, int vocab, int* status) {
    const int t = blockIdx.x;
    const int id = ids[t];
    float* out = residual + (size_t)t * hidden;
    if (id < 0 || id >= vocab) {
        if (threadIdx.x == 0) atomicOr(status, EG_STATUS_BAD_TOKEN);
        for (int j = threadIdx.x; j < hidden; j += blockDim.x) out[j] = 0.0f;
        return;
    }
    const T* row = table + (size_t)id * hidden;
    for (int j = threadIdx.x; j < hidden; j += blockDim.x) out[j] = to_f32<T>(row[j]);
}

EG_API int eg_embedding_gather(cudaStream_t stream, int dtype, const int* ids, const void* table, float* residual,
                               int tokens, int hidden, int vocab, int* status) {
    if (tokens <= 0) return 0;
    const int threads = hidden >= 1024 ? 256 : 128;
    if (dtype == EG_BF16)
        embedding_gather_kernel<bf16><<<tokens, threads, 0, stream>>>(ids, (const bf16*)table, residual, hidden, vocab, status);
    else
        embedding_gather_kernel<float><<<tokens, threads, 0, stream>>>(ids, (const float*)table, residual, hidden, vocab, status);
    return eg_launch_status();
}

// residual[t, :] = gain * x / sqrt(mean(x^2) + eps) with x = table[id[t], :], in float32: the gather and the norm behind it in one kernel.
namespace {
template <typename T>
__global__ void embedding_rmsnorm_kernel(const int* __restrict__ ids, const T* __restrict__ table, const float* __restrict__ gain, float eps,
                                         float* __restrict__ residual, int hidden, int vocab, int* status) {
    __shared__ float scratch[32];
    const int t = blockIdx.x;
    const int id = ids[t];
    float* out = residual + (size_t)t * hidden;
    if (id < 0 || id >= vocab) {
        if (threadIdx.x == 0) atomicOr(status, EG_STATUS_BAD_TOKEN);
        for (int j = threadIdx.x; j < hidden; j += blockDim.x) out[j] = 0.0f;
        return;
    }
    const T* row = table + (size_t)id * hidden;
    float ss = 0.f;
    for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
        const float v = to_f32<T>(row[j]);
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps);
    for (int j = threadIdx.x; j < hidden; j += blockDim.x) out[j] = gain[j] * (to_f32<T>(row[j]) * inv);
}
}  // namespace

EG_API int eg_embedding_rmsnorm(cudaStream_t stream, int dtype, const int* ids, const void* table, const float* gain, float eps, float* residual, int tokens,
                                int hidden, int vocab, int* status) {
    if (tokens <= 0) return 0;
    const int threads = hidden >= 1024 ? 256 : 128;
    if (dtype == EG_BF16) embedding_rmsnorm_kernel<bf16><<<tokens, threads, 0, stream>>>(ids, (const bf16*)table, gain, eps, residual, hidden, vocab, status);
    else embedding_rmsnorm_kernel<float><<<tokens, threads, 0, stream>>>(ids, (const float*)table, gain, eps, residual, hidden, vocab, status);
    return eg_launch_status();
}

// residual[t, 2i] += sin(a), residual[t, 2i + 1] += cos(a) with a = position * f_i, the frequency f_i = head[i] + tail[i] in two float32
// pieces: the angle's rounding error is worked out and taken into account, so that far positions keep a 32-bit angle.
namespace {
__global__ void add_waves_kernel(float* __restrict__ residual, const int* __restrict__ positions, const float* __restrict__ head, const float* __restrict__ tail,
                                 int tokens, int hidden) {
    const int pairs = (hidden + 1) / 2;
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * pairs) return;
    const int t = (int)(i / pairs), c = (int)(i % pairs);
    const float p = (float)positions[t], f = head[c], a = p * f, rest = fmaf(p, f, -a) + p * tail[c];
    float s, cs;
    sincosf(a, &s, &cs);
    float* x = residual + (size_t)t * hidden + 2 * c;
    x[0] += fmaf(cs, rest, s);                      // sin(a + rest), rest a few rounding errors of a
    if (2 * c + 1 < hidden) x[1] += fmaf(-s, rest, cs);
}
}  // namespace

EG_API int eg_add_waves(cudaStream_t stream, float* residual, const int* positions, const float* head, const float* tail, int tokens, int hidden) {
    if (tokens <= 0) return 0;
    const long long n = (long long)tokens * ((hidden + 1) / 2);
    add_waves_kernel<<<(unsigned)((n + 127) / 128), 128, 0, stream>>>(residual, positions, head, tail, tokens, hidden);
    return eg_launch_status();
}
