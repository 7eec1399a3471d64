// SwiGLU on the fused gate/up projection: out[t, i] = up[t, i] * silu(gate[t, i]),
// silu(g) = g * 1/(1 + exp(-g)) in float32 (src/tensor.cpp:159-174,
// src/cuda/ops/mlp.cu:152-162).  The projection's rows are interleaved, so the
// input row is [gate_0, up_0, gate_1, up_1, ...]: a tile of the product holds both
// halves of every output it covers, which lets the decode kernel apply this in its epilogue.
#include "common.cuh"

template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gate_up, int ld, T* __restrict__ out, int ldo, int inter) {
    const int t = blockIdx.x;
    const int i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= inter) return;
    const T* row = gate_up + (size_t)t * ld;
    const float g = to_f32<T>(row[2 * i]);
    const float u = to_f32<T>(row[2 * i + 1]);
    const float sig = 1.0f / (1.0f + expf(-g));
    out[(size_t)t * ldo + i] = from_f32<T>(u * (g * sig));
}

// Four outputs per thread: one 16-byte (bfloat16) or two 16-byte (float32) loads, one vector store.
template <typename T>
__global__ void swiglu_vec4_kernel(const T* __restrict__ gate_up, int ld, T* __restrict__ out, int ldo, int inter) {
    const int t = blockIdx.x;
    const int i = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
    if (i >= inter) return;
    const T* row = gate_up + (size_t)t * ld + 2 * i;
    float v[8];
    if (sizeof(T) == 2) {
        const uint4 raw = *reinterpret_cast<const uint4*>(row);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            v[2 * k] = __low2float(h[k]);
            v[2 * k + 1] = __high2float(h[k]);
        }
    } else {
        const float4 a = reinterpret_cast<const float4*>(row)[0], b = reinterpret_cast<const float4*>(row)[1];
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
    float r[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const float g = v[2 * k], u = v[2 * k + 1];
        r[k] = u * (g * (1.0f / (1.0f + expf(-g))));
    }
    T* o = out + (size_t)t * ldo + i;
    if (sizeof(T) == 2) {
        uint2 packed;
        __nv_bfloat162 lo = __floats2bfloat162_rn(r[0], r[1]), hi = __floats2bfloat162_rn(r[2], r[3]);
        packed.x = *reinterpret_cast<uint32_t*>(&lo);
        packed.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(o) = packed;
    } else {
        *reinterpret_cast<float4*>(o) = make_float4(r[0], r[1], r[2], r[3]);
    }
}

EG_API int eg_swiglu(cudaStream_t stream, int dtype, const void* gate_up, int ld, void* out, int ldo, int tokens, int inter) {
    if (tokens <= 0) return 0;
    const size_t es = dtype == EG_BF16 ? 2 : 4;
    if (inter % 4 == 0 && ((size_t)ld * es) % 16 == 0 && ((size_t)ldo * es) % (4 * es) == 0 &&
        ((uintptr_t)gate_up % 16) == 0 && ((uintptr_t)out % (4 * es)) == 0) {
        dim3 vgrid(tokens, (inter / 4 + 127) / 128);
        if (dtype == EG_BF16)
            swiglu_vec4_kernel<bf16><<<vgrid, 128, 0, stream>>>((const bf16*)gate_up, ld, (bf16*)out, ldo, inter);
        else
            swiglu_vec4_kernel<float><<<vgrid, 128, 0, stream>>>((const float*)gate_up, ld, (float*)out, ldo, inter);
        return eg_launch_status();
    }
    dim3 grid(tokens, (inter + 255) / 256);
    if (dtype == EG_BF16)
        swiglu_kernel<bf16><<<grid, 256, 0, stream>>>((const bf16*)gate_up, ld, (bf16*)out, ldo, inter);
    else
        swiglu_kernel<float><<<grid, 256, 0, stream>>>((const float*)gate_up, ld, (float*)out, ldo, inter);
    return eg_launch_status();
}

// More activations between the products of a feed-forward, element by element in float32:
//   eg_squared_relu   out[t, c] = max(x[t, c], 0)^2
//   eg_gelu           out[t, c] = x Phi(x), Phi the normal distribution's integral: x / 2 (1 + erf(x / sqrt 2))
//   eg_clamped_glu    on interleaved columns (gate_0, up_0, gate_1, up_1, ...): g = min(gate, limit), u = clamp(up, -limit, limit),
//                     out[t, i] = g * sigmoid(1.702 g) * (u + 1)
template <typename TI, typename TO>
__global__ void squared_relu_kernel(const TI* __restrict__ x, long long ldx, TO* __restrict__ out, long long ldo, int tokens, int n) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * n) return;
    const int t = (int)(i / n), c = (int)(i % n);
    const float z = fmaxf(to_f32<TI>(x[(size_t)t * ldx + c]), 0.f);
    out[(size_t)t * ldo + c] = from_f32<TO>(z * z);
}

// bias: float32 [2 n], interleaved like the columns and added to them first; or null
template <typename TI, typename TO>
__global__ void clamped_glu_kernel(const TI* __restrict__ x, long long ldx, TO* __restrict__ out, long long ldo, int tokens, int n, float limit,
                                   const float* __restrict__ bias) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * n) return;
    const int t = (int)(i / n), c = (int)(i % n);
    const float g = fminf(to_f32<TI>(x[(size_t)t * ldx + 2 * c]) + (bias ? bias[2 * c] : 0.f), limit);
    const float u = fminf(fmaxf(to_f32<TI>(x[(size_t)t * ldx + 2 * c + 1]) + (bias ? bias[2 * c + 1] : 0.f), -limit), limit);
    out[(size_t)t * ldo + c] = from_f32<TO>(g / (1.0f + expf(-1.702f * g)) * (u + 1.0f));
}

EG_API int eg_squared_relu(cudaStream_t stream, const void* x, int x_dtype, long long ldx, void* out, int out_dtype, long long ldo, int tokens, int n) {
    const long long total = (long long)tokens * n;
    if (total <= 0) return 0;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (x_dtype == EG_F32 && out_dtype == EG_F32) squared_relu_kernel<float, float><<<blocks, 256, 0, stream>>>((const float*)x, ldx, (float*)out, ldo, tokens, n);
    else if (x_dtype == EG_F32) squared_relu_kernel<float, bf16><<<blocks, 256, 0, stream>>>((const float*)x, ldx, (bf16*)out, ldo, tokens, n);
    else if (out_dtype == EG_F32) squared_relu_kernel<bf16, float><<<blocks, 256, 0, stream>>>((const bf16*)x, ldx, (float*)out, ldo, tokens, n);
    else squared_relu_kernel<bf16, bf16><<<blocks, 256, 0, stream>>>((const bf16*)x, ldx, (bf16*)out, ldo, tokens, n);
    return eg_launch_status();
}

// x [tokens, 2 n] interleaved -> out [tokens, n]; bias float32 [2 n] (interleaved alike, added to x first) or null
EG_API int eg_clamped_glu_bias(cudaStream_t stream, const void* x, int x_dtype, long long ldx, const float* bias, void* out, int out_dtype, long long ldo, int tokens,
                               int n, float limit) {
    const long long total = (long long)tokens * n;
    if (total <= 0) return 0;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (x_dtype == EG_F32 && out_dtype == EG_F32) clamped_glu_kernel<float, float><<<blocks, 256, 0, stream>>>((const float*)x, ldx, (float*)out, ldo, tokens, n, limit, bias);
    else if (x_dtype == EG_F32) clamped_glu_kernel<float, bf16><<<blocks, 256, 0, stream>>>((const float*)x, ldx, (bf16*)out, ldo, tokens, n, limit, bias);
    else if (out_dtype == EG_F32) clamped_glu_kernel<bf16, float><<<blocks, 256, 0, stream>>>((const bf16*)x, ldx, (float*)out, ldo, tokens, n, limit, bias);
    else clamped_glu_kernel<bf16, bf16><<<blocks, 256, 0, stream>>>((const bf16*)x, ldx, (bf16*)out, ldo, tokens, n, limit, bias);
    return eg_launch_status();
}

// x [tokens, 2 n] interleaved -> out [tokens, n]
EG_API int eg_clamped_glu(cudaStream_t stream, const void* x, int x_dtype, long long ldx, void* out, int out_dtype, long long ldo, int tokens, int n, float limit) {
    return eg_clamped_glu_bias(stream, x, x_dtype, ldx, nullptr, out, out_dtype, ldo, tokens, n, limit);
}

namespace {
template <typename TI, typename TO>
__global__ void gelu_kernel(const TI* __restrict__ x, long long ldx, TO* __restrict__ out, long long ldo, int tokens, int n) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * n) return;
    const int t = (int)(i / n), c = (int)(i % n);
    out[(size_t)t * ldo + c] = from_f32<TO>(gelu_erf(to_f32<TI>(x[(size_t)t * ldx + c])));
}

// values[t, c] *= sigmoid(gate[t, c / span]), in place: span 1 has a gate per value, span v one for every run of v values (a head)
template <typename T>
__global__ void sigmoid_gate_kernel(T* __restrict__ values, long long ldv, const float* __restrict__ gate, long long ldg, int tokens, int n, int span) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * n) return;
    const int t = (int)(i / n), c = (int)(i % n);
    T* v = values + (size_t)t * ldv + c;
    *v = from_f32<T>(to_f32<T>(*v) / (1.0f + expf(-gate[(size_t)t * ldg + c / span])));
}
}  // namespace

EG_API int eg_gelu(cudaStream_t stream, const void* x, int x_dtype, long long ldx, void* out, int out_dtype, long long ldo, int tokens, int n) {
    const long long total = (long long)tokens * n;
    if (total <= 0) return 0;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (x_dtype == EG_F32 && out_dtype == EG_F32) gelu_kernel<float, float><<<blocks, 256, 0, stream>>>((const float*)x, ldx, (float*)out, ldo, tokens, n);
    else if (x_dtype == EG_F32) gelu_kernel<float, bf16><<<blocks, 256, 0, stream>>>((const float*)x, ldx, (bf16*)out, ldo, tokens, n);
    else if (out_dtype == EG_F32) gelu_kernel<bf16, float><<<blocks, 256, 0, stream>>>((const bf16*)x, ldx, (float*)out, ldo, tokens, n);
    else gelu_kernel<bf16, bf16><<<blocks, 256, 0, stream>>>((const bf16*)x, ldx, (bf16*)out, ldo, tokens, n);
    return eg_launch_status();
}

// the same in bfloat16, eight values a thread: span 1, or a span that is a multiple of eight
namespace {
template <bool PER_VALUE>
__global__ void __launch_bounds__(256) sigmoid_gate_vec_kernel(bf16* __restrict__ values, long long ldv, const float* __restrict__ gate, long long ldg, int tokens, int n,
                                                               int span) {
    const int pieces = n / 8;
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * pieces) return;
    const int t = (int)(i / pieces), c = (int)(i % pieces) * 8;
    uint4* at = reinterpret_cast<uint4*>(values + (size_t)t * ldv + c);
    uint4 raw = *at;
    float g[8];
    const float* src = gate + (size_t)t * ldg + (PER_VALUE ? c : c / span);
#pragma unroll
    for (int q = 0; q < 8; ++q) g[q] = PER_VALUE ? src[q] : (q == 0 ? src[0] : g[0]);
#pragma unroll
    for (int q = 0; q < 4; ++q) {
        __nv_bfloat162& pair = reinterpret_cast<__nv_bfloat162*>(&raw)[q];
        const float2 f = __bfloat1622float2(pair);
        pair = __floats2bfloat162_rn(f.x / (1.0f + expf(-g[2 * q])), f.y / (1.0f + expf(-g[2 * q + 1])));
    }
    *at = raw;
}
}  // namespace

// values [tokens, ldv] in dtype, n columns; gate float32 [tokens, ldg], n / span columns
EG_API int eg_sigmoid_gate(cudaStream_t stream, int dtype, void* values, long long ldv, const float* gate, long long ldg, int tokens, int n, int span) {
    const long long total = (long long)tokens * n;
    if (total <= 0) return 0;
    if (span < 1 || n % span) return (int)cudaErrorInvalidValue;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (dtype == EG_BF16 && n % 8 == 0 && ldv % 8 == 0 && (span == 1 || span % 8 == 0) && (uintptr_t)values % 16 == 0) {
        const unsigned vec_blocks = (unsigned)((total / 8 + 255) / 256);
        if (span == 1) sigmoid_gate_vec_kernel<true><<<vec_blocks, 256, 0, stream>>>((bf16*)values, ldv, gate, ldg, tokens, n, span);
        else sigmoid_gate_vec_kernel<false><<<vec_blocks, 256, 0, stream>>>((bf16*)values, ldv, gate, ldg, tokens, n, span);
        return eg_launch_status();
    }
    if (dtype == EG_BF16) sigmoid_gate_kernel<bf16><<<blocks, 256, 0, stream>>>((bf16*)values, ldv, gate, ldg, tokens, n, span);
    else sigmoid_gate_kernel<float><<<blocks, 256, 0, stream>>>((float*)values, ldv, gate, ldg, tokens, n, span);
    return eg_launch_status();
}
