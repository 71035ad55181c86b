// RMSNorm fused with the residual addition before it:  h += delta;  out = h * rsqrt(mean(h^2) + eps) * gamma.
// The residual stream h is 32-bit and the sum, the mean of squares and the scaling are 32-bit; only
// `out` is rounded to the model's dtype.  Formula: src/transformer/norm.zig:14-32; the reference's
// device kernel (src/cuda/layer_kernels.cu:17-43) and its separate residual kernels (:46-59) are
// one kernel here.  The order of the reduction depends only on the row width, so a row's result
// does not depend on what else is in the batch.
#include "common.cuh"

template <typename T>
__global__ void add_rmsnorm_kernel(float* __restrict__ h, const T* __restrict__ delta,
                                   const float* __restrict__ gamma, T* __restrict__ out, float eps, int H) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float v = h[base + c];
        if (delta) {
            v += to_float(delta[base + c]);
            h[base + c] = v;
        }
        ss += v * v;
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x)
        out[base + c] = from_float<T>(h[base + c] * inv * gamma[c]);
}

// four consecutive elements (the address is a multiple of four elements) in one load or store
__device__ __forceinline__ void load4(const float* p, float (&d)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    d[0] = v.x; d[1] = v.y; d[2] = v.z; d[3] = v.w;
}
__device__ __forceinline__ void load4(const bf16* p, float (&d)[4]) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    d[0] = a.x; d[1] = a.y; d[2] = b.x; d[3] = b.y;
}
__device__ __forceinline__ void store4(float* p, float a, float b, float c, float d) {
    *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void store4(bf16* p, float a, float b, float c, float d) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    uint2 v;
    v.x = *reinterpret_cast<uint32_t*>(&lo);
    v.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = v;
}

// Rows with H a multiple of 4 and at most 4 * 256 * VEC: each thread keeps its 4 * VEC values in
// registers, so the row is read once.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) add_rmsnorm_vec_kernel(float* __restrict__ h, const T* __restrict__ delta,
                                                              const float* __restrict__ gamma, T* __restrict__ out,
                                                              float eps, int H) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * H;
    float4 v[VEC];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int c = (threadIdx.x + i * 256) * 4;
        v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < H) {
            v[i] = *reinterpret_cast<const float4*>(h + base + c);
            if (delta) {
                float d[4];
                load4(delta + base + c, d);
                v[i].x += d[0];
                v[i].y += d[1];
                v[i].z += d[2];
                v[i].w += d[3];
                *reinterpret_cast<float4*>(h + base + c) = v[i];
            }
            ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        }
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)H + eps);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int c = (threadIdx.x + i * 256) * 4;
        if (c < H) {
            const float4 g = *reinterpret_cast<const float4*>(gamma + c);
            store4(out + base + c, v[i].x * inv * g.x, v[i].y * inv * g.y, v[i].z * inv * g.z, v[i].w * inv * g.w);
        }
    }
}

// The same with a pending term that passes a norm of its own before it is added (a block with a norm
// after each sublayer):  h += delta * rsqrt(mean(delta^2) + eps_d) * gamma_d;  out = rms(h) * gamma.
template <typename T>
__global__ void add_normed_rmsnorm_kernel(float* __restrict__ h, const T* __restrict__ delta, const float* __restrict__ gamma_d,
                                          float eps_d, const float* __restrict__ gamma, T* __restrict__ out, float eps, int H) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * H;
    float sd = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float d = to_float(delta[base + c]);
        sd += d * d;
    }
    sd = block_sum(sd, red);
    const float inv_d = rsqrtf(sd / (float)H + eps_d);
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float v = h[base + c] + to_float(delta[base + c]) * inv_d * gamma_d[c];
        h[base + c] = v;
        ss += v * v;
    }
    if (!out) return;
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x)
        out[base + c] = from_float<T>(h[base + c] * inv * gamma[c]);
}

// `out` (and `gamma`) may be null: then only the residual stream is updated.
ZAI_API int zai_add_normed_rmsnorm(float* h, const void* delta, const float* gamma_d, float eps_d, const float* gamma, void* out,
                                   int dtype, float eps, int N, int H, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    const int threads = H >= 2048 ? 512 : 256;
    ZAI_DISPATCH(dtype, return launch_pdl(add_normed_rmsnorm_kernel<T>, dim3(N), dim3(threads), 0, stream, h, (const T*)delta,
                                          gamma_d, eps_d, gamma, (T*)out, eps, H));
}

ZAI_API int zai_add_rmsnorm(float* h, const void* delta, const float* gamma, void* out, int dtype, float eps,
                            int N, int H, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    const bool aligned = ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(delta) | reinterpret_cast<uintptr_t>(gamma) |
                           reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    if ((H & 3) == 0 && H <= 8192 && aligned) {
        if (H <= 1024) { ZAI_DISPATCH(dtype, return launch_pdl(add_rmsnorm_vec_kernel<T, 1>, dim3(N), dim3(256), 0, stream, h, (const T*)delta, gamma, (T*)out, eps, H)); }
        if (H <= 2048) { ZAI_DISPATCH(dtype, return launch_pdl(add_rmsnorm_vec_kernel<T, 2>, dim3(N), dim3(256), 0, stream, h, (const T*)delta, gamma, (T*)out, eps, H)); }
        if (H <= 4096) { ZAI_DISPATCH(dtype, return launch_pdl(add_rmsnorm_vec_kernel<T, 4>, dim3(N), dim3(256), 0, stream, h, (const T*)delta, gamma, (T*)out, eps, H)); }
        ZAI_DISPATCH(dtype, return launch_pdl(add_rmsnorm_vec_kernel<T, 8>, dim3(N), dim3(256), 0, stream, h, (const T*)delta, gamma, (T*)out, eps, H));
    }
    const int threads = H >= 2048 ? 512 : 256;
    ZAI_DISPATCH(dtype, return launch_pdl(add_rmsnorm_kernel<T>, dim3(N), dim3(threads), 0, stream, h, (const T*)delta, gamma, (T*)out, eps, H));
}

// A block whose two sublayers read the same stream through a norm each:  h += delta (with gamma_d: through the norm of its own);
// out_a = rms(h) * gamma_a,  out_b = rms(h) * gamma_b.  The row is read, summed and written once for both.
template <typename T>
__global__ void add_rmsnorm_pair_kernel(float* __restrict__ h, const T* __restrict__ delta, const float* __restrict__ gamma_d, float eps_d,
                                        const float* __restrict__ gamma_a, const float* __restrict__ gamma_b, T* __restrict__ out_a,
                                        T* __restrict__ out_b, float eps, int H) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * H;
    float inv_d = 1.f;
    if (delta && gamma_d) {
        float sd = 0.f;
        for (int c = threadIdx.x; c < H; c += blockDim.x) {
            const float d = to_float(delta[base + c]);
            sd += d * d;
        }
        inv_d = rsqrtf(block_sum(sd, red) / (float)H + eps_d);
    }
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float v = h[base + c];
        if (delta) {
            v += gamma_d ? to_float(delta[base + c]) * inv_d * gamma_d[c] : to_float(delta[base + c]);
            h[base + c] = v;
        }
        ss += v * v;
    }
    const float inv = rsqrtf(block_sum(ss, red) / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float v = h[base + c] * inv;
        out_a[base + c] = from_float<T>(v * gamma_a[c]);
        out_b[base + c] = from_float<T>(v * gamma_b[c]);
    }
}

// The same with a row's values in registers: H a multiple of 4 and at most 4 * 256 * VEC, 16-byte boundaries.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) add_rmsnorm_pair_vec_kernel(float* __restrict__ h, const T* __restrict__ delta,
                                                                   const float* __restrict__ gamma_d, float eps_d,
                                                                   const float* __restrict__ gamma_a, const float* __restrict__ gamma_b,
                                                                   T* __restrict__ out_a, T* __restrict__ out_b, float eps, int H) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * H;
    float4 v[VEC];
    float d[VEC][4];
    float inv_d = 1.f;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int c = (threadIdx.x + i * 256) * 4;
        v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        d[i][0] = d[i][1] = d[i][2] = d[i][3] = 0.f;
        if (c < H) {
            v[i] = *reinterpret_cast<const float4*>(h + base + c);
            if (delta) load4(delta + base + c, d[i]);
        }
    }
    if (delta) {
        if (gamma_d) {
            float sd = 0.f;
#pragma unroll
            for (int i = 0; i < VEC; ++i) sd += d[i][0] * d[i][0] + d[i][1] * d[i][1] + d[i][2] * d[i][2] + d[i][3] * d[i][3];
            inv_d = rsqrtf(block_sum(sd, red) / (float)H + eps_d);
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const int c = (threadIdx.x + i * 256) * 4;
            if (c < H) {
                float4 g = make_float4(1.f, 1.f, 1.f, 1.f);
                if (gamma_d) g = *reinterpret_cast<const float4*>(gamma_d + c);
                v[i].x += d[i][0] * inv_d * g.x;
                v[i].y += d[i][1] * inv_d * g.y;
                v[i].z += d[i][2] * inv_d * g.z;
                v[i].w += d[i][3] * inv_d * g.w;
                *reinterpret_cast<float4*>(h + base + c) = v[i];
            }
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    const float inv = rsqrtf(block_sum(ss, red) / (float)H + eps);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int c = (threadIdx.x + i * 256) * 4;
        if (c < H) {
            const float4 a = *reinterpret_cast<const float4*>(gamma_a + c), b = *reinterpret_cast<const float4*>(gamma_b + c);
            const float4 n = make_float4(v[i].x * inv, v[i].y * inv, v[i].z * inv, v[i].w * inv);
            store4(out_a + base + c, n.x * a.x, n.y * a.y, n.z * a.z, n.w * a.w);
            store4(out_b + base + c, n.x * b.x, n.y * b.y, n.z * b.z, n.w * b.w);
        }
    }
}

ZAI_API int zai_add_rmsnorm_pair(float* h, const void* delta, const float* gamma_d, float eps_d, const float* gamma_a,
                                 const float* gamma_b, void* out_a, void* out_b, int dtype, float eps, int N, int H,
                                 cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    const uintptr_t all = reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(delta) | reinterpret_cast<uintptr_t>(gamma_d) |
                          reinterpret_cast<uintptr_t>(gamma_a) | reinterpret_cast<uintptr_t>(gamma_b) |
                          reinterpret_cast<uintptr_t>(out_a) | reinterpret_cast<uintptr_t>(out_b);
#define PAIR_GO(KERNEL, THREADS)                                                                                                     \
    ZAI_DISPATCH(dtype, return launch_pdl(KERNEL, dim3(N), dim3(THREADS), 0, stream, h, (const T*)delta, gamma_d, eps_d, gamma_a,     \
                                          gamma_b, (T*)out_a, (T*)out_b, eps, H))
    if ((H & 3) == 0 && H <= 4096 && (all & 15) == 0) {
        if (H <= 1024) PAIR_GO((add_rmsnorm_pair_vec_kernel<T, 1>), 256);
        if (H <= 2048) PAIR_GO((add_rmsnorm_pair_vec_kernel<T, 2>), 256);
        PAIR_GO((add_rmsnorm_pair_vec_kernel<T, 4>), 256);
    }
    PAIR_GO((add_rmsnorm_pair_kernel<T>), H >= 2048 ? 512 : 256);
#undef PAIR_GO
}

// A block whose sublayers read the residual stream itself:  h += delta * rsqrt(mean(delta^2) + eps_d) * gamma_d  (or the
// plain delta without gamma_d, or nothing without delta);  out = h rounded to the activations' dtype.  Sum and norm 32-bit.
template <typename T>
__global__ void add_normed_cast_kernel(float* __restrict__ h, const T* __restrict__ delta, const float* __restrict__ gamma_d,
                                       float eps_d, T* __restrict__ out, int H, const T* __restrict__ delta2) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * H;
    float inv_d = 1.f;
    if (delta && gamma_d) {
        float sd = 0.f;
        for (int c = threadIdx.x; c < H; c += blockDim.x) {
            const float d = to_float(delta[base + c]);
            sd += d * d;
        }
        inv_d = rsqrtf(block_sum(sd, red) / (float)H + eps_d);
    }
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float v = h[base + c];
        if (delta) {
            v += gamma_d ? to_float(delta[base + c]) * inv_d * gamma_d[c] : to_float(delta[base + c]);
            if (delta2) v += to_float(delta2[base + c]);
            h[base + c] = v;
        }
        out[base + c] = from_float<T>(v);
    }
}

// The same for rows of a multiple of four values on 16-byte boundaries: four values a thread and access.
template <typename T>
__global__ void __launch_bounds__(256) add_normed_cast_vec_kernel(float* __restrict__ h, const T* __restrict__ delta,
                                                                  const float* __restrict__ gamma_d, float eps_d, T* __restrict__ out, int H,
                                                                  const T* __restrict__ delta2) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * H;
    float inv_d = 1.f;
    if (delta && gamma_d) {
        float sd = 0.f;
        for (int c = threadIdx.x * 4; c < H; c += blockDim.x * 4) {
            float d[4];
            load4(delta + base + c, d);
            sd += d[0] * d[0] + d[1] * d[1] + d[2] * d[2] + d[3] * d[3];
        }
        inv_d = rsqrtf(block_sum(sd, red) / (float)H + eps_d);
    }
    for (int c = threadIdx.x * 4; c < H; c += blockDim.x * 4) {
        float4 v = *reinterpret_cast<const float4*>(h + base + c);
        if (delta) {
            float d[4];
            load4(delta + base + c, d);
            if (gamma_d) {
                const float4 g = *reinterpret_cast<const float4*>(gamma_d + c);
                v.x += d[0] * inv_d * g.x; v.y += d[1] * inv_d * g.y; v.z += d[2] * inv_d * g.z; v.w += d[3] * inv_d * g.w;
            } else {
                v.x += d[0]; v.y += d[1]; v.z += d[2]; v.w += d[3];
            }
            if (delta2) {
                load4(delta2 + base + c, d);
                v.x += d[0]; v.y += d[1]; v.z += d[2]; v.w += d[3];
            }
            *reinterpret_cast<float4*>(h + base + c) = v;
        }
        store4(out + base + c, v.x, v.y, v.z, v.w);
    }
}

// `delta2`: a second term that is added as it is (or null; only with a first one).
ZAI_API int zai_add_normed_cast(float* h, const void* delta, const float* gamma_d, float eps_d, void* out, int dtype, int N, int H,
                                const void* delta2, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    if (delta2 && !delta) return ZAI_BAD_SIZE;
    const bool aligned = ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(delta) | reinterpret_cast<uintptr_t>(gamma_d) |
                           reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(delta2)) & 15) == 0;
    if ((H & 3) == 0 && aligned)
        ZAI_DISPATCH(dtype, return launch_pdl(add_normed_cast_vec_kernel<T>, dim3(N), dim3(256), 0, stream, h, (const T*)delta, gamma_d,
                                              eps_d, (T*)out, H, (const T*)delta2));
    const int threads = H >= 2048 ? 512 : 256;
    ZAI_DISPATCH(dtype, return launch_pdl(add_normed_cast_kernel<T>, dim3(N), dim3(threads), 0, stream, h, (const T*)delta, gamma_d,
                                          eps_d, (T*)out, H, (const T*)delta2));
}

// RMS norm of activation rows (not the residual stream): out[n, :] = x[n, :C] * rsqrt(mean(x^2) + eps) * gamma, the row
// read from a column slice (row stride x_stride) in the activations' dtype, everything between in 32-bit.
template <typename T>
__global__ void rmsnorm_rows_kernel(T* __restrict__ out, const T* __restrict__ x, int x_stride, const float* __restrict__ gamma,
                                    float eps, int C) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const T* row = x + (size_t)blockIdx.x * x_stride;
    float ss = 0.f;
    for (int c = threadIdx.x; c < C; c += blockDim.x) {
        const float v = to_float(row[c]);
        ss += v * v;
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)C + eps);
    for (int c = threadIdx.x; c < C; c += blockDim.x)
        out[(size_t)blockIdx.x * C + c] = from_float<T>(to_float(row[c]) * inv * (gamma ? gamma[c] : 1.f));
}

ZAI_API int zai_rmsnorm_rows(void* out, const void* x, int x_stride, int dtype, const float* gamma, float eps, int N, int C,
                             cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    if (C < 1 || x_stride < C) return ZAI_BAD_SIZE;
    const int threads = C >= 1024 ? 256 : 128;
    ZAI_DISPATCH(dtype, return launch_pdl(rmsnorm_rows_kernel<T>, dim3(N), dim3(threads), 0, stream, (T*)out, (const T*)x, x_stride,
                                          gamma, eps, C));
}
