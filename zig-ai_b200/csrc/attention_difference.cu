// The two maps of differential attention combined: the attention kernels leave o [N, 2 H, Dp], the heads' maps side by side
// (map 1 of head 0, map 2 of head 0, map 1 of head 1, ...), of every Dp values the first Dv being a head's own;
//
//   d = o1 - lambda o2,   out = factor * d / sqrt(mean(d^2) + eps)          per head over its Dv values, 32-bit
//
// A warp a (row, head); out [N, H Dv].
#include "common.cuh"

template <typename T>
__global__ void __launch_bounds__(128) attention_difference_kernel(T* __restrict__ out, const T* __restrict__ o, float lambda, float factor,
                                                                   float eps, int total, int Dv, int Dp) {
    pdl_trigger();
    pdl_wait();
    const int item = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= total) return;
    const T* a1 = o + (size_t)item * 2 * Dp;
    const T* a2 = a1 + Dp;
    T* dst = out + (size_t)item * Dv;
    float v[8], q = 0.f;                           // up to 256 values stay in registers; what lies beyond is read again
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        v[i] = c < Dv ? to_float(a1[c]) - lambda * to_float(a2[c]) : 0.f;
        q += v[i] * v[i];
    }
    for (int c = lane + 256; c < Dv; c += 32) {
        const float d = to_float(a1[c]) - lambda * to_float(a2[c]);
        q += d * d;
    }
    const float scale = factor * rsqrtf(warp_sum(q) / (float)Dv + eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        if (c < Dv) dst[c] = from_float<T>(v[i] * scale);
    }
    for (int c = lane + 256; c < Dv; c += 32) dst[c] = from_float<T>((to_float(a1[c]) - lambda * to_float(a2[c])) * scale);
}

ZAI_API int zai_attention_difference(void* out, const void* o, int dtype, float lambda, float factor, float eps, int N, int H, int Dv,
                                     int Dp, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    const long long total = (long long)N * H;
    if (H < 1 || Dv < 1 || Dp < Dv || total > 0x7fffffff - 4) return ZAI_BAD_SIZE;
    ZAI_DISPATCH(dtype, return launch_pdl(attention_difference_kernel<T>, dim3((unsigned)((total + 3) / 4)), dim3(128), 0, stream, (T*)out,
                                          (const T*)o, lambda, factor, eps, (int)total, Dv, Dp));
}
