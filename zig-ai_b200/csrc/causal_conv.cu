// Short causal depthwise convolution over time with a per-request history, an optional bias and an
// optional SiLU:
//
//   y[t, c] = act( b[c] + sum_{j < L} w[c, j] * u[t - (L-1) + j, c] ),   u = history ++ x
//
// Tap L-1 multiplies the current token.  The history is the last L-1 inputs of the request (zero for
// a new request), kept in 32-bit [slots, L-1, C], oldest first.  x may be a column slice of a wider
// matrix (its row stride is given).  Sums and the activation are 32-bit; y is rounded to the model's
// dtype.  A step of prompt portions runs two kernels (all outputs read the old history, then the
// history is replaced); a step of single tokens runs one.
#include "common.cuh"

#define ZAI_CONV_MAX_TAPS 16

template <typename T>
__global__ void causal_conv_kernel(T* __restrict__ out, int out_stride, const T* __restrict__ x, int x_stride,
                                   const float* __restrict__ taps, const float* __restrict__ bias,
                                   const float* __restrict__ state, const int* __restrict__ seq_idx,
                                   const int* __restrict__ cu_q, const int* __restrict__ slot_ids, int C, int L, int act,
                                   int num_slots, int* __restrict__ status) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= C) return;
    const int s = seq_idx[t], start = cu_q[s];
    const int slot = zai_checked_slot(slot_ids[s], num_slots, status);
    const float* hist = state + (size_t)slot * (L - 1) * C;
    float acc = bias ? bias[c] : 0.f;
    for (int j = 0; j < L; ++j) {
        const int tt = t - (L - 1) + j;
        const float u = tt >= start ? to_float(x[(size_t)tt * x_stride + c]) : hist[(size_t)(L - 1 + tt - start) * C + c];
        acc += taps[(size_t)c * L + j] * u;
    }
    if (act) acc = acc / (1.f + expf(-acc));
    out[(size_t)t * out_stride + c] = from_float<T>(acc);
}

// The same with a thread owning four neighbouring channels and walking R rows with the last L - 1 inputs in
// registers: every input is read once.  Rows of several requests may follow one another; at a request's first row the
// inputs before it come from its history.
template <typename T, int L, int R>
__global__ void __launch_bounds__(128) causal_conv_rows_kernel(T* __restrict__ out, int out_stride, const T* __restrict__ x, int x_stride,
                                                               const float* __restrict__ taps, const float* __restrict__ bias,
                                                               const float* __restrict__ state, const int* __restrict__ seq_idx,
                                                               const int* __restrict__ cu_q, const int* __restrict__ slot_ids, int N, int C,
                                                               int act, int num_slots, int* __restrict__ status) {
    constexpr int VEC = 4;
    struct __align__(VEC * sizeof(T)) Pack { T v[VEC]; };
    pdl_trigger();
    pdl_wait();
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC, t0 = blockIdx.x * R, t1 = min(t0 + R, N);
    if (c >= C) return;
    float w[VEC][L], b[VEC], u[L - 1][VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
        b[k] = bias ? bias[c + k] : 0.f;
#pragma unroll
        for (int j = 0; j < L; ++j) w[k][j] = 0.f;
    }
    if constexpr (L == 4) {
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            const float4 q = *reinterpret_cast<const float4*>(taps + (size_t)(c + k) * 4);
            w[k][0] = q.x; w[k][1] = q.y; w[k][2] = q.z; w[k][3] = q.w;
        }
    } else {
#pragma unroll
        for (int k = 0; k < VEC; ++k)
#pragma unroll
            for (int j = 0; j < L; ++j) w[k][j] = taps[(size_t)(c + k) * L + j];
    }
    int s = -1;
    Pack in[R];
#pragma unroll
    for (int i = 0; i < R; ++i)
        if (t0 + i < t1) in[i] = *reinterpret_cast<const Pack*>(x + (size_t)(t0 + i) * x_stride + c);
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int t = t0 + i;
        if (t >= t1) break;
        if (seq_idx[t] != s) {                            // the inputs before row t of this request
            s = seq_idx[t];
            const int start = cu_q[s], slot = zai_checked_slot(slot_ids[s], num_slots, status);
            const float* hist = state + (size_t)slot * (L - 1) * C + c;
#pragma unroll
            for (int j = 0; j < L - 1; ++j) {
                const int tt = t - (L - 1) + j;
                if (tt >= start) {
                    const Pack p = *reinterpret_cast<const Pack*>(x + (size_t)tt * x_stride + c);
#pragma unroll
                    for (int k = 0; k < VEC; ++k) u[j][k] = to_float(p.v[k]);
                } else {
#pragma unroll
                    for (int k = 0; k < VEC; ++k) u[j][k] = hist[(size_t)(L - 1 + tt - start) * C + k];
                }
            }
        }
        Pack o;
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            const float cur = to_float(in[i].v[k]);
            float acc = b[k];
#pragma unroll
            for (int j = 0; j < L - 1; ++j) acc += w[k][j] * u[j][k];
            acc += w[k][L - 1] * cur;
            // (a bfloat16 result: the fast exponential and division err by far less than its rounding)
            if (act) acc = sizeof(T) == 2 ? __fdividef(acc, 1.f + __expf(-acc)) : acc / (1.f + expf(-acc));
            o.v[k] = from_float<T>(acc);
#pragma unroll
            for (int j = 0; j + 1 < L - 1; ++j) u[j][k] = u[j + 1][k];
            u[L - 2][k] = cur;
        }
        *reinterpret_cast<Pack*>(out + (size_t)t * out_stride + c) = o;
    }
}

template <typename T, int L>
static int conv_rows(T* out, int out_stride, const T* x, int x_stride, const float* taps, const float* bias, const float* state,
                     const int* seq_idx, const int* cu_q, const int* slot_ids, int N, int C, int act, int num_slots, int* status,
                     cudaStream_t stream) {
    constexpr int VEC = 4, R = 8;
    return launch_pdl(causal_conv_rows_kernel<T, L, R>, dim3((N + R - 1) / R, (C / VEC + 127) / 128), dim3(128), 0, stream, out, out_stride,
                      x, x_stride, taps, bias, state, seq_idx, cu_q, slot_ids, N, C, act, num_slots, status);
}

// history <- the last L-1 rows of (history ++ the request's rows of this step)
template <typename T>
__global__ void causal_conv_state_kernel(const T* __restrict__ x, int x_stride, float* __restrict__ state,
                                         const int* __restrict__ cu_q, const int* __restrict__ slot_ids, int C, int L,
                                         int num_slots, int* __restrict__ status) {
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= C) return;
    const int start = cu_q[s], n = cu_q[s + 1] - start;
    if (n <= 0) return;
    const int slot = zai_checked_slot(slot_ids[s], num_slots, status);
    float* hist = state + (size_t)slot * (L - 1) * C;
    for (int i = 0; i < L - 1; ++i) {                 // reads run ahead of writes: row n+i > i
        const int src = n + i;
        hist[(size_t)i * C + c] = src < L - 1 ? hist[(size_t)src * C + c]
                                              : to_float(x[(size_t)(start + src - (L - 1)) * x_stride + c]);
    }
}

// every request brings one token: output and history in one pass
template <typename T>
__global__ void causal_conv_single_kernel(T* __restrict__ out, int out_stride, const T* __restrict__ x, int x_stride,
                                          const float* __restrict__ taps, const float* __restrict__ bias,
                                          float* __restrict__ state, const int* __restrict__ slot_ids, int C, int L,
                                          int act, int write_state, int num_slots, int* __restrict__ status) {
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= C) return;
    const int slot = zai_checked_slot(slot_ids[s], num_slots, status);
    float* hist = state + (size_t)slot * (L - 1) * C;
    const float cur = to_float(x[(size_t)s * x_stride + c]);
    float acc = (bias ? bias[c] : 0.f) + taps[(size_t)c * L + (L - 1)] * cur;
    for (int j = 0; j < L - 1; ++j) {
        const float u = hist[(size_t)j * C + c];
        acc += taps[(size_t)c * L + j] * u;
        if (write_state && j > 0) hist[(size_t)(j - 1) * C + c] = u;
    }
    if (write_state && L > 1) hist[(size_t)(L - 2) * C + c] = cur;
    if (act) acc = acc / (1.f + expf(-acc));
    out[(size_t)s * out_stride + c] = from_float<T>(acc);
}

ZAI_API int zai_causal_conv(void* out, int out_stride, const void* x, int x_stride, int dtype, const float* taps,
                            const float* bias, float* state, const int* seq_idx, const int* cu_q, const int* slot_ids,
                            int N, int S, int C, int L, int act, int single_tokens, int write_state, int num_slots,
                            int* status, cudaStream_t stream) {
    if (N <= 0 || C <= 0) return ZAI_OK;
    if (L < 1 || L > ZAI_CONV_MAX_TAPS || C > 65535 * 128) return ZAI_BAD_SIZE;
    const int threads = 128;
    const unsigned cb = (unsigned)((C + threads - 1) / threads);
    if (single_tokens && N == S) {
        ZAI_DISPATCH(dtype, return launch_pdl(causal_conv_single_kernel<T>, dim3(S, cb), dim3(threads), 0, stream, (T*)out,
            out_stride, (const T*)x, x_stride, taps, bias, state, slot_ids, C, L, act, write_state, num_slots, status));
    }
    int rc;
    if (L >= 2 && L <= 4 && C % 4 == 0 && x_stride % 4 == 0 && out_stride % 4 == 0
        && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(taps)) & 15) == 0) {
#define CONV_ROWS(LV) ZAI_DISPATCH(dtype, rc = (conv_rows<T, LV>((T*)out, out_stride, (const T*)x, x_stride, taps, bias, (const float*)state, \
                                                                 seq_idx, cu_q, slot_ids, N, C, act, num_slots, status, stream)))
        if (L == 2) CONV_ROWS(2);
        else if (L == 3) CONV_ROWS(3);
        else CONV_ROWS(4);
#undef CONV_ROWS
    } else
    ZAI_DISPATCH(dtype, rc = launch_pdl(causal_conv_kernel<T>, dim3(N, cb), dim3(threads), 0, stream, (T*)out, out_stride,
        (const T*)x, x_stride, taps, bias, (const float*)state, seq_idx, cu_q, slot_ids, C, L, act, num_slots, status));
    if (rc != 0 || !write_state || L == 1) return rc;
    ZAI_DISPATCH(dtype, return launch_pdl(causal_conv_state_kernel<T>, dim3(S, cb), dim3(threads), 0, stream, (const T*)x,
        x_stride, state, cu_q, slot_ids, C, L, num_slots, status));
}
