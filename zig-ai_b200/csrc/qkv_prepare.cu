// Between a stacked projection and attention, for mixers whose q and k are normed over the whole projection
// or per head, rotated from a table, and whose heads may be wider in the cache than in the projection:
//
//   zai_qkv_prepare     y = [q (Hq D) | k (Hkv D) | v (Hkv Dv) | ...] per row:
//                       q, k <- x * rsqrt(mean(x^2) + eps) * gamma   over the whole of q (of k), per head, or not at all
//                       pairs (x[i], x[i + rot/2]), i < rot/2, of every head turn by the row's (cos, sin) table
//                       q -> [N, Hq, Dp],  k, v -> pages[page(pos), 0|1, kv head, pos % page_size, :Dp]
//                       (Dp >= D, Dv: zeros behind a head's own values; zeros change neither a score nor a sum)
//                       optionally the queries times 1 + coef * ln(floor((pos + 1) / every) + 1), and the cached values
//                       (1 - lambda) v + lambda v_first with an earlier layer's values of the same rows
//   zai_latent_prepare  the rotated parts of the queries of latent attention, and per row the normed latent and the
//                       rotated shared key part into pages[page(pos), pos % page_size, :rank + rot]
//   zai_sigmoid_gate    out = o * sigmoid(gate), the gate one number per head or per element
//
// Norms, rotations and sigmoids are 32-bit; what is stored is rounded once to the model's dtype.  One block per row;
// the order of every reduction depends only on the sizes, so a row's result does not depend on its batch.
#include "common.cuh"

template <typename T>
__global__ void __launch_bounds__(256) qkv_prepare_kernel(
    const T* __restrict__ y, int y_stride, const float* __restrict__ q_gamma, const float* __restrict__ k_gamma, float eps,
    int scope, const float2* __restrict__ cs_table, int rot, const int* __restrict__ positions, const int* __restrict__ seq_idx,
    const int* __restrict__ block_table, int table_width, T* __restrict__ pages, int page_size, T* __restrict__ q_out,
    int Hq, int Hkv, int D, int Dv, int Dp, int write, int num_pages, int* __restrict__ status, float temp_coef, int temp_every,
    const T* __restrict__ v_first, int v_first_stride, const float* __restrict__ v_lambda) {
    extern __shared__ float smem[];
    __shared__ float red[33];
    const int half = rot / 2;
    const int nq = Hq * D, nk = Hkv * D;
    float* buf = smem;                      // [nq + nk] q then k, 32-bit
    float* cs = smem + nq + nk;             // [half] cos
    float* sn = cs + half;                  // [half] sin
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarp = blockDim.x >> 5;
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const T* row = y + (size_t)t * y_stride;
    for (int i = tid; i < half; i += blockDim.x) {
        const float2 v = cs_table[(size_t)t * half + i];
        cs[i] = v.x;
        sn[i] = v.y;
    }
    float sq = 0.f, sk = 0.f;
    for (int i = tid; i < nq + nk; i += blockDim.x) {
        const float v = to_float(row[i]);
        buf[i] = v;
        if (i < nq) sq += v * v; else sk += v * v;
    }
    if (scope == 2) {
        const float inv_q = rsqrtf(block_sum(sq, red) / (float)nq + eps);
        const float inv_k = rsqrtf(block_sum(sk, red) / (float)nk + eps);
        for (int i = tid; i < nq + nk; i += blockDim.x)
            buf[i] *= i < nq ? inv_q * q_gamma[i] : inv_k * k_gamma[i - nq];
    } else if (scope == 1) {
        __syncthreads();
        for (int h = warp; h < Hq + Hkv; h += nwarp) {
            float* x = buf + (size_t)h * D;
            const float* gamma = h < Hq ? q_gamma : k_gamma;
            float ss = 0.f;
            for (int d = lane; d < D; d += 32) ss += x[d] * x[d];
            const float inv = rsqrtf(warp_sum(ss) / (float)D + eps);
            for (int d = lane; d < D; d += 32) x[d] *= inv * gamma[d];
        }
    }
    __syncthreads();
    // rotated (or passed through) and padded to Dp: element d of head h
    auto turned = [&](const float* x, int d) -> float {
        if (d < half) return x[d] * cs[d] - x[d + half] * sn[d];
        if (d < rot) return x[d - half] * sn[d - half] + x[d] * cs[d - half];
        return d < D ? x[d] : 0.f;
    };
    const int pos = positions[t];
    // the queries' temperature: 1 + coef * ln(floor((pos + 1) / every) + 1), a step function of the position
    const float temp = temp_every > 0 ? 1.f + temp_coef * logf((float)((pos < 0 ? 0 : pos + 1) / temp_every + 1)) : 1.f;
    T* qrow = q_out + (size_t)t * Hq * Dp;
    for (int i = tid; i < Hq * Dp; i += blockDim.x) {
        const int h = i / Dp, d = i - h * Dp;
        qrow[i] = from_float<T>(turned(buf + (size_t)h * D, d) * temp);
    }
    if (!write) return;
    const int page = zai_checked_page(block_table + (size_t)seq_idx[t] * table_width, table_width,
                                      pos < 0 ? -1 : pos / page_size, num_pages, status);
    const int off = pos < 0 ? 0 : pos % page_size;
    T* kpage = pages + (size_t)page * 2 * Hkv * page_size * Dp;
    T* vpage = kpage + (size_t)Hkv * page_size * Dp;
    const T* vrow = row + nq + nk;
    // values mixed with an earlier layer's values of the same token: (1 - lambda) v + lambda v_first, in 32-bit
    const T* frow = v_first ? v_first + (size_t)t * v_first_stride : nullptr;
    const float lam = frow ? v_lambda[0] : 0.f;
    for (int i = tid; i < Hkv * Dp; i += blockDim.x) {
        const int g = i / Dp, d = i - g * Dp;
        const size_t at = ((size_t)g * page_size + off) * Dp + d;
        kpage[at] = from_float<T>(turned(buf + nq + (size_t)g * D, d));
        if (d >= Dv) vpage[at] = from_float<T>(0.f);
        else if (!frow) vpage[at] = vrow[(size_t)g * Dv + d];
        else vpage[at] = from_float<T>((1.f - lam) * to_float(vrow[(size_t)g * Dv + d]) + lam * to_float(frow[(size_t)g * Dv + d]));
    }
}

// The same work for bfloat16 heads of multiples of eight values (norm per head or none): eight lanes' worth of a head's row a
// time, `lanes` (a power of two) neighbouring lanes a head, eight values a lane, each in registers from the projection's row to
// the page; a row's heads of q, k and v are independent items.  A rotated pair's other half comes from the lane that holds it.
__device__ __forceinline__ void prep_load8(float (&v)[8], const bf16* p) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x; v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void prep_store8(bf16* p, const float (&v)[8]) {
    uint4 u;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = u;
}
__global__ void __launch_bounds__(256) qkv_prepare_heads_kernel(
    const bf16* __restrict__ y, int y_stride, const float* __restrict__ q_gamma, const float* __restrict__ k_gamma, float eps,
    const float2* __restrict__ cs_table, int rot, const int* __restrict__ positions, const int* __restrict__ seq_idx,
    const int* __restrict__ block_table, int table_width, bf16* __restrict__ pages, int page_size, bf16* __restrict__ q_out, int N,
    int Hq, int Hkv, int D, int Dv, int Dp, int write, int num_pages, int* __restrict__ status, float temp_coef, int temp_every,
    const bf16* __restrict__ v_first, int v_first_stride, const float* __restrict__ v_lambda, int lanes) {
    pdl_trigger();
    pdl_wait();
    const unsigned heads = Hq + (write ? 2 * Hkv : 0), per_block = blockDim.x / lanes;
    const unsigned item = blockIdx.x * per_block + threadIdx.x / lanes;
    const bool live = item < (unsigned)N * heads;                        // (whole groups of lanes; all lanes stay for the exchanges)
    const unsigned t = live ? item / heads : 0, hh = live ? item - t * heads : 0;
    const int sub = threadIdx.x & (lanes - 1), d = sub * 8, half = rot / 2;
    const int kind = hh < (unsigned)Hq ? 0 : hh < (unsigned)(Hq + Hkv) ? 1 : 2, h = hh - (kind == 0 ? 0 : kind == 1 ? Hq : Hq + Hkv);
    const int own = kind == 2 ? Dv : D;
    const bf16* src = y + (size_t)t * y_stride + (kind == 0 ? (size_t)h * D : (size_t)Hq * D + (kind == 1 ? (size_t)h * D : (size_t)Hkv * D + (size_t)h * Dv));
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    const bool mine = live && d < own;
    if (mine) prep_load8(v, src + d);
    const int pos = positions[t];
    const float* gamma = kind == 0 ? q_gamma : k_gamma;
    if (gamma) {                                                         // (uniform over the launch; values' lanes discard it)
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) ss += v[i] * v[i];
        for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (mine && kind != 2) {
            const float inv = rsqrtf(ss / (float)D + eps);
            const float4 ga = *reinterpret_cast<const float4*>(gamma + d), gb = *reinterpret_cast<const float4*>(gamma + d + 4);
            v[0] *= inv * ga.x; v[1] *= inv * ga.y; v[2] *= inv * ga.z; v[3] *= inv * ga.w;
            v[4] *= inv * gb.x; v[5] *= inv * gb.y; v[6] *= inv * gb.z; v[7] *= inv * gb.w;
        }
    }
    if (rot) {
        const bool low = d < half;
        const int base = (threadIdx.x & 31) & ~(lanes - 1), other = base + ((sub + (low ? half / 8 : -(half / 8))) & (lanes - 1));
        float w[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) w[i] = __shfl_sync(0xffffffffu, v[i], other);
        if (mine && kind != 2 && d < rot) {
            const float2* cs = cs_table + (size_t)t * half + (low ? d : d - half);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float2 c = cs[i];
                v[i] = low ? v[i] * c.x - w[i] * c.y : w[i] * c.y + v[i] * c.x;
            }
        }
    }
    if (!live || d >= Dp) return;
    if (kind == 0) {
        if (temp_every > 0) {
            const float temp = 1.f + temp_coef * logf((float)((pos < 0 ? 0 : pos + 1) / temp_every + 1));
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] *= temp;
        }
        prep_store8(q_out + ((size_t)t * Hq + h) * Dp + d, v);
        return;
    }
    if (kind == 2 && v_first && mine) {
        float f[8];
        prep_load8(f, v_first + (size_t)t * v_first_stride + (size_t)h * Dv + d);
        const float lam = v_lambda[0];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = (1.f - lam) * v[i] + lam * f[i];
    }
    const int page = zai_checked_page(block_table + (size_t)seq_idx[t] * table_width, table_width, pos < 0 ? -1 : pos / page_size, num_pages,
                                      status);
    const int off = pos < 0 ? 0 : pos % page_size;
    prep_store8(pages + (((size_t)page * 2 * Hkv + (kind == 1 ? 0 : Hkv) + h) * page_size + off) * Dp + d, v);
}

ZAI_API int zai_qkv_prepare(const void* y, int y_stride, int dtype, const float* q_gamma, const float* k_gamma, float eps, int scope,
                            const float2* cs_table, int rot, const int* positions, const int* seq_idx, const int* block_table,
                            int table_width, void* pages, int page_size, void* q_out, int N, int Hq, int Hkv, int D, int Dv,
                            int Dp, int write, int num_pages, int* status, float temp_coef, int temp_every, const void* v_first,
                            int v_first_stride, const float* v_lambda, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    if (Hq < 1 || Hkv < 1 || D < 1 || Dv < 1 || Dp < D || Dp < Dv || rot < 0 || rot > D || rot % 2 || scope < 0 || scope > 2
        || (scope && (!q_gamma || !k_gamma)) || (rot && !cs_table) || temp_every < 0 || (v_first && !v_lambda))
        return ZAI_BAD_SIZE;
    const uintptr_t at = reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(pages) | reinterpret_cast<uintptr_t>(q_out) |
                         reinterpret_cast<uintptr_t>(v_first) | reinterpret_cast<uintptr_t>(q_gamma) | reinterpret_cast<uintptr_t>(k_gamma);
    if (dtype == ZAI_BF16 && scope < 2 && ((D | Dv | Dp | y_stride | v_first_stride) & 7) == 0 && rot % 16 == 0 && Dp <= 256 && (at & 15) == 0
        && (long long)N * (Hq + 2 * Hkv) < (1 << 30)) {
        int lanes = 1;
        while (lanes * 8 < Dp) lanes *= 2;
        const long long items = (long long)N * (Hq + (write ? 2 * Hkv : 0));
        const int per_block = 256 / lanes;
        return launch_pdl(qkv_prepare_heads_kernel, dim3((unsigned)((items + per_block - 1) / per_block)), dim3(256), 0, stream, (const bf16*)y,
                          y_stride, scope ? q_gamma : nullptr, scope ? k_gamma : nullptr, eps, cs_table, rot, positions, seq_idx, block_table,
                          table_width, (bf16*)pages, page_size, (bf16*)q_out, N, Hq, Hkv, D, Dv, Dp, write, num_pages, status, temp_coef,
                          temp_every, (const bf16*)v_first, v_first_stride, v_lambda, lanes);
    }
    const size_t smem = ((size_t)(Hq + Hkv) * D + rot) * sizeof(float);
    if (smem > 200 * 1024) return ZAI_BAD_SIZE;
    static unsigned long long done_f32 = 0, done_bf16 = 0;
    if (smem > 48 * 1024) {
        if (dtype == ZAI_F32 && zai_first_on_device(&done_f32))
            cudaFuncSetAttribute(qkv_prepare_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (dtype == ZAI_BF16 && zai_first_on_device(&done_bf16))
            cudaFuncSetAttribute(qkv_prepare_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    }
    ZAI_DISPATCH(dtype, return launch_pdl(qkv_prepare_kernel<T>, dim3(N), dim3(256), smem, stream, (const T*)y, y_stride, q_gamma,
                                          k_gamma, eps, scope, cs_table, rot, positions, seq_idx, block_table, table_width, (T*)pages,
                                          page_size, (T*)q_out, Hq, Hkv, D, Dv, Dp, write, num_pages, status, temp_coef, temp_every,
                                          (const T*)v_first, v_first_stride, v_lambda));
    return launch_status();
}

// q [N, H, D + Dr] (row stride q_stride): its rotated parts -> q_rot [N, H, Dr].  dkv [N, R + Dr] (row stride dkv_stride, may be
// null): c = rms(dkv[:R]) * gamma, r = rotate(dkv[R:]) -> pages[page(pos), pos % page_size, :R + Dr].
template <typename T>
__global__ void __launch_bounds__(256) latent_prepare_kernel(
    const T* __restrict__ q, int q_stride, const T* __restrict__ dkv, int dkv_stride, const float* __restrict__ gamma, float eps,
    const float2* __restrict__ cs_table, const int* __restrict__ positions, const int* __restrict__ seq_idx,
    const int* __restrict__ block_table, int table_width, T* __restrict__ pages, int page_size, T* __restrict__ q_rot,
    int H, int D, int Dr, int R, int num_pages, int* __restrict__ status) {
    extern __shared__ float smem[];
    __shared__ float red[33];
    const int half = Dr / 2;
    float* cs = smem;                       // [half]
    float* sn = smem + half;                // [half]
    const int tid = threadIdx.x;
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    for (int i = tid; i < half; i += blockDim.x) {
        const float2 v = cs_table[(size_t)t * half + i];
        cs[i] = v.x;
        sn[i] = v.y;
    }
    __syncthreads();
    const T* qrow = q + (size_t)t * q_stride;
    T* orow = q_rot + (size_t)t * H * Dr;
    for (int i = tid; i < H * half; i += blockDim.x) {
        const int h = i / half, d = i - h * half;
        const T* x = qrow + (size_t)h * (D + Dr) + D;
        const float a = to_float(x[d]), b = to_float(x[d + half]);
        orow[(size_t)h * Dr + d] = from_float<T>(a * cs[d] - b * sn[d]);
        orow[(size_t)h * Dr + d + half] = from_float<T>(b * cs[d] + a * sn[d]);
    }
    if (!dkv) return;
    const T* drow = dkv + (size_t)t * dkv_stride;
    float ss = 0.f;
    for (int i = tid; i < R; i += blockDim.x) {
        const float v = to_float(drow[i]);
        ss += v * v;
    }
    const float inv = rsqrtf(block_sum(ss, red) / (float)R + eps);
    const int pos = positions[t];
    const int page = zai_checked_page(block_table + (size_t)seq_idx[t] * table_width, table_width,
                                      pos < 0 ? -1 : pos / page_size, num_pages, status);
    const int off = pos < 0 ? 0 : pos % page_size;
    T* dst = pages + ((size_t)page * page_size + off) * (R + Dr);
    for (int i = tid; i < R; i += blockDim.x) dst[i] = from_float<T>(to_float(drow[i]) * inv * gamma[i]);
    for (int d = tid; d < half; d += blockDim.x) {
        const float a = to_float(drow[R + d]), b = to_float(drow[R + d + half]);
        dst[R + d] = from_float<T>(a * cs[d] - b * sn[d]);
        dst[R + d + half] = from_float<T>(b * cs[d] + a * sn[d]);
    }
}

ZAI_API int zai_latent_prepare(const void* q, int q_stride, const void* dkv, int dkv_stride, int dtype, const float* gamma, float eps,
                               const float2* cs_table, const int* positions, const int* seq_idx, const int* block_table,
                               int table_width, void* pages, int page_size, void* q_rot, int N, int H, int D, int Dr, int R,
                               int num_pages, int* status, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    if (H < 1 || D < 0 || Dr < 2 || Dr % 2 || R < 1 || !cs_table || (dkv && !gamma) || Dr > 8192) return ZAI_BAD_SIZE;
    ZAI_DISPATCH(dtype, return launch_pdl(latent_prepare_kernel<T>, dim3(N), dim3(256), (size_t)Dr * sizeof(float), stream,
                                          (const T*)q, q_stride, (const T*)dkv, dkv_stride, gamma, eps, cs_table, positions, seq_idx,
                                          block_table, table_width, (T*)pages, page_size, (T*)q_rot, H, D, Dr, R, num_pages, status));
    return launch_status();
}

// out[n, h, d] = in[n * in_row + h * in_head + d] * sigmoid(gate[n * gate_stride + (per_head ? h : h * Dh + d)])
template <typename T>
__global__ void sigmoid_gate_kernel(T* __restrict__ out, const T* __restrict__ in, long long in_row, long long in_head,
                                    const T* __restrict__ gate, int gate_stride, int per_head, long long total, int H, int Dh) {
    pdl_trigger();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const int d = (int)(i % Dh);
    const long long nh = i / Dh;
    const int h = (int)(nh % H);
    const long long n = nh / H;
    const float g = to_float(gate[n * gate_stride + (per_head ? h : h * Dh + d)]);
    const float v = to_float(in[n * in_row + h * in_head + d]);
    out[i] = from_float<T>(v / (1.f + expf(-g)));
}

// The same for bfloat16 heads of a multiple of eight values on 16-byte boundaries: eight values a thread.
__global__ void __launch_bounds__(256) sigmoid_gate_bf16x8_kernel(bf16* __restrict__ out, const bf16* __restrict__ in, int in_row, int in_head,
                                                                  const bf16* __restrict__ gate, int gate_stride, int per_head, unsigned total8,
                                                                  unsigned H, unsigned Dh8) {
    pdl_trigger();
    pdl_wait();
    const unsigned i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total8) return;
    const unsigned nh = i / Dh8, d = (i - nh * Dh8) * 8, n = nh / H, h = nh - n * H;
    const uint4 v4 = *reinterpret_cast<const uint4*>(in + (size_t)n * in_row + (size_t)h * in_head + d);
    const __nv_bfloat162* vp = reinterpret_cast<const __nv_bfloat162*>(&v4);
    const bf16* gp = gate + (size_t)n * gate_stride + (per_head ? h : h * Dh8 * 8 + d);
    uint4 o4;
    __nv_bfloat162* op = reinterpret_cast<__nv_bfloat162*>(&o4);
    const float one = per_head ? 1.f + expf(-__bfloat162float(gp[0])) : 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const float2 v = __bfloat1622float2(vp[j]);
        const float g0 = per_head ? one : 1.f + expf(-__bfloat162float(gp[2 * j]));
        const float g1 = per_head ? one : 1.f + expf(-__bfloat162float(gp[2 * j + 1]));
        op[j] = __floats2bfloat162_rn(v.x / g0, v.y / g1);
    }
    *reinterpret_cast<uint4*>(out + (size_t)i * 8) = o4;
}

ZAI_API int zai_sigmoid_gate(void* out, const void* in, long long in_row, long long in_head, const void* gate, int gate_stride,
                             int dtype, int per_head, int N, int H, int Dh, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    if (H < 1 || Dh < 1) return ZAI_BAD_SIZE;
    const long long total = (long long)N * H * Dh;
    if (dtype == ZAI_BF16 && Dh % 8 == 0 && in_row % 8 == 0 && in_head % 8 == 0 && in_row < (1 << 30) && total / 8 < (1u << 31)
        && ((reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(in)) & 15) == 0)
        return launch_pdl(sigmoid_gate_bf16x8_kernel, dim3((unsigned)((total / 8 + 255) / 256)), dim3(256), 0, stream, (bf16*)out, (const bf16*)in,
                          (int)in_row, (int)in_head, (const bf16*)gate, gate_stride, per_head, (unsigned)(total / 8), (unsigned)H,
                          (unsigned)(Dh / 8));
    const unsigned blocks = (unsigned)((total + 255) / 256);
    ZAI_DISPATCH(dtype, return launch_pdl(sigmoid_gate_kernel<T>, dim3(blocks), dim3(256), 0, stream, (T*)out, (const T*)in, in_row,
                                          in_head, (const T*)gate, gate_stride, per_head, total, H, Dh));
    return launch_status();
}
