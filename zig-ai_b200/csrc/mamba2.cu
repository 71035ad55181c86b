// The state-space recurrence with one decay per head (Mamba-2, state-space duality), per request and head:
//
//   d_t = softplus(dt_t + bias),   S_t = exp(a d_t) S_(t-1) + d_t B_t x_t^T,   a = -exp(A_log)
//   y_t = S_t^T C_t + D x_t                                S [N, V], x and y [V], B and C [N] shared by a group of heads
//   out = parts of (y silu(z)) divided by their root mean square, times a weight
//
// x, B and C come out of a short causal convolution; the state [heads, N, V] and the convolution's history are the request's,
// 32-bit, zero for a new request.  Step sizes, decays, the state, its sums and the norm are 32-bit in both modes.
//
// Three ways through the rows of a step, which differ by rounding only:
//   * `mamba2_scan_kernel`: a block walks the rows of one request for one head and 32 columns of S in order; a warp holds 32
//     rows of S (a lane a column) in registers, the warps' sums over N are added per tile of rows.  Any sizes, both modes:
//     the 32-bit mode and the short spans of the bfloat16 mode.
//   * chunks of 64 rows on the tensor cores (bfloat16 mode, spans of MAMBA2_CHUNKED_MIN rows or more).  With
//     L_i = a sum_{k <= i} d_k inside a chunk:
//       pass 1   E = sum_j exp(L_last - L_j) d_j B_j x_j^T for every chunk at once
//       pass 2   S <- exp(L_last) S + E across the chunks of a request, E replaced by the state before its chunk
//       pass 3   y_i = exp(L_i) S^T C_i + sum_{j <= i} exp(L_i - L_j) d_j (C_i . B_j) x_j + D x_i for every chunk at once
//     x, B and C are bfloat16 and go into the products as they are; what is 32-bit (the weighted x, the state, the weighted
//     scores) goes in as a sum of three bfloat16 numbers, which hold its 24 bits, with 32-bit accumulation.
//   * `mamba2_single_kernel`: every request brings one token.  The convolution, the step size, the state's update and the
//     read-out in one kernel that streams the state through the SMs once; the norm's kernel behind it moves the history.
#include "mma_helpers.cuh"

#define M2_Q 64                     // rows of a chunk
#define M2_PAD 8                    // bfloat16 values behind every row in shared memory (no bank conflicts for ldmatrix)
#define M2_TT 16                    // rows that the scan stages at a time
#define MAMBA2_MAX_STATE 512
#define M2_MAX_TAPS 16

__device__ __forceinline__ float m2_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float m2_silu(float x) { return x / (1.f + expf(-x)); }

struct Mamba2Args {
    const void* u;                  // [N rows, u_stride]: x | B | C after the convolution
    int u_stride;
    const void* dt;                 // [N rows, dt_stride]: the heads' raw step sizes
    int dt_stride;
    const float *dt_bias, *a_log, *skip;
    float* out;                     // [N rows, H V] 32-bit
    float* state;                   // [num_slots, H, N, V]
    const int *cu_q, *slot_ids;
    int* status;
    int num_slots, n_seqs, H, G, N, V, write_state;
    int min_rows, max_rows;         // spans with fewer or more rows are another kernel's
};

// ------------------------------------------------------------------------------------------------ the walk
template <typename T>
__global__ void __launch_bounds__(512) mamba2_scan_kernel(const Mamba2Args a) {
    extern __shared__ __align__(16) float m2_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5, np = nw * 32;
    float* sB = m2_smem;                         // [TT][np]
    float* sC = sB + M2_TT * np;                 // [TT][np]
    float* part = sC + M2_TT * np;               // [TT][nw][32]
    float* sx = part + M2_TT * nw * 32;          // [TT][32]
    float* sd = sx + M2_TT * 32;                 // [TT][2]: decay, step size
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y, v = blockIdx.z * 32 + lane, g = h / (a.H / a.G);
    const int r0 = a.cu_q[s], r1 = a.cu_q[s + 1];
    if (r1 - r0 < a.min_rows || r1 - r0 > a.max_rows || r1 <= r0) return;
    const T* u = (const T*)a.u;
    const T* dt = (const T*)a.dt;
    const int b_at = a.H * a.V + g * a.N, c_at = a.H * a.V + (a.G + g) * a.N;
    const float neg_a = -expf(a.a_log[h]), bias = a.dt_bias[h], skip = a.skip[h];
    const int slot = zai_checked_slot(a.slot_ids[s], a.num_slots, a.status);
    float* st = a.state + ((size_t)slot * a.H + h) * a.N * a.V;
    const int n0 = warp * 32;
    float S[32];
#pragma unroll
    for (int k = 0; k < 32; ++k) S[k] = (v < a.V && n0 + k < a.N) ? st[(size_t)(n0 + k) * a.V + v] : 0.f;
    for (int t0 = r0; t0 < r1; t0 += M2_TT) {
        const int nt = min(M2_TT, r1 - t0);
        __syncthreads();                         // the tile before has been walked and written
        for (int i = threadIdx.x; i < M2_TT * np; i += blockDim.x) {
            const int tt = i / np, n = i % np;
            const bool ok = tt < nt && n < a.N;
            sB[i] = ok ? to_float(u[(size_t)(t0 + tt) * a.u_stride + b_at + n]) : 0.f;
            sC[i] = ok ? to_float(u[(size_t)(t0 + tt) * a.u_stride + c_at + n]) : 0.f;
        }
        for (int i = threadIdx.x; i < M2_TT * 32; i += blockDim.x) {
            const int tt = i >> 5, c = blockIdx.z * 32 + (i & 31);
            sx[i] = (tt < nt && c < a.V) ? to_float(u[(size_t)(t0 + tt) * a.u_stride + h * a.V + c]) : 0.f;
        }
        if (threadIdx.x < nt) {
            const float d = m2_softplus(to_float(dt[(size_t)(t0 + threadIdx.x) * a.dt_stride + h]) + bias);
            sd[2 * threadIdx.x] = expf(neg_a * d);
            sd[2 * threadIdx.x + 1] = d;
        }
        __syncthreads();
        for (int tt = 0; tt < nt; ++tt) {
            const float keep = sd[2 * tt], take = sd[2 * tt + 1] * sx[tt * 32 + lane];
            const float* b = sB + tt * np + n0;
            const float* c = sC + tt * np + n0;
            float y0 = 0.f, y1 = 0.f, y2 = 0.f, y3 = 0.f;
#pragma unroll
            for (int k = 0; k < 32; k += 4) {
                const float4 b4 = *reinterpret_cast<const float4*>(b + k), c4 = *reinterpret_cast<const float4*>(c + k);
                S[k] = fmaf(keep, S[k], take * b4.x);
                S[k + 1] = fmaf(keep, S[k + 1], take * b4.y);
                S[k + 2] = fmaf(keep, S[k + 2], take * b4.z);
                S[k + 3] = fmaf(keep, S[k + 3], take * b4.w);
                y0 = fmaf(S[k], c4.x, y0);
                y1 = fmaf(S[k + 1], c4.y, y1);
                y2 = fmaf(S[k + 2], c4.z, y2);
                y3 = fmaf(S[k + 3], c4.w, y3);
            }
            part[(tt * nw + warp) * 32 + lane] = (y0 + y1) + (y2 + y3);
        }
        __syncthreads();
        for (int i = threadIdx.x; i < nt * 32; i += blockDim.x) {
            const int tt = i >> 5, c = blockIdx.z * 32 + (i & 31);
            if (c >= a.V) continue;
            float y = 0.f;
            for (int w = 0; w < nw; ++w) y += part[(tt * nw + w) * 32 + (i & 31)];
            a.out[((size_t)(t0 + tt) * a.H + h) * a.V + c] = fmaf(skip, sx[i], y);
        }
    }
    if (a.write_state && v < a.V) {
#pragma unroll
        for (int k = 0; k < 32; ++k)
            if (n0 + k < a.N) st[(size_t)(n0 + k) * a.V + v] = S[k];
    }
}

// ------------------------------------------------------------------------------------------------ chunks
// Chunk b among all chunks of the step: the spans of min_rows rows or more in order, each cut into chunks of M2_Q rows.
__device__ __forceinline__ bool m2_find_chunk(const Mamba2Args& a, int b, int& seq, int& t0, int& t1) {
    int seen = 0;
    for (int s = 0; s < a.n_seqs; ++s) {
        const int lo = a.cu_q[s], hi = a.cu_q[s + 1];
        if (hi - lo < a.min_rows || hi <= lo) continue;
        const int n = (hi - lo + M2_Q - 1) / M2_Q;
        if (b < seen + n) {
            seq = s;
            t0 = lo + (b - seen) * M2_Q;
            t1 = min(t0 + M2_Q, hi);
            return true;
        }
        seen += n;
    }
    return false;
}

// The chunk's step sizes d_j and the running sums L_j of a d, in units of ln 2 (both 64 values; rows beyond the chunk have
// d = 0), by the first 64 threads of the block; everyone calls it.  The sums are made in 64-bit and kept as two 32-bit numbers
// each, so that a difference of two of them is good to the last bits whatever the chunk's rows before it have summed up to.
__device__ __forceinline__ void m2_decays(const Mamba2Args& a, int h, int t0, int t1, float* s_d, float2* s_l, double* s_carry) {
    const int j = threadIdx.x, lane = threadIdx.x & 31;
    double l = 0.0;
    if (j < M2_Q) {
        float d = 0.f;
        if (t0 + j < t1) d = m2_softplus(to_float(((const bf16*)a.dt)[(size_t)(t0 + j) * a.dt_stride + h]) + a.dt_bias[h]);
        s_d[j] = d;
        l = -1.4426950408889634 * (double)(expf(a.a_log[h]) * d);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, l, o);
            if (lane >= o) l += up;
        }
        if (j == 31) *s_carry = l;
    }
    __syncthreads();
    if (j < M2_Q) {
        if (j >= 32) l += *s_carry;
        const float hi = (float)l;
        s_l[j] = make_float2(hi, (float)(l - (double)hi));
    }
    __syncthreads();
}
__device__ __forceinline__ float m2_between(float2 later, float2 earlier) { return (later.x - earlier.x) + (later.y - earlier.y); }

// rows t0.. of a column slice of u into shared memory [M2_Q][ld] (zeros beyond the chunk and beyond `cols` up to `cols_p`)
__device__ __forceinline__ void m2_load_rows(bf16* dst, int ld, const Mamba2Args& a, int at, int cols, int cols_p, int t0, int t1) {
    const bf16* u = (const bf16*)a.u;
    const bool vec = ((cols | at | a.u_stride) & 7) == 0 && (reinterpret_cast<uintptr_t>(u) & 15) == 0;
    if (vec) {
        const int per = cols_p >> 3;
        for (int i = threadIdx.x; i < M2_Q * per; i += blockDim.x) {
            const int r = i / per, c = (i % per) * 8;
            const bool ok = t0 + r < t1 && c < cols;
            cp_async16(dst + r * ld + c, u + (ok ? (size_t)(t0 + r) * a.u_stride + at + c : 0), ok);
        }
    } else {
        for (int i = threadIdx.x; i < M2_Q * cols_p; i += blockDim.x) {
            const int r = i / cols_p, c = i % cols_p;
            dst[r * ld + c] = (t0 + r < t1 && c < cols) ? u[(size_t)(t0 + r) * a.u_stride + at + c] : __float2bfloat16_rn(0.f);
        }
    }
}

// v as a sum of three bfloat16 numbers
__device__ __forceinline__ void m2_split(float v, float& hi, float& mid, float& lo) {
    hi = __bfloat162float(__float2bfloat16_rn(v));
    const float r = v - hi;
    mid = __bfloat162float(__float2bfloat16_rn(r));
    lo = r - mid;
}
// two neighbouring values, each split: p[k] holds the k-th parts
__device__ __forceinline__ void m2_split2(float v0, float v1, uint32_t (&p)[3]) {
    float a0, a1, a2, b0, b1, b2;
    m2_split(v0, a0, a1, a2);
    m2_split(v1, b0, b1, b2);
    p[0] = pack_bf16(a0, b0);
    p[1] = pack_bf16(a1, b1);
    p[2] = pack_bf16(a2, b2);
}

// pass 1: ends [chunk, H, N, V] and last [chunk, H] (the chunk's L_last).  VT columns of V a block; eight warps, each in turn
// 16 states x 32 columns.
template <int VT>
__global__ void __launch_bounds__(256) mamba2_chunk_state_kernel(const Mamba2Args a, float* __restrict__ ends, float* __restrict__ last) {
    extern __shared__ __align__(16) unsigned char m2_raw[];
    __shared__ float s_d[M2_Q], s_w[M2_Q];
    __shared__ float2 s_l[M2_Q];
    __shared__ double s_carry;
    constexpr int LDX = VT + M2_PAD, VW = 32, VG = VT / VW;
    const int np = (a.N + 15) & ~15, ldb = np + M2_PAD;
    bf16* sb = reinterpret_cast<bf16*>(m2_raw);              // [Q][ldb]
    bf16* sx = sb + M2_Q * ldb;                              // [3][Q][LDX]
    pdl_trigger();
    pdl_wait();
    int seq, t0, t1;
    if (!m2_find_chunk(a, blockIdx.x, seq, t0, t1)) return;
    const int h = blockIdx.y, g = h / (a.H / a.G), v0 = blockIdx.z * VT, nv = min(VT, a.V - v0);
    m2_load_rows(sx, LDX, a, h * a.V + v0, nv, VT, t0, t1);
    cp_async_commit();
    m2_load_rows(sb, ldb, a, a.H * a.V + g * a.N, a.N, np, t0, t1);
    cp_async_commit();
    m2_decays(a, h, t0, t1, s_d, s_l, &s_carry);
    if (threadIdx.x < M2_Q) s_w[threadIdx.x] = exp2f(m2_between(s_l[M2_Q - 1], s_l[threadIdx.x])) * s_d[threadIdx.x];
    if (threadIdx.x == 0 && v0 == 0) last[(size_t)blockIdx.x * a.H + h] = s_l[M2_Q - 1].x;
    cp_async_wait<1>();
    __syncthreads();
#pragma unroll
    for (int i = threadIdx.x; i < M2_Q * VT / 2; i += 256) {
        const int j = i / (VT / 2), c = (i % (VT / 2)) * 2;
        uint32_t* p = reinterpret_cast<uint32_t*>(sx + j * LDX + c);
        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
        const float w = s_w[j];
        uint32_t q[3];
        m2_split2(x.x * w, x.y * w, q);
        p[0] = q[0];
        p[M2_Q * LDX / 2] = q[1];
        p[M2_Q * LDX] = q[2];
    }
    cp_async_wait<0>();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mi = lane >> 3, r8 = lane & 7;
    float* e = ends + ((size_t)blockIdx.x * a.H + h) * a.N * a.V;
    for (int item = warp; item < np / 16 * VG; item += 8) {
        const int mt = item / VG, vb = (item % VG) * VW;
        float acc[VW / 8][4];
#pragma unroll
        for (int i = 0; i < VW / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < M2_Q / 16; ++ks) {
            uint32_t fa[4];
            ldmatrix_x4_trans(fa, sb + (ks * 16 + (mi >> 1) * 8 + r8) * ldb + mt * 16 + (mi & 1) * 8);
#pragma unroll
            for (int p = 2; p >= 0; --p) {                   // the small parts first
#pragma unroll
                for (int vp = 0; vp < VW / 16; ++vp) {
                    uint32_t fb[4];
                    ldmatrix_x4_trans(fb, sx + (p * M2_Q + ks * 16 + (mi & 1) * 8 + r8) * LDX + vb + vp * 16 + (mi >> 1) * 8);
                    mma_bf16(acc[2 * vp], fa, fb[0], fb[1]);
                    mma_bf16(acc[2 * vp + 1], fa, fb[2], fb[3]);
                }
            }
        }
        const int n = mt * 16 + (lane >> 2), tq = lane & 3;
        const bool even = ((a.V | v0) & 1) == 0;
#pragma unroll
        for (int i = 0; i < VW / 8; ++i) {
            const int c = vb + i * 8 + 2 * tq;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int nn = n + 8 * half;
                if (nn >= a.N || c >= nv) continue;
                float* p = e + (size_t)nn * a.V + v0 + c;
                if (even && c + 1 < nv) *reinterpret_cast<float2*>(p) = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
                else { p[0] = acc[i][2 * half]; if (c + 1 < nv) p[1] = acc[i][2 * half + 1]; }
            }
        }
    }
}

// pass 2: a thread carries VEC elements of the state across every chunk of a request (blockIdx.y)
template <int VEC>
__global__ void __launch_bounds__(128) mamba2_state_pass_kernel(const Mamba2Args a, float* __restrict__ ends, const float* __restrict__ last) {
    constexpr int AHEAD = 8;                                 // chunks whose loads are in flight
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.y;
    const int rows = a.cu_q[s + 1] - a.cu_q[s];
    if (rows < a.min_rows || rows <= 0) return;
    int c0 = 0;
    for (int q = 0; q < s; ++q) {
        const int n = a.cu_q[q + 1] - a.cu_q[q];
        if (n >= a.min_rows && n > 0) c0 += (n + M2_Q - 1) / M2_Q;
    }
    const int nc = (rows + M2_Q - 1) / M2_Q;
    const size_t NV = (size_t)a.N * a.V, HNV = NV * a.H;
    const size_t idx = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (idx >= HNV) return;
    const int h = (int)(idx / NV);
    const int slot = zai_checked_slot(a.slot_ids[s], a.num_slots, a.status);
    float* st = a.state + (size_t)slot * HNV + idx;
    float S[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) S[k] = st[k];
    for (int c = 0; c < nc; c += AHEAD) {
        float e[AHEAD][VEC], l[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (c + i >= nc) continue;
            const float* p = ends + (size_t)(c0 + c + i) * HNV + idx;
            if constexpr (VEC == 4) {
                const float4 v = *reinterpret_cast<const float4*>(p);
                e[i][0] = v.x; e[i][1] = v.y; e[i][2] = v.z; e[i][3] = v.w;
            } else e[i][0] = *p;
            l[i] = last[(size_t)(c0 + c + i) * a.H + h];
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (c + i >= nc) continue;
            float* p = ends + (size_t)(c0 + c + i) * HNV + idx;
            if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(S[0], S[1], S[2], S[3]);
            else *p = S[0];
            const float keep = exp2f(l[i]);
#pragma unroll
            for (int k = 0; k < VEC; ++k) S[k] = fmaf(keep, S[k], e[i][k]);
        }
    }
    if (a.write_state) {
#pragma unroll
        for (int k = 0; k < VEC; ++k) st[k] = S[k];
    }
}

// pass 3: starts [chunk, H, N, V] is the state before every chunk.  Eight warps: 16 rows x half of the columns each.
template <int VT>
__global__ void __launch_bounds__(256) mamba2_chunk_out_kernel(const Mamba2Args a, const float* __restrict__ starts) {
    extern __shared__ __align__(16) unsigned char m2_raw[];
    __shared__ float s_d[M2_Q];
    __shared__ float2 s_l[M2_Q];
    __shared__ double s_carry;
    constexpr int LDX = VT + M2_PAD, VW = VT / 2;
    const int np = (a.N + 15) & ~15, ldb = np + M2_PAD;
    bf16* sc = reinterpret_cast<bf16*>(m2_raw);              // [Q][ldb]
    bf16* sb = sc + M2_Q * ldb;                              // [Q][ldb]
    bf16* sx = sb + M2_Q * ldb;                              // [Q][LDX]
    bf16* ss = sx + M2_Q * LDX;                              // [3][np][LDX]
    pdl_trigger();
    pdl_wait();
    int seq, t0, t1;
    if (!m2_find_chunk(a, blockIdx.x, seq, t0, t1)) return;
    const int h = blockIdx.y, g = h / (a.H / a.G), v0 = blockIdx.z * VT, nv = min(VT, a.V - v0);
    m2_load_rows(sc, ldb, a, a.H * a.V + (a.G + g) * a.N, a.N, np, t0, t1);
    m2_load_rows(sb, ldb, a, a.H * a.V + g * a.N, a.N, np, t0, t1);
    m2_load_rows(sx, LDX, a, h * a.V + v0, nv, VT, t0, t1);
    cp_async_commit();
    const float* S = starts + ((size_t)blockIdx.x * a.H + h) * a.N * a.V + v0;
    if ((a.V & 3) == 0 && (nv & 3) == 0) {
        constexpr int PER = VT / 4, U = 4;                   // four loads in flight a thread
        for (int i0 = threadIdx.x; i0 < np * PER; i0 += 256 * U) {
            float4 v[U];
#pragma unroll
            for (int k = 0; k < U; ++k) {
                const int i = i0 + 256 * k, n = i / PER, c = (i % PER) * 4;
                v[k] = (n < a.N && c < nv) ? *reinterpret_cast<const float4*>(S + (size_t)n * a.V + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int k = 0; k < U; ++k) {
                const int i = i0 + 256 * k, n = i / PER, c = (i % PER) * 4;
                if (n >= np) continue;
                uint32_t p[3], q[3];
                m2_split2(v[k].x, v[k].y, p);
                m2_split2(v[k].z, v[k].w, q);
#pragma unroll
                for (int m = 0; m < 3; ++m) *reinterpret_cast<uint2*>(ss + (m * np + n) * LDX + c) = make_uint2(p[m], q[m]);
            }
        }
    } else {
        for (int i = threadIdx.x; i < np * VT; i += 256) {
            const int n = i / VT, c = i % VT;
            float hi, mid, lo;
            m2_split((n < a.N && c < nv) ? S[(size_t)n * a.V + c] : 0.f, hi, mid, lo);
            ss[n * LDX + c] = __float2bfloat16_rn(hi);
            ss[(np + n) * LDX + c] = __float2bfloat16_rn(mid);
            ss[(2 * np + n) * LDX + c] = __float2bfloat16_rn(lo);
        }
    }
    m2_decays(a, h, t0, t1, s_d, s_l, &s_carry);
    cp_async_wait<0>();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mi = lane >> 3, r8 = lane & 7;
    const int wr = warp & 3, vb = (warp >> 2) * VW;
    const int i0 = wr * 16, ra = i0 + (lane >> 2), rb = ra + 8, tq = lane & 3;
    const float2 la = s_l[ra], lb = s_l[rb];

    // scores C . B of this warp's rows with the rows up to its own last one, and the read-out of the state before the chunk
    float sco[M2_Q / 8][4], acc[VW / 8][4];
#pragma unroll
    for (int i = 0; i < M2_Q / 8; ++i) sco[i][0] = sco[i][1] = sco[i][2] = sco[i][3] = 0.f;
#pragma unroll
    for (int i = 0; i < VW / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll 2
    for (int ks = 0; ks < np / 16; ++ks) {
        uint32_t fa[4];
        ldmatrix_x4(fa, sc + (i0 + (mi & 1) * 8 + r8) * ldb + ks * 16 + (mi >> 1) * 8);
#pragma unroll
        for (int jp = 0; jp < M2_Q / 16; ++jp) {
            if (jp > wr) continue;
            uint32_t fb[4];
            ldmatrix_x4(fb, sb + (jp * 16 + (mi >> 1) * 8 + r8) * ldb + ks * 16 + (mi & 1) * 8);
            mma_bf16(sco[2 * jp], fa, fb[0], fb[1]);
            mma_bf16(sco[2 * jp + 1], fa, fb[2], fb[3]);
        }
#pragma unroll
        for (int p = 2; p >= 0; --p) {
#pragma unroll
            for (int vp = 0; vp < VW / 16; ++vp) {
                uint32_t fb[4];
                ldmatrix_x4_trans(fb, ss + (p * np + ks * 16 + (mi & 1) * 8 + r8) * LDX + vb + vp * 16 + (mi >> 1) * 8);
                mma_bf16(acc[2 * vp], fa, fb[0], fb[1]);
                mma_bf16(acc[2 * vp + 1], fa, fb[2], fb[3]);
            }
        }
    }
    const float ea = exp2f(la.x), eb = exp2f(lb.x);
#pragma unroll
    for (int i = 0; i < VW / 8; ++i) {
        acc[i][0] *= ea; acc[i][1] *= ea; acc[i][2] *= eb; acc[i][3] *= eb;
    }
    // the chunk's own rows
#pragma unroll
    for (int ks = 0; ks < M2_Q / 16; ++ks) {
        if (ks > wr) continue;
        uint32_t f[3][4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {               // columns ks * 16 + 8 half + 2 tq, + 1
            const int j = ks * 16 + 8 * half + 2 * tq;
            const float d0 = s_d[j], d1 = s_d[j + 1];
            const float2 l0 = s_l[j], l1 = s_l[j + 1];
            const float* g4 = sco[2 * ks + half];
            uint32_t p[3], q[3];
            m2_split2(j <= ra ? g4[0] * (fast_exp2(m2_between(la, l0)) * d0) : 0.f, j + 1 <= ra ? g4[1] * (fast_exp2(m2_between(la, l1)) * d1) : 0.f, p);
            m2_split2(j <= rb ? g4[2] * (fast_exp2(m2_between(lb, l0)) * d0) : 0.f, j + 1 <= rb ? g4[3] * (fast_exp2(m2_between(lb, l1)) * d1) : 0.f, q);
#pragma unroll
            for (int k = 0; k < 3; ++k) {
                f[k][2 * half] = p[k];
                f[k][2 * half + 1] = q[k];
            }
        }
#pragma unroll
        for (int vp = 0; vp < VW / 16; ++vp) {
            uint32_t fb[4];
            ldmatrix_x4_trans(fb, sx + (ks * 16 + (mi & 1) * 8 + r8) * LDX + vb + vp * 16 + (mi >> 1) * 8);
#pragma unroll
            for (int p = 2; p >= 0; --p) {
                mma_bf16(acc[2 * vp], f[p], fb[0], fb[1]);
                mma_bf16(acc[2 * vp + 1], f[p], fb[2], fb[3]);
            }
        }
    }
    const float skip = a.skip[h];
    const bool even = ((a.V | v0) & 1) == 0;
#pragma unroll
    for (int i = 0; i < VW / 8; ++i) {
        const int c = vb + i * 8 + 2 * tq;
        if (c >= nv) continue;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int r = half ? rb : ra;
            if (t0 + r >= t1) continue;
            float* o = a.out + ((size_t)(t0 + r) * a.H + h) * a.V + v0 + c;
            const float y0 = fmaf(skip, __bfloat162float(sx[r * LDX + c]), acc[i][2 * half]);
            const float y1 = fmaf(skip, __bfloat162float(sx[r * LDX + c + 1]), acc[i][2 * half + 1]);
            if (even && c + 1 < nv) *reinterpret_cast<float2*>(o) = make_float2(y0, y1);
            else { o[0] = y0; if (c + 1 < nv) o[1] = y1; }
        }
    }
}

// ------------------------------------------------------------------------------------------------ one token a request
// Block (request, head).  y_in [S, stride]: the in-projection's rows, with x | B | C at `xbc_at` and the heads' step sizes at
// `dt_at`; the history [num_slots, L - 1, channels] is read only.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) mamba2_single_kernel(const Mamba2Args a, const T* __restrict__ y_in, int stride, int xbc_at,
                                                            int dt_at, const float* __restrict__ taps, const float* __restrict__ conv_bias,
                                                            const float* __restrict__ history, int L) {
    extern __shared__ __align__(16) float m2_smem[];
    float* sx = m2_smem;                         // [V rounded up to 4]
    float* sB = sx + ((a.V + 3) & ~3);           // [N]
    float* sC = sB + a.N;                        // [N]
    float* part = sC + a.N;                      // [blockDim.x * VEC]
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y, g = h / (a.H / a.G);
    const int slot = zai_checked_slot(a.slot_ids[s], a.num_slots, a.status);
    const int inner = a.H * a.V, ch = inner + 2 * a.G * a.N;
    const T* row = y_in + (size_t)s * stride;
    const float* hist = history + (size_t)slot * max(L - 1, 1) * ch;
    float* st = a.state + ((size_t)slot * a.H + h) * a.N * a.V;
    const int lv = min((a.V + VEC - 1) / VEC, (int)blockDim.x), rg_n = blockDim.x / lv, vi = threadIdx.x % lv, rg = threadIdx.x / lv;
    constexpr int U = 8;                         // rows of the state a thread has in flight
    float S[U][VEC];
    auto load = [&](int v, int n0) {
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const int n = n0 + i * rg_n;
            if (n >= a.N) continue;
            const float* p = st + (size_t)n * a.V + v;
            if constexpr (VEC == 4) {
                const float4 q = *reinterpret_cast<const float4*>(p);
                S[i][0] = q.x; S[i][1] = q.y; S[i][2] = q.z; S[i][3] = q.w;
            } else S[i][0] = *p;
        }
    };
    if (vi * VEC < a.V && rg < rg_n) load(vi * VEC, rg);      // (the first rows are on their way while the convolution runs)
    for (int i = threadIdx.x; i < a.V + 2 * a.N; i += blockDim.x) {
        const int c = i < a.V ? h * a.V + i : i < a.V + a.N ? inner + g * a.N + (i - a.V) : inner + (a.G + g) * a.N + (i - a.V - a.N);
        float acc = (conv_bias ? conv_bias[c] : 0.f) + taps[(size_t)c * L + (L - 1)] * to_float(row[xbc_at + c]);
        for (int j = 0; j < L - 1; ++j) acc += taps[(size_t)c * L + j] * hist[(size_t)j * ch + c];
        const float v = to_float(from_float<T>(m2_silu(acc)));
        if (i < a.V) sx[i] = v;
        else sB[i - a.V] = v;                    // (C lies behind B)
    }
    const float d = m2_softplus(to_float(row[dt_at + h]) + a.dt_bias[h]);
    const float keep = expf(-expf(a.a_log[h]) * d), skip = a.skip[h];
    __syncthreads();
    for (int v0 = 0; v0 < a.V; v0 += lv * VEC) {
        const int v = v0 + vi * VEC;
        const bool live = v < a.V && rg < rg_n;
        float x[VEC], y[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            x[k] = live ? d * sx[v + k] : 0.f;
            y[k] = 0.f;
        }
        for (int n0 = rg; n0 < a.N && live; n0 += rg_n * U) {
            if (v0 > 0 || n0 > rg) load(v, n0);
#pragma unroll
            for (int i = 0; i < U; ++i) {
                const int n = n0 + i * rg_n;
                if (n >= a.N) continue;
                const float b = sB[n], c = sC[n];
#pragma unroll
                for (int k = 0; k < VEC; ++k) {
                    S[i][k] = fmaf(keep, S[i][k], x[k] * b);
                    y[k] = fmaf(S[i][k], c, y[k]);
                }
                if (a.write_state) {
                    float* p = st + (size_t)n * a.V + v;
                    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
                    else *p = S[i][0];
                }
            }
        }
        __syncthreads();                         // (the sums of the columns before have been read)
        if (rg < rg_n) {
#pragma unroll
            for (int k = 0; k < VEC; ++k) part[(rg * lv + vi) * VEC + k] = y[k];
        }
        __syncthreads();
        for (int c = threadIdx.x; c < lv * VEC && v0 + c < a.V; c += blockDim.x) {
            float sum = 0.f;
            for (int r = 0; r < rg_n; ++r) sum += part[r * lv * VEC + c];
            a.out[((size_t)s * a.H + h) * a.V + v0 + c] = fmaf(skip, sx[v0 + c], sum);
        }
    }
}

// ------------------------------------------------------------------------------------------------ gate and norm
// out[t, c] = v[c] / sqrt(mean over c's part of v^2 + eps) * weight[c],  v = y silu(z); block (row, part).  With `history` (steps
// of single tokens) further blocks of a row move its request's convolution history on by the row's x | B | C.
template <typename T>
__global__ void __launch_bounds__(256) mamba2_norm_kernel(T* __restrict__ out, const float* __restrict__ y, const T* __restrict__ rows,
                                                          int stride, int z_at, const float* __restrict__ weight, float eps, int I,
                                                          int parts, int vec, float* __restrict__ history, int xbc_at, int ch, int L,
                                                          const int* __restrict__ slot_ids, int num_slots, int* __restrict__ status) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, part = blockIdx.y, len = I / parts;
    const T* row = rows + (size_t)t * stride;
    if (part >= parts) {
        const int c = (part - parts) * blockDim.x + threadIdx.x;
        if (c >= ch) return;
        const int slot = zai_checked_slot(slot_ids[t], num_slots, status);
        float* hist = history + (size_t)slot * (L - 1) * ch + c;
        float keep[M2_MAX_TAPS];
#pragma unroll
        for (int j = 1; j < M2_MAX_TAPS; ++j) keep[j] = j < L - 1 ? hist[(size_t)j * ch] : 0.f;
        const float cur = to_float(row[xbc_at + c]);
#pragma unroll
        for (int j = 1; j < M2_MAX_TAPS; ++j)
            if (j < L - 1) hist[(size_t)(j - 1) * ch] = keep[j];
        hist[(size_t)(L - 2) * ch] = cur;
        return;
    }
    const float* yp = y + (size_t)t * I + part * len;
    const T* zp = row + z_at + part * len;
    const float* wp = weight + part * len;
    T* op = out + (size_t)t * I + part * len;
    float q = 0.f;
    if (vec) {                                   // eight values a thread and step; the first two steps' stay in registers
        float v[2][8];
        auto load8 = [&](int c, float (&d)[8]) {
            const float4 a = *reinterpret_cast<const float4*>(yp + c), b = *reinterpret_cast<const float4*>(yp + c + 4);
            const float yv[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
            float zv[8];
            if constexpr (sizeof(T) == 2) {
                const uint4 u = *reinterpret_cast<const uint4*>(zp + c);
                const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float2 f = __bfloat1622float2(h[i]);
                    zv[2 * i] = f.x; zv[2 * i + 1] = f.y;
                }
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) zv[i] = to_float(zp[c + i]);
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) d[i] = yv[i] * m2_silu(zv[i]);
        };
        auto store8 = [&](int c, const float (&d)[8], float inv) {
            const float4 a = *reinterpret_cast<const float4*>(wp + c), b = *reinterpret_cast<const float4*>(wp + c + 4);
            const float w[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
            if constexpr (sizeof(T) == 2) {
                uint32_t u[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) u[i] = pack_bf16(d[2 * i] * inv * w[2 * i], d[2 * i + 1] * inv * w[2 * i + 1]);
                *reinterpret_cast<uint4*>(op + c) = make_uint4(u[0], u[1], u[2], u[3]);
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) op[c + i] = from_float<T>(d[i] * inv * w[i]);
            }
        };
        const int step = blockDim.x * 8, c0 = threadIdx.x * 8;
#pragma unroll
        for (int k = 0; k < 2; ++k)
            if (c0 + k * step < len) {
                load8(c0 + k * step, v[k]);
#pragma unroll
                for (int i = 0; i < 8; ++i) q += v[k][i] * v[k][i];
            }
        for (int c = c0 + 2 * step; c < len; c += step) {
            float d[8];
            load8(c, d);
#pragma unroll
            for (int i = 0; i < 8; ++i) q += d[i] * d[i];
        }
        const float inv = rsqrtf(block_sum(q, red) / (float)len + eps);
#pragma unroll
        for (int k = 0; k < 2; ++k)
            if (c0 + k * step < len) store8(c0 + k * step, v[k], inv);
        for (int c = c0 + 2 * step; c < len; c += step) {
            float d[8];
            load8(c, d);
            store8(c, d, inv);
        }
        return;
    }
    for (int c = threadIdx.x; c < len; c += blockDim.x) {
        const float v = yp[c] * m2_silu(to_float(zp[c]));
        q += v * v;
    }
    const float inv = rsqrtf(block_sum(q, red) / (float)len + eps);
    for (int c = threadIdx.x; c < len; c += blockDim.x) op[c] = from_float<T>(yp[c] * m2_silu(to_float(zp[c])) * inv * wp[c]);
}

// ------------------------------------------------------------------------------------------------ launchers
static size_t m2_state_smem(int N, int vt) {
    const size_t np = (N + 15) & ~15;
    return (M2_Q * (np + M2_PAD) + (size_t)3 * M2_Q * (vt + M2_PAD)) * 2;
}
static size_t m2_out_smem(int N, int vt) {
    const size_t np = (N + 15) & ~15;
    return (2 * M2_Q * (np + M2_PAD) + (size_t)(M2_Q + 3 * np) * (vt + M2_PAD)) * 2;
}
static const size_t M2_SMEM_LIMIT = 220 * 1024;
// The columns of V that a block of the chunked kernels takes, 0 if the sizes do not fit them.
static int m2_chunk_cols(int N, int V) {
    const int vt = V > 32 ? 64 : 32;
    if (m2_out_smem(N, vt) <= M2_SMEM_LIMIT) return vt;
    return m2_out_smem(N, 32) <= M2_SMEM_LIMIT ? 32 : 0;
}

// 1 if spans of `M2_Q`-row chunks can go to the tensor cores with these sizes (bfloat16)
ZAI_API int zai_mamba2_chunked_supports(int N, int V) { return N >= 1 && V >= 1 && m2_chunk_cols(N, V) > 0; }
ZAI_API int zai_mamba2_chunk_rows() { return M2_Q; }

// The walk over every span of min_rows..max_rows rows.  u [rows, u_stride]: x (H V) | B (G N) | C (G N); dt [rows, dt_stride];
// out [rows, H V] 32-bit; state [num_slots, H, N, V] 32-bit.
ZAI_API int zai_mamba2_scan(float* out, const void* u, int u_stride, const void* dt, int dt_stride, int dtype, const float* dt_bias,
                            const float* a_log, const float* skip, float* state, const int* cu_q, const int* slot_ids, int num_slots,
                            int* status, int n_seqs, int H, int G, int N, int V, int write_state, int min_rows, int max_rows,
                            cudaStream_t stream) {
    if (n_seqs <= 0) return ZAI_OK;
    if (H < 1 || H > 65535 || G < 1 || H % G || N < 1 || N > MAMBA2_MAX_STATE || V < 1) return ZAI_BAD_SIZE;
    const Mamba2Args a = {u, u_stride, dt, dt_stride, dt_bias, a_log, skip, out, state, cu_q, slot_ids, status, num_slots, n_seqs,
                          H, G, N, V, write_state, min_rows, max_rows};
    const int nw = (N + 31) / 32;
    const size_t smem = ((size_t)M2_TT * nw * 32 * 3 + M2_TT * 34) * sizeof(float);
    static unsigned long long done[2] = {0, 0};
    if (dtype != ZAI_F32 && dtype != ZAI_BF16) return ZAI_BAD_DTYPE;
    if (zai_first_on_device(&done[dtype])) {
        const int most = (int)(((size_t)M2_TT * 16 * 32 * 3 + M2_TT * 34) * sizeof(float));
        cudaError_t e;
        if (dtype == ZAI_F32) e = cudaFuncSetAttribute(mamba2_scan_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
        else e = cudaFuncSetAttribute(mamba2_scan_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
        if (e != cudaSuccess) return (int)e;
    }
    ZAI_DISPATCH(dtype, return launch_pdl(mamba2_scan_kernel<T>, dim3(n_seqs, H, (V + 31) / 32), dim3(nw * 32), smem, stream, a));
}

template <int VT>
static int m2_chunked(const Mamba2Args& a, float* ends, float* last, int max_chunks, cudaStream_t stream) {
    static unsigned long long done = 0;
    if (zai_first_on_device(&done)) {
        cudaError_t e = cudaFuncSetAttribute(mamba2_chunk_state_kernel<VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)M2_SMEM_LIMIT);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(mamba2_chunk_out_kernel<VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)M2_SMEM_LIMIT);
        if (e != cudaSuccess) return (int)e;
    }
    const dim3 grid(max_chunks, a.H, (a.V + VT - 1) / VT);
    int rc = launch_pdl(mamba2_chunk_state_kernel<VT>, grid, dim3(256), m2_state_smem(a.N, VT), stream, a, ends, last);
    if (rc) return rc;
    const size_t total = (size_t)a.H * a.N * a.V;
    if (((size_t)a.N * a.V) % 4 == 0)
        rc = launch_pdl(mamba2_state_pass_kernel<4>, dim3((unsigned)((total / 4 + 127) / 128), a.n_seqs), dim3(128), 0, stream, a, ends, (const float*)last);
    else
        rc = launch_pdl(mamba2_state_pass_kernel<1>, dim3((unsigned)((total + 127) / 128), a.n_seqs), dim3(128), 0, stream, a, ends, (const float*)last);
    if (rc) return rc;
    return launch_pdl(mamba2_chunk_out_kernel<VT>, grid, dim3(256), m2_out_smem(a.N, VT), stream, a, (const float*)ends);
}

// The same over every span of min_rows rows or more, bfloat16, in chunks on the tensor cores.  ends [max_chunks, H, N, V] and
// last [max_chunks, H] are 32-bit scratch; rows / M2_Q + n_seqs chunks are always enough.
ZAI_API int zai_mamba2_chunked(float* out, const void* u, int u_stride, const void* dt, int dt_stride, const float* dt_bias,
                               const float* a_log, const float* skip, float* state, const int* cu_q, const int* slot_ids,
                               int num_slots, int* status, int n_seqs, int H, int G, int N, int V, int write_state, int min_rows,
                               float* ends, float* last, int max_chunks, cudaStream_t stream) {
    if (n_seqs <= 0 || max_chunks <= 0) return ZAI_OK;
    if (H < 1 || H > 65535 || n_seqs > 65535 || G < 1 || H % G || N < 1 || V < 1) return ZAI_BAD_SIZE;
    const Mamba2Args a = {u, u_stride, dt, dt_stride, dt_bias, a_log, skip, out, state, cu_q, slot_ids, status, num_slots, n_seqs,
                          H, G, N, V, write_state, min_rows < 1 ? 1 : min_rows, 0x7fffffff};
    const int vt = m2_chunk_cols(N, V);
    if (vt == 64) return m2_chunked<64>(a, ends, last, max_chunks, stream);
    if (vt == 32) return m2_chunked<32>(a, ends, last, max_chunks, stream);
    return ZAI_BAD_SIZE;
}

// A step of single tokens, row i of request i: rows [S, stride] with x | B | C at xbc_at and dt at dt_at; taps [channels, L],
// history [num_slots, L - 1, channels] (read; `zai_mamba2_norm` moves it on); out [S, H V] 32-bit.
ZAI_API int zai_mamba2_single(float* out, const void* rows, int stride, int dtype, int xbc_at, int dt_at, const float* taps,
                              const float* conv_bias, const float* history, int L, const float* dt_bias, const float* a_log,
                              const float* skip, float* state, const int* slot_ids, int num_slots, int* status, int S, int H, int G,
                              int N, int V, int write_state, cudaStream_t stream) {
    if (S <= 0) return ZAI_OK;
    if (H < 1 || H > 65535 || G < 1 || H % G || N < 1 || N > MAMBA2_MAX_STATE || V < 1 || V > 4096 || L < 1 || L > M2_MAX_TAPS) return ZAI_BAD_SIZE;
    const Mamba2Args a = {nullptr, 0, nullptr, 0, dt_bias, a_log, skip, out, state, nullptr, slot_ids, status, num_slots, S,
                          H, G, N, V, write_state, 0, 0};
    const bool vec = V % 4 == 0;
    const size_t smem = ((size_t)((V + 3) & ~3) + 2 * N + 256 * (vec ? 4 : 1)) * sizeof(float);
    if (vec) { ZAI_DISPATCH(dtype, return launch_pdl(mamba2_single_kernel<T, 4>, dim3(S, H), dim3(256), smem, stream, a, (const T*)rows, stride,
                                                     xbc_at, dt_at, taps, conv_bias, history, L)); }
    ZAI_DISPATCH(dtype, return launch_pdl(mamba2_single_kernel<T, 1>, dim3(S, H), dim3(256), smem, stream, a, (const T*)rows, stride, xbc_at,
                                          dt_at, taps, conv_bias, history, L));
}

// out [N, I] in `dtype` from y [N, I] 32-bit and z at z_at of rows [N, stride].  With `history` every row is its request's only
// one, and the history [num_slots, L - 1, ch] takes in the row's ch values at xbc_at.
ZAI_API int zai_mamba2_norm(void* out, const float* y, const void* rows, int stride, int dtype, int z_at, const float* weight, float eps,
                            int N, int I, int parts, float* history, int xbc_at, int ch, int L, const int* slot_ids, int num_slots,
                            int* status, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    if (I < 1 || parts < 1 || I % parts || L > M2_MAX_TAPS) return ZAI_BAD_SIZE;
    const int len = I / parts;
    const int vec = len % 8 == 0 && stride % 8 == 0 && z_at % 8 == 0
                    && ((reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(rows) | reinterpret_cast<uintptr_t>(weight)) & 15) == 0;
    int threads = ((vec ? len / 8 : len) + 31) / 32 * 32;
    threads = threads > 256 ? 256 : threads;
    const int moving = (history && L > 1) ? (ch + threads - 1) / threads : 0;
    if (parts + moving > 65535) return ZAI_BAD_SIZE;
    ZAI_DISPATCH(dtype, return launch_pdl(mamba2_norm_kernel<T>, dim3(N, parts + moving), dim3(threads), 0, stream, (T*)out, y,
                                          (const T*)rows, stride, z_at, weight, eps, I, parts, vec, history, xbc_at, ch, L, slot_ids,
                                          num_slots, status));
}
