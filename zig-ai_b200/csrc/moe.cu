// A mixture of small gated feed-forwards: every row of the step goes to its `top` experts by router score.
//
//   z = x . Wr^T (32-bit),  s = sigmoid(z),  the `top` largest s choose the experts (ties: the lower index),
//   weights w = s of the chosen (divided by their sum with `renorm`); or the logits themselves, z plus an optional bias,
//   choose, and w = softmax over the chosen logits alone
//   y = sum over the chosen e of  down_e( silu(gate_e(x_e)) * up_e(x_e) ),   x_e = w_e x   (`weight_on` input)
//                                or of  w_e down_e( silu(gate_e(x)) * up_e(x) )             (`weight_on` output)
//
// The choice may differ from the scores: choice = s + a correction per expert, the experts may form groups of neighbours of
// which only the best few (by their largest choice value) are chosen from, and the weights may be multiplied by a factor.  The
// last experts of the router may be identities: they have no matrices and give the row itself, so their rows never enter the
// sorted layout and join in the combine.
//
// The experts may also be units without a gate, down_e( act(up_e(x)) ), act the square of relu; and a unit that every row
// passes beside its experts joins in the combine, weighed by the sigmoid of one more 32-bit product of the row.
//
// Five kernels, none of which tells the host anything (the step stays a fixed list of launches):
//   * route: a block a row; the router's products summed in 32-bit in an order that depends on the width alone, the
//     choice, and the row's place among its expert's rows (a counter per expert);
//   * gather: the rows, scaled, into a layout sorted by expert in which every expert's rows start at a multiple of
//     the tile height TM (padding rows hold whatever was there: a row's result never depends on another row), and the
//     expert of every tile;
//   * two grouped products over that layout (gate|up with the activation as epilogue, then down): a block owns a
//     tile of TM rows x 32 or 64 output columns of one expert; bfloat16 on the tensor cores (mma.sync m16n8k16, cp.async
//     ring), any other case by 32-bit multiply-adds.  Steps with many rows an expert gather with a
//     tile height of 128 and run both products in the grouped mode of the tcgen05 kernel (gemm_tc.cu) instead;
//   * combine: a row's `top` results summed in 32-bit in the order of the choice and rounded once; or the sum, unrounded, and
//     the rows of a mixer beside the experts are added to the 32-bit residual stream, which is then rounded for its next reader.
// A row's result depends on the row alone: on which tile it lands, what else the tile holds and in which order the
// counter was taken changes nothing, since every output element is a sum over k in a fixed order.
#include "mma_helpers.cuh"

#define MOE_PLAIN_TN 64    // output columns of a block of the plain kernel
#define MOE_PLAIN_TK 32    // k per stage of the plain kernel
// The tensor-core kernel's block by the tile height TM and its output columns TN: warps, k per stage, stages.  With few rows a
// block mostly brings its weights in, one pass, so what it keeps in flight is what hides the way to memory; narrow tiles
// where wide ones would leave SMs without a block.  An output element is the same sum in the same order whatever TN is.
template <int TM, int TN> struct MoeTile {
    static constexpr int WARPS = TM == 16 ? TN / 16 : 4, TK = 64, ST = TK + 8, STAGES = TM == 16 ? (TN == 32 ? 10 : 6) : 4;
    static constexpr size_t BYTES = (size_t)STAGES * (TM + TN) * ST * 2;
};
#define MOE_WIDE_BLOCKS 296      // from this many blocks of 64 columns on, 64 columns a block

// Eight neighbouring values as 32-bit numbers by 16-byte accesses (the caller has checked the alignment).
__device__ __forceinline__ void moe_load8(float (&v)[8], const bf16* p) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x; v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void moe_load8(float (&v)[8], const float* p) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void moe_store8(bf16* p, const float (&v)[8]) {
    uint4 u;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = u;
}
__device__ __forceinline__ void moe_store8(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
template <typename T>
__device__ __forceinline__ bool moe_rows_aligned(const T* p, size_t stride, int W) {
    return (W & 7) == 0 && (stride & 7) == 0 && (reinterpret_cast<uintptr_t>(p) & 15) == 0;
}

// ------------------------------------------------------------------------------------------------ route
enum { MOE_SIGMOID = 0, MOE_SOFTMAX = 1, MOE_LOGITS = 2 };          // what the scores are
// How the choice differs from the scores (all zero: it does not).  `real`: the experts that have matrices; those behind them
// are identities.
struct MoeChoice {
    const float* correction;       // [E] or null
    int groups, keep, real;        // groups 0: none
    float scale;                   // on the weights
    __host__ __device__ bool own() const { return correction != nullptr || groups > 0; }      // a choice value beside the score
};
// ROWS rows a block (their values are read once per expert row of the router for all of them); a row's sums have the same order
// whatever ROWS and the number of warps are.
template <typename T, int ROWS>
__global__ void __launch_bounds__(512) moe_route_kernel(int* __restrict__ ids, float* __restrict__ wts, int* __restrict__ rank,
                                                        int* __restrict__ counts, const T* __restrict__ x, int x_stride,
                                                        const float* __restrict__ wr, int N, int W, int E, int top, int renorm,
                                                        int score, const float* __restrict__ bias, float* __restrict__ unit_gate,
                                                        const MoeChoice choice) {
    extern __shared__ float sc_all[];                    // [ROWS][E] scores, then (a choice of its own) [ROWS][E + groups]
    const int tr = blockIdx.x * ROWS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    pdl_trigger();
    pdl_wait();
    // (which of the two loops runs depends on the sizes and addresses alone, never on the other rows of the step)
    const bool vec = moe_rows_aligned(x, (size_t)x_stride, W) && (reinterpret_cast<uintptr_t>(wr) & 15) == 0;
    for (int e = warp; e < E + (unit_gate ? 1 : 0); e += nw) {
        const float* w = wr + (size_t)e * W;
        float acc[ROWS];
#pragma unroll
        for (int r = 0; r < ROWS; ++r) acc[r] = 0.f;
        if (vec) {
#pragma unroll 4
            for (int c = lane * 8; c < W; c += 256) {
                float xv[8], wv[8];
                moe_load8(wv, w + c);
#pragma unroll
                for (int r = 0; r < ROWS; ++r) {
                    moe_load8(xv, x + (size_t)min(tr + r, N - 1) * x_stride + c);
#pragma unroll
                    for (int i = 0; i < 8; ++i) acc[r] += xv[i] * wv[i];
                }
            }
        } else {
            for (int c = lane; c < W; c += 32) {
                const float wv = w[c];
#pragma unroll
                for (int r = 0; r < ROWS; ++r) acc[r] += to_float(x[(size_t)min(tr + r, N - 1) * x_stride + c]) * wv;
            }
        }
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            const float z = warp_sum(acc[r]);
            if (lane != 0 || tr + r >= N) continue;
            if (e == E) unit_gate[tr + r] = 1.f / (1.f + expf(-z));      // (the row behind the router's: the unit beside the experts)
            else sc_all[r * E + e] = score == MOE_SIGMOID ? 1.f / (1.f + expf(-z)) : bias ? z + bias[e] : z;
        }
    }
    __syncthreads();
    const int t = tr + warp;
    if (warp >= ROWS || t >= N) return;
    float* sc = sc_all + warp * E;
    if (score == MOE_SOFTMAX) {                          // scores = softmax of the logits over all experts, in a fixed order
        float top_z = -INFINITY;
        for (int e = lane; e < E; e += 32) top_z = fmaxf(top_z, sc[e]);
        top_z = warp_max(top_z);
        float total = 0.f;
        for (int e = lane; e < E; e += 32) total += expf(sc[e] - top_z);
        total = warp_sum(total);
        for (int e = lane; e < E; e += 32) sc[e] = expf(sc[e] - top_z) / total;
        __syncwarp();
    }
    float* ch = sc;                                      // what the choice goes by
    if (choice.own()) {
        ch = sc_all + ROWS * E + warp * (E + choice.groups);
        for (int e = lane; e < E; e += 32) ch[e] = choice.correction ? sc[e] + choice.correction[e] : sc[e];
        __syncwarp();
        if (choice.groups > 0) {                         // a group's value is its largest; the `keep` best groups stay (ties: the lower)
            float* gv = ch + E;
            const int size = E / choice.groups;
            for (int q = lane; q < choice.groups; q += 32) {
                float v = ch[q * size];
                for (int i = 1; i < size; ++i) v = fmaxf(v, ch[q * size + i]);
                gv[q] = v;
            }
            __syncwarp();
            for (int q = lane; q < choice.groups; q += 32) {
                int above = 0;
                for (int o = 0; o < choice.groups; ++o) above += gv[o] > gv[q] || (gv[o] == gv[q] && o < q);
                if (above >= choice.keep)
                    for (int i = 0; i < size; ++i) ch[q * size + i] = -INFINITY;
            }
            __syncwarp();
        }
    }
    float sum = 0.f, mine = -INFINITY, first = 0.f;      // (`mine`: lane k keeps the k-th choice's score)
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int at = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            const float v = ch[e];
            if (v > best) { best = v; at = e; }          // (ascending e: the first of equals stays)
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (ov > best || (ov == best && oa < at)) { best = ov; at = oa; }
        }
        if (at >= E) at = 0;                             // (scores that are no numbers: any expert, never an index outside)
        if (choice.own()) best = sc[at];                 // the weight is the score, whatever the choice went by
        __syncwarp();
        if (lane == 0) {
            ids[(size_t)t * top + k] = at;
            wts[(size_t)t * top + k] = best;
            rank[(size_t)t * top + k] = at < choice.real ? atomicAdd(&counts[at], 1) : -1;
            ch[at] = -INFINITY;
        }
        if (lane == k) mine = best;
        if (k == 0) first = best;
        sum += best;
        __syncwarp();
    }
    __syncwarp();
    if (score == MOE_LOGITS) {                           // softmax over the chosen logits, the first of which is the largest
        const float w = lane < top ? expf(mine - first) : 0.f;
        const float total = warp_sum(w);
        if (lane < top) wts[(size_t)t * top + lane] = w / total;
        return;
    }
    if (lane >= top) return;
    if (renorm) wts[(size_t)t * top + lane] = wts[(size_t)t * top + lane] / (sum + 1e-20f) * choice.scale;
    else if (choice.scale != 1.f) wts[(size_t)t * top + lane] *= choice.scale;
}

// ------------------------------------------------------------------------------------------------ gather
// One block per (row, choice) and one more that writes the tiles' experts.  The first row of expert e in the sorted
// layout is sum_{e' < e} roundup(counts[e'], TM).
template <typename T>
__global__ void __launch_bounds__(128) moe_gather_kernel(T* __restrict__ xs, int* __restrict__ dest, int* __restrict__ tile_expert,
                                                         const T* __restrict__ x, int x_stride, const int* __restrict__ ids,
                                                         const float* __restrict__ wts, const int* __restrict__ rank,
                                                         const int* __restrict__ counts, int items, int W, int E, int top, int TM,
                                                         int max_tiles, int scale_input) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    if ((int)blockIdx.x == items) {                      // the tiles' experts (-1: a tile that no expert uses)
        __shared__ int s_tiles;
        if (threadIdx.x == 0) {
            int at = 0;
            for (int e = 0; e < E; ++e) {
                const int n = (counts[e] + TM - 1) / TM;
                for (int i = 0; i < n && at + i < max_tiles; ++i) tile_expert[at + i] = e;
                at += n;
            }
            s_tiles = at < max_tiles ? at : max_tiles;
        }
        __syncthreads();
        for (int i = s_tiles + threadIdx.x; i < max_tiles; i += blockDim.x) tile_expert[i] = -1;
        return;
    }
    const int item = blockIdx.x, t = item / top, e = ids[item];
    if (e >= E) {                                        // an identity: nothing to sort
        if (threadIdx.x == 0) dest[item] = -1;
        return;
    }
    float before = 0.f;                                  // (whole numbers below 2^24: exact in 32-bit floats)
    for (int o = threadIdx.x; o < e; o += blockDim.x) before += (float)(((counts[o] + TM - 1) / TM) * TM);
    const int first = (int)block_sum(before, red);
    const int d = first + rank[item];
    if (threadIdx.x == 0) dest[item] = d;
    const float w = scale_input ? wts[item] : 1.f;
    const T* src = x + (size_t)t * x_stride;
    T* dst = xs + (size_t)d * W;
    if (moe_rows_aligned(x, (size_t)x_stride, W) && (reinterpret_cast<uintptr_t>(xs) & 15) == 0) {
        for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
            float v[8];
            moe_load8(v, src + c);
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = to_float(from_float<T>(v[i] * w));
            moe_store8(dst + c, v);
        }
        return;
    }
    for (int c = threadIdx.x; c < W; c += blockDim.x) dst[c] = from_float<T>(to_float(src[c]) * w);
}

// ------------------------------------------------------------------------------------------------ grouped products
// epilogue 0: out[row, n] (TO); 1: out[row, f] = silu(gate f) * up f, the weights being [E, 2 F, K] (gate rows, up rows)
template <typename TO>
__device__ __forceinline__ void moe_store(TO* p, float v);
template <> __device__ __forceinline__ void moe_store<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void moe_store<bf16>(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float moe_silu(float g) { return g / (1.f + expf(-g)); }
// The gated epilogues: 1  silu(g) u;  2  g' sigmoid(alpha g') (u' + 1) with g' = min(g, limit), u' = clamp(u, -limit, limit).
// Without a gate: 0  v;  3  relu(v)^2
struct MoeAct {
    int kind;
    float limit, alpha;
    __device__ __forceinline__ float operator()(float g, float u) const {
        if (kind != 2) return moe_silu(g) * u;
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g / (1.f + expf(-alpha * g)) * (u + 1.f);
    }
    __device__ __forceinline__ float plain(float v) const {
        if (kind != 3) return v;
        v = fmaxf(v, 0.f);
        return v * v;
    }
};

// The weight row that row r (0..TN - 1) of a block's tile of weights holds, or -1.  Plain: output column n0 + r.  Gated:
// groups of eight rows alternate between the gate and the up rows of the same eight features.
template <int TN>
__device__ __forceinline__ int moe_weight_row(int r, int col_block, int n_out, int gated) {
    if (!gated) {
        const int n = col_block * TN + r;
        return n < n_out ? n : -1;
    }
    const int f = col_block * (TN / 2) + (r >> 4) * 8 + (r & 7);
    return f < n_out ? ((r >> 3) & 1) * n_out + f : -1;
}

template <int TM, int TN, typename TO>
__global__ void __launch_bounds__(MoeTile<TM, TN>::WARPS * 32) moe_gemm_mma_kernel(TO* __restrict__ out, const bf16* __restrict__ xs,
                                                           const bf16* __restrict__ w, const int* __restrict__ tile_expert,
                                                           int K, int n_out, int gated, const MoeAct act) {
    constexpr int MOE_TN = TN, THREADS = MoeTile<TM, TN>::WARPS * 32;
    constexpr int WM = TM / 16, WN = MoeTile<TM, TN>::WARPS / WM, NT = MOE_TN / 8 / WN;   // warps along rows and columns; 8-column tiles a warp
    constexpr int MOE_TK = MoeTile<TM, TN>::TK, MOE_ST = MoeTile<TM, TN>::ST, MOE_STAGES = MoeTile<TM, TN>::STAGES;
    extern __shared__ __align__(16) unsigned char moe_raw[];
    bf16 (*sa)[TM][MOE_ST] = reinterpret_cast<bf16 (*)[TM][MOE_ST]>(moe_raw);
    bf16 (*sb)[MOE_TN][MOE_ST] = reinterpret_cast<bf16 (*)[MOE_TN][MOE_ST]>(moe_raw + (size_t)MOE_STAGES * TM * MOE_ST * 2);
    pdl_trigger();
    pdl_wait();
    const int e = tile_expert[blockIdx.x];
    if (e < 0) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int wm = warp % WM, wn = warp / WM;
    const size_t row0 = (size_t)blockIdx.x * TM;
    const bf16* wexp = w + (size_t)e * (gated ? 2 : 1) * n_out * K;
    const int n_k = (K + MOE_TK - 1) / MOE_TK;
    auto load = [&](int kt, int buf) {
        const int k0 = kt * MOE_TK;
        for (int i = tid; i < TM * (MOE_TK / 8); i += THREADS) {
            const int r = i / (MOE_TK / 8), c = (i % (MOE_TK / 8)) * 8;
            const bool ok = k0 + c < K;
            cp_async16(&sa[buf][r][c], xs + (row0 + r) * K + (ok ? k0 + c : 0), ok);
        }
        for (int i = tid; i < MOE_TN * (MOE_TK / 8); i += THREADS) {
            const int r = i / (MOE_TK / 8), c = (i % (MOE_TK / 8)) * 8;
            const int wr = moe_weight_row<MOE_TN>(r, blockIdx.y, n_out, gated);
            const bool ok = wr >= 0 && k0 + c < K;
            cp_async16(&sb[buf][r][c], wexp + (ok ? (size_t)wr * K + k0 + c : 0), ok);
        }
    };
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int s = 0; s < MOE_STAGES - 1; ++s) {
        if (s < n_k) load(s, s);
        cp_async_commit();
    }
    const int a_row = (((lane >> 3) & 1) << 3) + (lane & 7), a_dof = (lane >> 4) << 3;
    const int b_row = ((lane >> 4) << 3) + (lane & 7), b_dof = ((lane >> 3) & 1) << 3;
    for (int kt = 0; kt < n_k; ++kt) {
        cp_async_wait<MOE_STAGES - 2>();
        __syncthreads();                                 // stage kt has landed; stage kt - 1 has been read by every warp
        if (kt + MOE_STAGES - 1 < n_k) load(kt + MOE_STAGES - 1, (kt + MOE_STAGES - 1) % MOE_STAGES);
        cp_async_commit();
        const int buf = kt % MOE_STAGES;
#pragma unroll
        for (int ks = 0; ks < MOE_TK / 16; ++ks) {
            uint32_t a[4];
            ldmatrix_x4(a, &sa[buf][wm * 16 + a_row][ks * 16 + a_dof]);
#pragma unroll
            for (int np = 0; np < NT / 2; ++np) {
                uint32_t b[4];
                ldmatrix_x4(b, &sb[buf][(wn * NT + np * 2) * 8 + b_row][ks * 16 + b_dof]);
                mma_bf16(acc[np * 2], a, b[0], b[1]);
                mma_bf16(acc[np * 2 + 1], a, b[2], b[3]);
            }
        }
    }
    cp_async_wait<0>();
    const int g = lane >> 2, tq = lane & 3;
    const size_t ra = row0 + wm * 16 + g, rb = ra + 8;
    if (gated) {
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                const int f = blockIdx.y * (MOE_TN / 2) + (wn * (NT / 2) + np) * 8 + 2 * tq + c;
                if (f < n_out) {
                    moe_store<TO>(out + ra * n_out + f, act(acc[np * 2][c], acc[np * 2 + 1][c]));
                    moe_store<TO>(out + rb * n_out + f, act(acc[np * 2][2 + c], acc[np * 2 + 1][2 + c]));
                }
            }
        }
        return;
    }
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            const int n = blockIdx.y * MOE_TN + (wn * NT + nt) * 8 + 2 * tq + c;
            if (n < n_out) {
                moe_store<TO>(out + ra * n_out + n, act.plain(acc[nt][c]));
                moe_store<TO>(out + rb * n_out + n, act.plain(acc[nt][2 + c]));
            }
        }
    }
}

// Any element type and any K: a tile of 16 rows x 64 columns by 32-bit multiply-adds, k in ascending order.
template <typename T, typename TO>
__global__ void __launch_bounds__(128) moe_gemm_plain_kernel(TO* __restrict__ out, const T* __restrict__ xs, const T* __restrict__ w,
                                                             const int* __restrict__ tile_expert, int K, int n_out, int gated,
                                                             const MoeAct act) {
    __shared__ float sa[16][MOE_PLAIN_TK + 1];
    __shared__ float sb[MOE_PLAIN_TN][MOE_PLAIN_TK + 1];
    pdl_trigger();
    pdl_wait();
    const int e = tile_expert[blockIdx.x];
    if (e < 0) return;
    const int tid = threadIdx.x, r = tid >> 3, c8 = tid & 7;
    const size_t row0 = (size_t)blockIdx.x * 16;
    const T* wexp = w + (size_t)e * (gated ? 2 : 1) * n_out * K;
    float acc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = 0.f;
    for (int k0 = 0; k0 < K; k0 += MOE_PLAIN_TK) {
        __syncthreads();
        for (int i = tid; i < 16 * MOE_PLAIN_TK; i += 128) {
            const int rr = i / MOE_PLAIN_TK, kk = i % MOE_PLAIN_TK;
            sa[rr][kk] = k0 + kk < K ? to_float(xs[(row0 + rr) * K + k0 + kk]) : 0.f;
        }
        for (int i = tid; i < MOE_PLAIN_TN * MOE_PLAIN_TK; i += 128) {
            const int rr = i / MOE_PLAIN_TK, kk = i % MOE_PLAIN_TK;
            const int wr = moe_weight_row<MOE_PLAIN_TN>(rr, blockIdx.y, n_out, gated);
            sb[rr][kk] = (wr >= 0 && k0 + kk < K) ? to_float(wexp[(size_t)wr * K + k0 + kk]) : 0.f;
        }
        __syncthreads();
#pragma unroll 4
        for (int kk = 0; kk < MOE_PLAIN_TK; ++kk) {
            const float a = sa[r][kk];
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[j] = fmaf(a, sb[c8 + 8 * j][kk], acc[j]);
        }
    }
    // column c8 + 8 j of the tile: gated, groups of eight alternate gate / up, so j even is a gate and j + 1 its up
    if (gated) {
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
            const int f = blockIdx.y * (MOE_PLAIN_TN / 2) + (j / 2) * 8 + c8;
            if (f < n_out) moe_store<TO>(out + (row0 + r) * n_out + f, act(acc[j], acc[j + 1]));
        }
        return;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        const int n = blockIdx.y * MOE_PLAIN_TN + c8 + 8 * j;
        if (n < n_out) moe_store<TO>(out + (row0 + r) * n_out + n, act.plain(acc[j]));
    }
}

// ------------------------------------------------------------------------------------------------ combine
// What the combine adds beside the experts' results.  `h`: the residual stream [N, W]; the row's sum and `other` (the rows of
// a mixer that read the same stream, or null) are added to it and `out` (which may then be null) gets the stream rounded.
template <typename T>
struct MoeBeside {
    const T* unit;                 // [N, W] rows of the unit beside the experts, or null
    const float* unit_gate;        // [N] its weights, or null
    const T* x;                    // the rows that identities give (dest < 0), row stride x_stride
    int x_stride;
    float* h;
    const T* other;
};
template <typename T>
__global__ void moe_combine_kernel(T* __restrict__ out, const float* __restrict__ y, const int* __restrict__ dest,
                                   const float* __restrict__ wts, int W, int top, int scale_output, const MoeBeside<T> a) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const float ug = a.unit_gate ? a.unit_gate[t] : 1.f;
    const T* xrow = a.x ? a.x + (size_t)t * a.x_stride : nullptr;
    const uintptr_t addresses = reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(a.unit) |
                                reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.h) | reinterpret_cast<uintptr_t>(a.other);
    if ((W & 7) == 0 && (addresses & 15) == 0 && (a.x_stride & 7) == 0) {
        for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {      // the same sums in the same order, eight columns at a time
            float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            for (int k = 0; k < top; ++k) {
                float v[8];
                const int d = dest[(size_t)t * top + k];
                if (d >= 0) moe_load8(v, y + (size_t)d * W + c);
                else moe_load8(v, xrow + c);
                const bool scaled = scale_output || d < 0;
                const float wk = scaled ? wts[(size_t)t * top + k] : 1.f;
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[i] += scaled ? v[i] * wk : v[i];
            }
            if (a.unit) {
                float v[8];
                moe_load8(v, a.unit + (size_t)t * W + c);
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[i] += ug * v[i];
            }
            if (a.h) {
                float v[8];
                if (a.other) {
                    moe_load8(v, a.other + (size_t)t * W + c);
#pragma unroll
                    for (int i = 0; i < 8; ++i) acc[i] += v[i];
                }
                moe_load8(v, a.h + (size_t)t * W + c);
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[i] += v[i];
                moe_store8(a.h + (size_t)t * W + c, acc);
            }
            if (out) moe_store8(out + (size_t)t * W + c, acc);
        }
        return;
    }
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        float acc = 0.f;
        for (int k = 0; k < top; ++k) {
            const int d = dest[(size_t)t * top + k];
            const float v = d >= 0 ? y[(size_t)d * W + c] : to_float(xrow[c]);
            acc += scale_output || d < 0 ? v * wts[(size_t)t * top + k] : v;
        }
        if (a.unit) acc += ug * to_float(a.unit[(size_t)t * W + c]);
        if (a.h) {
            if (a.other) acc += to_float(a.other[(size_t)t * W + c]);
            acc += a.h[(size_t)t * W + c];
            a.h[(size_t)t * W + c] = acc;
        }
        if (out) out[(size_t)t * W + c] = from_float<T>(acc);
    }
}

// ------------------------------------------------------------------------------------------------ launchers
// ids, rank [N, top] int; wts [N, top] 32-bit; counts [E] int, zeroed here; x [N, x_stride] in `dtype`; wr [E, W] 32-bit.
// score: 0 sigmoid, 1 softmax over all experts, 2 the logits with softmax over the chosen (`bias` [E] 32-bit or null is added to
// the logits; modes 1 and 2).  With `unit_gate` [N] wr has one row more, whose product's sigmoid goes there.
// E counts identities too; `real` of them have matrices (and counts).  `correction` [E] or null, `groups` (0: none) of which `keep`
// are chosen from, `scale` on the weights: see MoeChoice.
ZAI_API int zai_moe_route(int* ids, float* wts, int* rank, int* counts, const void* x, int x_stride, int dtype, const float* wr,
                          int N, int W, int E, int top, int renorm, int score, const float* bias, float* unit_gate,
                          const float* correction, int groups, int keep, int real, float scale, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    const MoeChoice choice = {correction, groups, keep, real, scale};
    if (real < 1 || real > E || groups < 0 || (groups && (E % groups || keep < 1 || keep > groups || (long long)keep * (E / groups) < top))
        || (score == MOE_LOGITS && (choice.own() || scale != 1.f)) || (choice.own() && E > 4096)) return ZAI_BAD_SIZE;
    if (E < 1 || top < 1 || top > E || top > 32 || E > 8192 || W < 1 || score < MOE_SIGMOID || score > MOE_LOGITS || (bias && score == MOE_SIGMOID)) return ZAI_BAD_SIZE;
    cudaError_t rc = cudaMemsetAsync(counts, 0, (size_t)real * sizeof(int), stream);
    if (rc != cudaSuccess) return (int)rc;
    const int rows = E + (unit_gate ? 1 : 0);
    const size_t smem = (size_t)(E + (choice.own() ? E + groups : 0)) * sizeof(float);      // a row's scores and choice values
    if (N >= 512 && 4 * smem <= 32 * 1024) {
        ZAI_DISPATCH(dtype, return launch_pdl(moe_route_kernel<T, 4>, dim3((N + 3) / 4), dim3(rows <= 4 ? 128 : 256), 4 * smem,
                                              stream, ids, wts, rank, counts, (const T*)x, x_stride, wr, N, W, E, top, renorm, score, bias, unit_gate,
                                              choice));
    }
    const int warps = rows < 4 ? 4 : rows > 16 ? 16 : rows;
    ZAI_DISPATCH(dtype, return launch_pdl(moe_route_kernel<T, 1>, dim3(N), dim3(warps * 32), smem, stream, ids, wts,
                                          rank, counts, (const T*)x, x_stride, wr, N, W, E, top, renorm, score, bias, unit_gate, choice));
}

// The most tiles of TM rows that N x top choices over E experts can take.
ZAI_API int zai_moe_max_tiles(int N, int top, int E, int TM) {
    const long long items = (long long)N * top;
    const long long t = items / TM + (items < E ? items : E);
    return t > 0x7fffffff ? -1 : (int)t;
}

// xs [max_tiles * TM, W] in `dtype`; dest [N, top]; tile_expert [max_tiles]
ZAI_API int zai_moe_gather(void* xs, int* dest, int* tile_expert, const void* x, int x_stride, int dtype, const int* ids,
                           const float* wts, const int* rank, const int* counts, int N, int W, int E, int top, int TM, int max_tiles,
                           int scale_input, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    const long long items = (long long)N * top;
    if (items >= 0x7fffffff || (TM != 16 && TM != 64 && TM != 128) || (long long)max_tiles * TM >= (1 << 24)) return ZAI_BAD_SIZE;
    ZAI_DISPATCH(dtype, return launch_pdl(moe_gather_kernel<T>, dim3((unsigned)items + 1), dim3(128), 0, stream, (T*)xs, dest,
                                          tile_expert, (const T*)x, x_stride, ids, wts, rank, counts, (int)items, W, E, top, TM,
                                          max_tiles, scale_input));
}

template <int TM, int TN, typename TO>
static int moe_launch_mma(dim3 grid, TO* out, const bf16* xs, const bf16* w, const int* tile_expert, int K, int n_out, int gated,
                          const MoeAct& act, cudaStream_t stream) {
    static unsigned long long done = 0;
    if (zai_first_on_device(&done)) {
        cudaError_t e = cudaFuncSetAttribute(moe_gemm_mma_kernel<TM, TN, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MoeTile<TM, TN>::BYTES);
        if (e != cudaSuccess) return (int)e;
    }
    return launch_pdl(moe_gemm_mma_kernel<TM, TN, TO>, grid, dim3(MoeTile<TM, TN>::WARPS * 32), MoeTile<TM, TN>::BYTES, stream, out, xs, w, tile_expert, K, n_out, gated, act);
}

// out [max_tiles * TM, n_out] (32-bit if out_f32, else `dtype`) = xs [max_tiles * TM, K] . w[expert of the tile]^T;
// w [E, n_out, K], or with kind 1 or 2 [E, 2 n_out, K] and out = silu(gate) * up (kind 1) or the bounded gated activation with
// `limit` and `alpha` (kind 2); kind 3: the square of relu on the plain products.  TM 16 or 64 (the gather's).
ZAI_API int zai_moe_gemm(void* out, int out_f32, const void* xs, const void* w, int dtype, const int* tile_expert, int max_tiles,
                         int TM, int K, int n_out, int kind, float limit, float alpha, cudaStream_t stream) {
    if (max_tiles <= 0) return ZAI_OK;
    if (kind < 0 || kind > 3) return ZAI_BAD_SIZE;
    const MoeAct act = {kind, limit, alpha};
    const int gated = kind == 1 || kind == 2;
    if (K < 1 || n_out < 1 || (TM != 16 && TM != 64)) return ZAI_BAD_SIZE;
    const bool mma = dtype == ZAI_BF16 && K % 8 == 0;
    const auto blocks_of = [&](int tn) { const int cols = gated ? tn / 2 : tn; return (n_out + cols - 1) / cols; };
    const bool wide = !mma || TM == 64 || (long long)max_tiles * blocks_of(64) >= MOE_WIDE_BLOCKS;
    const dim3 grid(max_tiles, blocks_of(wide ? 64 : 32));
    if (grid.y > 65535) return ZAI_BAD_SIZE;
    if (mma) {
#define MOE_GO(TMV, TNV, TOV) return moe_launch_mma<TMV, TNV, TOV>(grid, (TOV*)out, (const bf16*)xs, (const bf16*)w, tile_expert, K, n_out, gated, act, stream)
        if (TM == 64) { if (out_f32) MOE_GO(64, 64, float); else MOE_GO(64, 64, bf16); }
        if (wide) { if (out_f32) MOE_GO(16, 64, float); else MOE_GO(16, 64, bf16); }
        if (out_f32) MOE_GO(16, 32, float); else MOE_GO(16, 32, bf16);
#undef MOE_GO
    }
    if (TM != 16) return ZAI_BAD_SIZE;                   // the plain kernel's tiles are 16 rows high
    if (dtype == ZAI_BF16) {
        if (out_f32) return launch_pdl(moe_gemm_plain_kernel<bf16, float>, grid, dim3(128), 0, stream, (float*)out, (const bf16*)xs,
                                       (const bf16*)w, tile_expert, K, n_out, gated, act);
        return launch_pdl(moe_gemm_plain_kernel<bf16, bf16>, grid, dim3(128), 0, stream, (bf16*)out, (const bf16*)xs, (const bf16*)w,
                          tile_expert, K, n_out, gated, act);
    }
    if (dtype != ZAI_F32) return ZAI_BAD_DTYPE;
    return launch_pdl(moe_gemm_plain_kernel<float, float>, grid, dim3(128), 0, stream, (float*)out, (const float*)xs, (const float*)w,
                      tile_expert, K, n_out, gated, act);
}

// out [N, W] in `dtype` = sum over a row's choices of y[dest], times the choice's weight with `scale_output`; plus, with `unit`
// [N, W] in `dtype`, that row times unit_gate[row] (32-bit; null: times 1).  A choice with dest < 0 gives its weight times the
// row of x (may be null where there is none).  With `h` [N, W] 32-bit: h += that sum + other (or null), out (or null) = h rounded.
ZAI_API int zai_moe_combine(void* out, int dtype, const float* y, const int* dest, const float* wts, int N, int W, int top,
                            int scale_output, const void* unit, const float* unit_gate, const void* x, int x_stride, float* h,
                            const void* other, cudaStream_t stream) {
    if (N <= 0) return ZAI_OK;
    if (!out && !h) return ZAI_BAD_SIZE;
    ZAI_DISPATCH(dtype, const MoeBeside<T> a = {(const T*)unit, unit_gate, (const T*)x, x_stride, h, (const T*)other};
                 return launch_pdl(moe_combine_kernel<T>, dim3(N), dim3(W >= 1024 ? 256 : 128), 0, stream, (T*)out, y, dest, wts, W, top,
                                   scale_output, a));
}
