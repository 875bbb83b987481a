// Time mixing with a decay per key channel (the WKV recurrence of RWKV-6). Per head, with a bonus u for the current token:
//
//     o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t,      S_t = diag(w_t) S_(t-1) + k_t v_t^T
//
// where w_t = exp(-exp(z_t + w0)), z_t a low-rank projection W2 tanh(.) of the token. Rows arrive in bf16 or in 32-bit (as
// planes that are summed in order); everything else is 32-bit.
//   k_token_mix   the inputs of the projections: every stream's own mix of a row and the row before it
//   k_tanh_rows   tanh of the low-rank projection's rows
//   k_wkv_scan    token by token, for single tokens, short steps and the true 32-bit path: a warp per state column
//   k_wkv_state   for long prompts: what every run of WR_C tokens adds to the state, all runs side by side
//   k_wkv_prefix  the states at the starts of the runs, in order
//   k_wkv_out     the outputs of every run from the state at its start and from its own tokens
// A run is cut into pieces of WR_P tokens. With l = log w, every decay between two places is the exponential of a sum of l
// over the tokens between them, and the sums are put together from sums inside pieces (from a piece's start to a token, from
// a token to its end, over whole pieces): all terms have one sign, nothing is subtracted, and no exponent is above zero.
// Inside a piece the scores are plain 32-bit sums in which the decay is carried along as a running product. Between pieces,
// to and from the state they are tensor-core products (mma.sync): r, k and v are bf16 rows, and every 32-bit operand (the
// decayed r and k, the state, the scores) enters as a sum of three bf16 numbers, so that the products carry 24 bits.
// The state is kept per cache slot as [H][dv][d]. Rows of a step that belong to no sequence (padding of a recorded step) are
// not touched; their mixes are zeros.
#include "sm100.cuh"
#include "mma_sync.cuh"
#include "runs.cuh"
#include <math.h>

// an element that came either as it is or as 32-bit planes whose sum (in order) it is
template <typename T>
__device__ __forceinline__ float wk_rd(const T* p, int n_planes, size_t plane_stride) {
    float v = kb_to_f<T>(p[0]);
    for (int s = 1; s < n_planes; s++) v += kb_to_f<T>(p[(size_t)s * plane_stride]);
    return v;
}

// ------------------------------------------------------------------------------------------------ token mix
// out[t][s][c] = y[t][c] + (y'[c] - y[t][c]) * mu[s][c], y' the row before: inside a step the step's own, for the first row
// of a sequence's share of the step what its last step left in `last` (zeros when the sequence starts). The thread that
// reads `last` for a column also writes the column of the share's last row there. V neighbouring columns a thread.
template <typename T, int V>
__global__ void __launch_bounds__(256) k_token_mix(const T* KB_STEP_DATA y, int E, const float* __restrict__ mu, int n,
        const int* __restrict__ pos, const int* __restrict__ seq, const int* __restrict__ slot,
        const int* __restrict__ q_start, float* last, size_t last_stride, T* __restrict__ out, int ldo) {
    kb_pdl_launch();
    const int t = blockIdx.x, c = (blockIdx.y * 256 + threadIdx.x) * V;
    const int p = pos[t], b = seq[t];
    const int r0 = q_start[b], r1 = q_start[b + 1];
    const int sl = slot[b];
    kb_pdl_wait();
    if (c >= E) return;
    struct __align__(V * sizeof(T)) Pack { T v[V]; };
    Pack o;
    T* dst = out + (size_t)t * ldo + c;
    if (p < 0) {
#pragma unroll
        for (int i = 0; i < V; i++) o.v[i] = kb_from_f<T>(0.0f);
        for (int s = 0; s < n; s++) *(Pack*)(dst + (size_t)s * E) = o;
        return;
    }
    const Pack cur = *(const Pack*)(y + (size_t)t * E + c);
    float x[V], d[V];
    if (t == r0) {
        float* lp = last + (size_t)sl * last_stride + c;
        const Pack nl = *(const Pack*)(y + (size_t)(r1 - 1) * E + c);
#pragma unroll
        for (int i = 0; i < V; i++) {
            x[i] = kb_to_f<T>(cur.v[i]);
            d[i] = lp[i] - x[i];
            lp[i] = kb_to_f<T>(nl.v[i]);
        }
    } else {
        const Pack pv = *(const Pack*)(y + (size_t)(t - 1) * E + c);
#pragma unroll
        for (int i = 0; i < V; i++) {
            x[i] = kb_to_f<T>(cur.v[i]);
            d[i] = kb_to_f<T>(pv.v[i]) - x[i];
        }
    }
#pragma unroll 5
    for (int s = 0; s < n; s++) {
        float m[V];
        if (V % 4 == 0) {
#pragma unroll
            for (int i = 0; i < V; i += 4) *(float4*)(m + i) = __ldg((const float4*)(mu + (size_t)s * E + c + i));
        } else {
#pragma unroll
            for (int i = 0; i < V; i++) m[i] = mu[(size_t)s * E + c + i];
        }
#pragma unroll
        for (int i = 0; i < V; i++) o.v[i] = kb_from_f<T>(fmaf(d[i], m[i], x[i]));
        *(Pack*)(dst + (size_t)s * E) = o;
    }
}

// y [T][E] contiguous, out [T][ldo] with the n mixes side by side, mu [n][E]
extern "C" int kb_token_mix(const void* y, int dtype, int E, const float* mu, int n, const int* pos, const int* seq,
                            const int* slot, const int* q_start, float* last, long long last_stride, void* out, int ldo, int T,
                            cudaStream_t st) {
    if (T <= 0 || n <= 0) return 0;
    const int el = dtype == KB_F32 ? 4 : 2;
    const int v = dtype == KB_F32 ? 4 : 8;
    const bool vec = E % v == 0 && ldo % v == 0 && (uintptr_t)y % (v * el) == 0 && (uintptr_t)out % (v * el) == 0 &&
                     (uintptr_t)mu % 16 == 0;
#define TM_GO(TT, V)                                                                                                   \
    kb_launch(k_token_mix<TT, V>, dim3(T, (E + 256 * V - 1) / (256 * V)), 256, 0, st, \
              (const TT*)y, E, mu, n, pos, seq, slot, q_start, last, (size_t)last_stride, (TT*)out, ldo)
    if (dtype == KB_F32) {
        if (vec) TM_GO(float, 4); else TM_GO(float, 1);
    } else {
        if (vec) TM_GO(bf16, 8); else TM_GO(bf16, 1);
    }
#undef TM_GO
    KB_LAUNCH_RET();
}

// ------------------------------------------------------------------------------------------------ tanh
template <typename TIN, typename T>
__global__ void __launch_bounds__(256) k_tanh_rows(const TIN* KB_STEP_DATA a, int n_planes, size_t plane_stride, int lda,
                                                   T* __restrict__ out, int N, long long n) {
    kb_pdl_launch();
    kb_pdl_wait();
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i >= n) return;
    out[i] = kb_from_f<T>(tanhf(wk_rd<TIN>(a + (i / N) * lda + i % N, n_planes, plane_stride)));
}

extern "C" int kb_tanh_rows(const void* a, int adtype, int n_planes, long long plane_stride, int lda, void* out, int dtype, int T,
                            int N, cudaStream_t st) {
    const long long n = (long long)T * N;
    if (n <= 0) return 0;
    const unsigned grid = (unsigned)((n + 255) / 256);
#define TR_GO(TIN, TO)                                                                                                 \
    kb_launch(k_tanh_rows<TIN, TO>, grid, 256, 0, st, (const TIN*)a, n_planes, (size_t)plane_stride, lda, (TO*)out, N, n)
    if (adtype == KB_F32 && dtype == KB_F32) TR_GO(float, float);
    else if (adtype == KB_F32) TR_GO(float, bf16);
    else if (dtype == KB_BF16) TR_GO(bf16, bf16);
    else return (int)cudaErrorInvalidValue;
#undef TR_GO
    KB_LAUNCH_RET();
}

// ------------------------------------------------------------------------------------------------ token by token
struct WkvArgs {
    const void* r;              // [.., T, ld] each: head h's elements at columns h d (r, k) and h dv (v)
    const void* k;
    const void* v;
    int n_planes;
    size_t plane_stride;
    int ld;
    // the decay's exponent z: finished rows (z [T][ldz]), or the low-rank projection's planes (low) with W2 [H d][rank]
    const float* z;
    int ldz;
    const void* low;
    int low_planes;
    size_t low_stride;
    int ld_low;
    const void* w2;
    int rank;
    const float* w0;            // [H d]
    const float* u;             // [H d]
    int B, H, d, dv;
    const int* q_start;
    const int* slot;
    float* state;               // [slots][H][dv][d]
    size_t state_stride;
    float* out;                 // [T][ldo]
    int ldo;
};

// a channel's decay from its exponent
__device__ __forceinline__ float wk_decay(float z) { return expf(-expf(z)); }

// A block works one (sequence, head) and WK_COLS * NC columns of the state, a warp NC columns with the d key channels over
// the lanes; tokens are staged WK_STAGE at a time.
#define WK_COLS 8
#define WK_STAGE 16
template <typename T, typename TW, int DPL, int NC>
__global__ void __launch_bounds__(32 * WK_COLS, DPL * NC > 16 ? 2 : 3) k_wkv_scan(WkvArgs a) {
    extern __shared__ float sm[];
    constexpr int COLS = WK_COLS * NC;
    const int d = a.d, dv = a.dv, H = a.H;
    float* rs = sm;                                   // [WK_STAGE][d]
    float* ks = rs + WK_STAGE * d;                    // [WK_STAGE][d]
    float* ws = ks + WK_STAGE * d;                    // [WK_STAGE][d]: decays
    float* vs = ws + WK_STAGE * d;                    // [WK_STAGE][COLS]
    float* lo = vs + WK_STAGE * COLS;                 // [WK_STAGE][rank]: tanh of the low-rank projection
    kb_pdl_launch();
    const int b = blockIdx.x / H, h = blockIdx.x % H;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int e0 = blockIdx.y * COLS, e = e0 + warp;   // this warp's columns: e, e + WK_COLS, ...
    const int r0 = a.q_start[b], r1 = a.q_start[b + 1];
    float* srow = a.state + (size_t)a.slot[b] * a.state_stride + (size_t)h * dv * d;
    // (left by earlier steps, which are complete before this step's first kernel starts)
    float S[NC][DPL], uu[DPL];
#pragma unroll
    for (int i = 0; i < DPL; i++) {
        const int j = lane + 32 * i;
        uu[i] = j < d ? a.u[(size_t)h * d + j] : 0.0f;
#pragma unroll
        for (int c = 0; c < NC; c++) {
            const int ec = e + c * WK_COLS;
            S[c][i] = (ec < dv && j < d) ? srow[(size_t)ec * d + j] : 0.0f;
        }
    }
    kb_pdl_wait();
    const size_t ok = (size_t)h * d, ov = (size_t)h * dv;
    const bool w2_vec = a.rank % 8 == 0 && ((uintptr_t)a.w2 & 15) == 0;
    for (int c0 = r0; c0 < r1; c0 += WK_STAGE) {
        const int n = min(WK_STAGE, r1 - c0);
        if (a.z == nullptr) {
            for (int idx = threadIdx.x; idx < n * a.rank; idx += 32 * WK_COLS) {
                const int t = idx / a.rank, q = idx % a.rank;
                lo[idx] = tanhf(wk_rd<T>((const T*)a.low + (size_t)(c0 + t) * a.ld_low + q, a.low_planes, a.low_stride));
            }
            __syncthreads();
        }
        for (int idx = threadIdx.x; idx < n * d; idx += 32 * WK_COLS) {
            const int t = idx / d, j = idx % d;
            const size_t at = (size_t)(c0 + t) * a.ld + ok + j;
            rs[idx] = wk_rd<T>((const T*)a.r + at, a.n_planes, a.plane_stride);
            ks[idx] = wk_rd<T>((const T*)a.k + at, a.n_planes, a.plane_stride);
            if (a.z != nullptr) ws[idx] = wk_decay(a.z[(size_t)(c0 + t) * a.ldz + ok + j] + a.w0[ok + j]);
        }
        if (a.z == nullptr) {
            // the exponent from the low-rank projection: four lanes a channel, a quarter of the sum each (the bound is rounded
            // up so that whole warps meet at the exchange)
            for (int i4 = threadIdx.x; i4 < (n * d * 4 + 31) / 32 * 32; i4 += 32 * WK_COLS) {
                const int idx = min(i4 >> 2, n * d - 1), sub = i4 & 3, t = idx / d, j = idx % d;
                const TW* w = (const TW*)a.w2 + (ok + j) * a.rank;
                const float* l = lo + t * a.rank;
                float z = 0.0f;
                if (sizeof(TW) == 2 && w2_vec) {
                    for (int q = sub * 8; q < a.rank; q += 32) {
                        const uint4 v = *(const uint4*)(w + q);
                        const __nv_bfloat162* v2 = (const __nv_bfloat162*)&v;
#pragma unroll
                        for (int e = 0; e < 4; e++) {
                            const float2 f = __bfloat1622float2(v2[e]);
                            z = fmaf(l[q + 2 * e], f.x, z);
                            z = fmaf(l[q + 2 * e + 1], f.y, z);
                        }
                    }
                } else {
                    for (int q = sub; q < a.rank; q += 4) z = fmaf(l[q], kb_to_f<TW>(w[q]), z);
                }
                z += __shfl_xor_sync(0xffffffffu, z, 1);
                z += __shfl_xor_sync(0xffffffffu, z, 2);
                if (sub == 0 && i4 < n * d * 4) ws[idx] = wk_decay(z + a.w0[ok + j]);
            }
        }
        for (int idx = threadIdx.x; idx < n * COLS; idx += 32 * WK_COLS) {
            const int t = idx / COLS, c = e0 + idx % COLS;
            vs[idx] = c < dv ? wk_rd<T>((const T*)a.v + (size_t)(c0 + t) * a.ld + ov + c, a.n_planes, a.plane_stride) : 0.0f;
        }
        __syncthreads();
        for (int t = 0; t < n; t++) {
            float v[NC], o[NC];
#pragma unroll
            for (int c = 0; c < NC; c++) {
                v[c] = vs[t * COLS + c * WK_COLS + warp];
                o[c] = 0.0f;
            }
#pragma unroll
            for (int i = 0; i < DPL; i++) {
                const int j = lane + 32 * i;
                if (j < d) {
                    const float k = ks[t * d + j], r = rs[t * d + j], w = ws[t * d + j];
                    const float uk = __fmul_rn(uu[i], k);
#pragma unroll
                    for (int c = 0; c < NC; c++) {
                        o[c] = fmaf(fmaf(uk, v[c], S[c][i]), r, o[c]);
                        S[c][i] = fmaf(k, v[c], __fmul_rn(w, S[c][i]));
                    }
                }
            }
#pragma unroll
            for (int c = 0; c < NC; c++) o[c] = kb_warp_sum(o[c]);
#pragma unroll
            for (int c = 0; c < NC; c++) {
                const int ec = e + c * WK_COLS;
                if (lane == 0 && ec < dv) a.out[(size_t)(c0 + t) * a.ldo + ov + ec] = o[c];
            }
        }
        __syncthreads();
    }
    if (r1 > r0) {
#pragma unroll
        for (int c = 0; c < NC; c++)
#pragma unroll
            for (int i = 0; i < DPL; i++) {
                const int j = lane + 32 * i, ec = e + c * WK_COLS;
                if (ec < dv && j < d) srow[(size_t)ec * d + j] = S[c][i];
            }
    }
}

// ------------------------------------------------------------------------------------------------ runs of long prompts
#define WR_C 64                 // tokens of a run
#define WR_P 16                 // tokens of a piece
#define WR_E 64                 // state columns (values) of a block
#define WR_LD 72                // row of a 64-wide bf16 tile in shared memory
#define WR_SLD 72               // row of the 32-bit score tile
#define WR_THREADS 256
// All tiles have DP channels, the head's size rounded up to 16: channels from d on hold zeros.
// vec, bit 0: rows of r, k and v may be read in 16-byte words; bit 1: the output is written in pairs; bit 2: z, w0 and the
// states are read in 16-byte words

__device__ __forceinline__ float wr_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// a block's [WR_C][cols] tile of bf16 rows; columns from d to DP and rows from n on are zero. Whole 16-byte words go by
// asynchronous copies: the caller waits for them before its barrier
template <int DP>
__device__ __forceinline__ void wr_tile(bf16* dst, int dst_ld, const bf16* src, int ld, int n, int d, bool vec) {
    if (vec) {
#pragma unroll
        for (int idx = threadIdx.x; idx < WR_C * (DP / 8); idx += WR_THREADS) {
            const int t = idx / (DP / 8), c = (idx % (DP / 8)) * 8;
            const bool ok = t < n && c < d;
            cp_async16(smem_u32(dst + t * dst_ld + c), ok ? (const void*)(src + (size_t)t * ld + c) : (const void*)src, ok);
        }
        return;
    }
    for (int idx = threadIdx.x; idx < WR_C * DP; idx += WR_THREADS) {
        const int t = idx / DP, c = idx % DP;
        dst[t * dst_ld + c] = (t < n && c < d) ? src[(size_t)t * ld + c] : __float2bfloat16_rn(0.0f);
    }
}
// log2 w = -log2(e) exp(z + w0) of a run's tokens, [WR_C][ld] floats; rows from n on and channels from d on: 0
template <int DP>
__device__ __forceinline__ void wr_logs(float* dst, int ld, const WkvArgs& a, int r0, int n, int h, bool vec) {
    const float* z = a.z + (size_t)r0 * a.ldz + (size_t)h * a.d;
    const float* w0 = a.w0 + (size_t)h * a.d;
    constexpr float L2E = -1.4426950408889634f;
    if (vec) {
        constexpr int PER = WR_C * (DP / 4), N = (PER + WR_THREADS - 1) / WR_THREADS;
        float4 v[N];
#pragma unroll
        for (int i = 0; i < N; i++) {
            const int idx = threadIdx.x + i * WR_THREADS, t = idx / (DP / 4), j = (idx % (DP / 4)) * 4;
            v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (idx < PER && t < n && j < a.d) v[i] = *(const float4*)(z + (size_t)t * a.ldz + j);
        }
#pragma unroll
        for (int i = 0; i < N; i++) {
            const int idx = threadIdx.x + i * WR_THREADS, t = idx / (DP / 4), j = (idx % (DP / 4)) * 4;
            if (idx >= PER) continue;
            const bool on = t < n && j < a.d;
            const float4 b = j < a.d ? *(const float4*)(w0 + j) : make_float4(0.f, 0.f, 0.f, 0.f);
            float2* p = (float2*)(dst + t * ld + j);
            p[0] = on ? make_float2(L2E * expf(v[i].x + b.x), L2E * expf(v[i].y + b.y)) : make_float2(0.f, 0.f);
            p[1] = on ? make_float2(L2E * expf(v[i].z + b.z), L2E * expf(v[i].w + b.w)) : make_float2(0.f, 0.f);
        }
        return;
    }
    for (int idx = threadIdx.x; idx < WR_C * DP; idx += WR_THREADS) {
        const int t = idx / DP, j = idx % DP;
        dst[t * ld + j] = (t < n && j < a.d) ? L2E * expf(z[(size_t)t * a.ldz + j] + w0[j]) : 0.0f;
    }
}
// a 32-bit pair as three bf16 pairs, one per plane of a split tile
__device__ __forceinline__ void wr_put_split(bf16* tile, int plane, int at, float x, float y) {
    uint32_t p[KB_SPLIT];
    split_pack_bf16(x, y, p);
#pragma unroll
    for (int u = 0; u < KB_SPLIT; u++) *(uint32_t*)(tile + u * plane + at) = p[u];
}
// channels j, j + 1 of a bf16 row in global memory (zeros where off)
__device__ __forceinline__ float2 wr_pair(const bf16* row, int j, int d, bool on, bool vec) {
    if (!on || j >= d) return make_float2(0.f, 0.f);
    if (vec) return __bfloat1622float2(*(const __nv_bfloat162*)(row + j));
    return make_float2(__bfloat162float(row[j]), j + 1 < d ? __bfloat162float(row[j + 1]) : 0.0f);
}

template <int DP>
struct WrSmem {
    static constexpr int KLD = DP + 8, WLD = DP + 2, RLD = DP + 8;
    static constexpr int KPLANE = WR_C * KLD, SPLANE = WR_E * WR_LD;
    // k_wkv_state: split keys, values, keys, logs, sums over pieces
    static constexpr int STATE = (KB_SPLIT * KPLANE + WR_C * WR_LD + KPLANE) * 2 + (WR_C * WLD + 4 * DP) * 4;
    // k_wkv_out: split keys (later the state's tile), keys, values, logs / decays, decayed r, tables, scores in two parts
    static constexpr int USZ = KB_SPLIT * (KPLANE > SPLANE ? KPLANE : SPLANE);
    static constexpr int OUT = (USZ + KPLANE + WR_C * WR_LD) * 2 +
                               (WR_C * WLD + WR_C * RLD + 8 * DP + WR_C * WR_SLD + WR_C * (WR_P + 2)) * 4;
};

// part [runs][H][dv][d]: sum over the run's tokens of (decay from the token to the run's end) k_s v_s^T; keep [runs][H][d]:
// the decay over the whole run. grid (runs, H, ceil(dv / WR_E))
template <int DP>
__global__ void __launch_bounds__(WR_THREADS) k_wkv_state(WkvArgs a, float* __restrict__ part, float* __restrict__ keep, int vec) {
    using S = WrSmem<DP>;
    extern __shared__ __align__(16) uint8_t sm8[];
    bf16* kw = (bf16*)sm8;                             // [KB_SPLIT][WR_C][KLD]: the decayed keys
    bf16* vs = kw + KB_SPLIT * S::KPLANE;              // [WR_C][WR_LD]
    bf16* ks = vs + WR_C * WR_LD;                      // [WR_C][KLD]
    float* lt = (float*)(ks + S::KPLANE);              // [WR_C][WLD]
    float* dsum = lt + WR_C * S::WLD;                  // [4][DP]: sums over pieces
    kb_pdl_launch();
    const KbRun r = kb_find_run(a.q_start, a.B, WR_C, blockIdx.x);
    kb_pdl_wait();
    if (r.n <= 0) return;
    const int h = blockIdx.y, e0 = blockIdx.z * WR_E;
    const int d = a.d, dv = a.dv;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int ne = min(WR_E, dv - e0);
    const size_t row0 = (size_t)r.r0 * a.ld;
    wr_tile<DP>(ks, S::KLD, (const bf16*)a.k + row0 + (size_t)h * d, a.ld, r.n, d, vec & 1);
    wr_tile<WR_E>(vs, WR_LD, (const bf16*)a.v + row0 + (size_t)h * dv + e0, a.ld, r.n, ne, (vec & 1) && ne % 8 == 0);
    wr_logs<DP>(lt, S::WLD, a, r.r0, r.n, h, vec & 4);
    cp_async_wait_all();
    __syncthreads();
    for (int idx = threadIdx.x; idx < 4 * DP; idx += WR_THREADS) {
        const int pc = idx / DP, j = idx % DP;
        float* p = lt + pc * WR_P * S::WLD + j;
        float l[WR_P], s = 0.0f;
#pragma unroll
        for (int i = 0; i < WR_P; i++) l[i] = p[i * S::WLD];
#pragma unroll
        for (int i = WR_P - 1; i >= 0; i--) {          // the sum behind a token, then over the piece
            p[i * S::WLD] = s;
            s += l[i];
        }
        dsum[idx] = s;
    }
    __syncthreads();
#pragma unroll
    for (int idx = threadIdx.x; idx < WR_C * (DP / 2); idx += WR_THREADS) {
        const int t = idx / (DP / 2), j = (idx % (DP / 2)) * 2;
        float2 x = *(const float2*)(lt + t * S::WLD + j);
        for (int c = t / WR_P + 1; c < 4; c++) {
            const float2 g = *(const float2*)(dsum + c * DP + j);
            x.x += g.x;
            x.y += g.y;
        }
        const float2 k2 = __bfloat1622float2(*(const __nv_bfloat162*)(ks + t * S::KLD + j));
        wr_put_split(kw, S::KPLANE, t * S::KLD + j, k2.x * wr_ex2(x.x), k2.y * wr_ex2(x.y));
    }
    if (blockIdx.z == 0)
        for (int j = threadIdx.x; j < d; j += WR_THREADS)
            keep[((size_t)blockIdx.x * a.H + h) * d + j] =
                wr_ex2(((dsum[j] + dsum[DP + j]) + dsum[2 * DP + j]) + dsum[3 * DP + j]);
    __syncthreads();
    float* pb = part + ((size_t)blockIdx.x * a.H + h) * dv * d;
    // this warp: 16 columns of the state against every other 16 of the channels
    const int m0 = (warp >> 1) * 16;
    if (m0 >= ne) return;
    uint32_t av[WR_C / 16][4];
#pragma unroll
    for (int k = 0; k < WR_C / 16; k++) {
        const int row = k * 16 + ((lane >> 4) & 1) * 8 + (lane & 7), col = m0 + ((lane >> 3) & 1) * 8;
        ldsm_x4_t(smem_u32(vs + row * WR_LD + col), av[k][0], av[k][1], av[k][2], av[k][3]);
    }
#pragma unroll 1
    for (int j0 = (warp & 1) * 16; j0 < DP; j0 += 32) {
        float acc[KB_SPLIT][2][4] = {};                // (a sum per part: chains of products that do not wait for one another)
#pragma unroll
        for (int k = 0; k < WR_C / 16; k++) {
            const int row = k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, col = j0 + (lane >> 4) * 8;
#pragma unroll
            for (int i = 0; i < KB_SPLIT; i++) {
                uint32_t bf[4];
                ldsm_x4_t(smem_u32(kw + i * S::KPLANE + row * S::KLD + col), bf[0], bf[1], bf[2], bf[3]);
                mma_bf16(acc[i][0], av[k], bf[0], bf[1]);
                mma_bf16(acc[i][1], av[k], bf[2], bf[3]);
            }
        }
#pragma unroll
        for (int u = 0; u < 2; u++) {
            const int j = j0 + u * 8 + (lane & 3) * 2;
#pragma unroll
            for (int hf = 0; hf < 2; hf++) {
                const int e = e0 + m0 + (lane >> 2) + hf * 8;
                if (e >= dv) continue;
                const float x = (acc[2][u][2 * hf] + acc[1][u][2 * hf]) + acc[0][u][2 * hf];
                const float y = (acc[2][u][2 * hf + 1] + acc[1][u][2 * hf + 1]) + acc[0][u][2 * hf + 1];
                float* p = pb + (size_t)e * d + j;
                if (j + 1 < d && !(d & 1)) *(float2*)p = make_float2(x, y);
                else {
                    if (j < d) p[0] = x;
                    if (j + 1 < d) p[1] = y;
                }
            }
        }
    }
}

// part[run] <- the state at the run's start; the sequence's state <- the state after its last run. A thread per VW
// neighbouring elements of a (sequence, head), four runs' loads in flight. grid (ceil(elements / (256 VW)), H, B)
template <int VW>
__global__ void __launch_bounds__(256) k_wkv_prefix(WkvArgs a, float* part, const float* KB_STEP_DATA keep) {
    kb_pdl_launch();
    const int h = blockIdx.y, b = blockIdx.z, d = a.d, n_el = a.dv * a.d;
    const int s0 = a.q_start[b], len = a.q_start[b + 1] - s0;
    const int nr = (len + WR_C - 1) / WR_C, run0 = s0 / WR_C + b;
    const size_t at = ((size_t)blockIdx.x * 256 + threadIdx.x) * VW;
    kb_pdl_wait();
    if (at >= (size_t)n_el || nr <= 0) return;
    typedef typename std::conditional<VW == 4, float4, float>::type V;
    float* st = a.state + (size_t)a.slot[b] * a.state_stride + (size_t)h * n_el + at;
    const size_t step = (size_t)a.H * n_el, kstep = (size_t)a.H * d;
    float* p = part + (size_t)run0 * step + (size_t)h * n_el + at;
    const float* kp = keep + (size_t)run0 * kstep + (size_t)h * d + at % d;
    V S = *(const V*)st;
    float* Sf = (float*)&S;
    for (int c0 = 0; c0 < nr; c0 += 4) {
        V x[4], g[4];
#pragma unroll
        for (int k = 0; k < 4; k++)
            if (c0 + k < nr) {
                x[k] = *(const V*)(p + (size_t)(c0 + k) * step);
                g[k] = *(const V*)(kp + (size_t)(c0 + k) * kstep);
            }
#pragma unroll
        for (int k = 0; k < 4; k++)
            if (c0 + k < nr) {
                *(V*)(p + (size_t)(c0 + k) * step) = S;
                const float* xf = (const float*)&x[k], *gf = (const float*)&g[k];
#pragma unroll
                for (int i = 0; i < VW; i++) Sf[i] = fmaf(gf[i], Sf[i], xf[i]);
            }
    }
    *(V*)st = S;
}

// 16 rows x 16 columns of a 32-bit tile (the sum of two, where there is a second), times a factor per column, as the A
// operand of a product, in three bf16 parts
__device__ __forceinline__ void wr_frag(const float* tile, int ld, const float* more, int ld2, int c0, const float* f, int lane,
                                        uint32_t (&s)[KB_SPLIT][4]) {
#pragma unroll
    for (int q = 0; q < 4; q++) {
        const int row = (lane >> 2) + (q & 1) * 8, c = (lane & 3) * 2 + (q >> 1) * 8;
        float2 v = *(const float2*)(tile + row * ld + c0 + c);
        if (more != nullptr) {
            const float2 w = *(const float2*)(more + row * ld2 + c);
            v.x += w.x;
            v.y += w.y;
        }
        if (f != nullptr) {
            const float2 g = *(const float2*)(f + c0 + c);
            v.x *= g.x;
            v.y *= g.y;
        }
        uint32_t p[KB_SPLIT];
        split_pack_bf16(v.x, v.y, p);
#pragma unroll
        for (int u = 0; u < KB_SPLIT; u++) s[u][q] = p[u];
    }
}
// c += A B of two split operands (16 columns of B: two tiles), the six products that carry 24 bits, small ones first
__device__ __forceinline__ void wr_mma6(float (&c)[2][4], const uint32_t (&a)[KB_SPLIT][4], const uint32_t (&b)[KB_SPLIT][4]) {
#pragma unroll
    for (int x = KB_SPLIT - 1; x >= 0; x--)
#pragma unroll
        for (int i = x; i >= 0; i--)
#pragma unroll
            for (int u = 0; u < 2; u++) mma_bf16(c[u], a[i], b[x - i][2 * u], b[x - i][2 * u + 1]);
}

// grid (runs, H, ceil(dv / WR_E)); two warps work the 16 tokens of a piece, each against half of the block's state columns
template <int DP>
__global__ void __launch_bounds__(WR_THREADS, DP <= 64 ? 2 : 1) k_wkv_out(WkvArgs a, const float* KB_STEP_DATA part, int vec) {
    using S = WrSmem<DP>;
    extern __shared__ __align__(16) uint8_t sm8[];
    bf16* kw = (bf16*)sm8;                             // [KB_SPLIT][WR_C][KLD]: keys decayed to their piece's end; later
    bf16* ss = kw;                                     // [KB_SPLIT][WR_E][WR_LD]: 64 channels of the state's columns
    bf16* ks = kw + S::USZ;                            // [WR_C][KLD]
    bf16* vs = ks + S::KPLANE;                         // [WR_C][WR_LD]
    float* wt = (float*)(vs + WR_C * WR_LD);           // [WR_C][WLD]: log2 of the decays, then decays
    float* rh = wt + WR_C * S::WLD;                    // [WR_C][RLD]: r decayed from its piece's start
    float* tab = rh + WR_C * S::RLD;                   // [8][DP]: sums over pieces; decays between pieces
    float* sc = tab + 8 * DP;                          // [WR_C][WR_SLD]: scores
    float* sc2 = sc + WR_C * WR_SLD;                   // [WR_C][WR_P + 2]: the other half's share of the scores inside a piece
    kb_pdl_launch();
    const KbRun r = kb_find_run(a.q_start, a.B, WR_C, blockIdx.x);
    kb_pdl_wait();
    if (r.n <= 0) return;
    const int h = blockIdx.y, e0 = blockIdx.z * WR_E;
    const int d = a.d, dv = a.dv;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int ne = min(WR_E, dv - e0);
    const size_t row0 = (size_t)r.r0 * a.ld;
    const bf16* rg = (const bf16*)a.r + row0 + (size_t)h * d;
    const float* S0 = part + (((size_t)blockIdx.x * a.H + h) * dv + e0) * d;
    wr_tile<DP>(ks, S::KLD, (const bf16*)a.k + row0 + (size_t)h * d, a.ld, r.n, d, vec & 1);
    wr_tile<WR_E>(vs, WR_LD, (const bf16*)a.v + row0 + (size_t)h * dv + e0, a.ld, r.n, ne, (vec & 1) && ne % 8 == 0);
    wr_logs<DP>(wt, S::WLD, a, r.r0, r.n, h, vec & 4);
    // a pair of channels of a piece a thread: half of the threads decay r from the piece's start, the others the keys to its end
    const int role = threadIdx.x >> 7;
    float2 rr[WR_P];
    const int u0 = threadIdx.x & 127;
    if (role == 0 && u0 < 2 * DP) {
        const int pc = u0 / (DP / 2), j = (u0 % (DP / 2)) * 2;
#pragma unroll
        for (int i = 0; i < WR_P; i++)
            rr[i] = wr_pair(rg + (size_t)(pc * WR_P + i) * a.ld, j, d, pc * WR_P + i < r.n, vec & 1);
    }
    // (and r as it is, with the bonuses, for the sums inside a piece further down)
    constexpr int NP = DP / 8;
    const int pa = warp >> 1, hf = warp & 1, t0 = pa * WR_P;
    const int ti = lane & 15, jl = hf * (DP / 2) + (lane >> 4) * 2;
    float2 p[NP], bonus[NP];
#pragma unroll
    for (int q = 0; q < NP; q++) {
        const int j = jl + 4 * q;
        p[q] = wr_pair(rg + (size_t)(t0 + ti) * a.ld, j, d, t0 + ti < r.n, vec & 1);
        bonus[q] = make_float2(j < d ? __ldg(a.u + (size_t)h * d + j) : 0.0f, j + 1 < d ? __ldg(a.u + (size_t)h * d + j + 1) : 0.0f);
    }
    cp_async_wait_all();
    __syncthreads();
#pragma unroll
    for (int u = u0; u < 2 * DP; u += 128) {
        const int pc = u / (DP / 2), j = (u % (DP / 2)) * 2;
        const float* lp = wt + pc * WR_P * S::WLD + j;
        float2 x = make_float2(0.f, 0.f);
        if (role == 0) {
#pragma unroll
            for (int i = 0; i < WR_P; i++) {
                const int t = pc * WR_P + i;
                const float2 l = *(const float2*)(lp + i * S::WLD);
                const float2 v = u == u0 ? rr[i] : wr_pair(rg + (size_t)t * a.ld, j, d, t < r.n, vec & 1);
                *(float2*)(rh + t * S::RLD + j) = make_float2(v.x * wr_ex2(x.x), v.y * wr_ex2(x.y));
                x.x += l.x;
                x.y += l.y;
            }
            *(float2*)(tab + pc * DP + j) = x;
        } else if (pc < 3) {                           // (the last piece's keys are only needed inside it)
#pragma unroll
            for (int i = WR_P - 1; i >= 0; i--) {
                const int t = pc * WR_P + i;
                const float2 l = *(const float2*)(lp + i * S::WLD);
                const float2 k2 = __bfloat1622float2(*(const __nv_bfloat162*)(ks + t * S::KLD + j));
                wr_put_split(kw, S::KPLANE, t * S::KLD + j, k2.x * wr_ex2(x.x), k2.y * wr_ex2(x.y));
                x.x += l.x;
                x.y += l.y;
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int idx = threadIdx.x; idx < WR_C * (DP / 2); idx += WR_THREADS) {
        float2* p = (float2*)(wt + idx / (DP / 2) * S::WLD + (idx % (DP / 2)) * 2);
        const float2 l = *p;
        *p = make_float2(wr_ex2(l.x), wr_ex2(l.y));
    }
    for (int j = threadIdx.x; j < DP; j += WR_THREADS) {
        const float d0 = tab[j], d1 = tab[DP + j], d2 = tab[2 * DP + j];
        // rows 0..2: the decay from the run's start to pieces 1, 2, 3; row 4: over piece 1, 5: over piece 2, 6: over both
        tab[j] = wr_ex2(d0);
        tab[DP + j] = wr_ex2(d0 + d1);
        tab[2 * DP + j] = wr_ex2((d0 + d1) + d2);
        tab[4 * DP + j] = wr_ex2(d1);
        tab[5 * DP + j] = wr_ex2(d2);
        tab[6 * DP + j] = wr_ex2(d1 + d2);
    }
    __syncthreads();
    // ---- scores inside the piece: lane = (token, half of this warp's channel pairs); the decay is carried along as a product
    {
        const int t = t0 + ti;
        const bool first = lane < 16;
        float own = 0.0f;
#pragma unroll
        for (int q = 0; q < NP; q++) {
            const int j = jl + 4 * q;
            const float2 k2 = __bfloat1622float2(*(const __nv_bfloat162*)(ks + t * S::KLD + j));
            own = fmaf(p[q].x * bonus[q].x, k2.x, own);
            own = fmaf(p[q].y * bonus[q].y, k2.y, own);
        }
        own += __shfl_xor_sync(0xffffffffu, own, 16);
        float* dst = hf ? sc2 + t * (WR_P + 2) : sc + t * WR_SLD + t0;
        if (first) dst[ti] = own;
        const bf16* kp = ks + t0 * S::KLD + jl;
        const float* wp = wt + t0 * S::WLD + jl;
#pragma unroll 3
        for (int i = 1; i < WR_P; i++) {
            // key ti - i; from the second on its decay over the token behind it comes in
            const int s = max(ti - i, 0);
            float a0 = 0.0f, a1 = 0.0f;
#pragma unroll
            for (int q = 0; q < NP; q++) {
                if (i > 1) {
                    const float2 w2 = *(const float2*)(wp + (s + 1) * S::WLD + 4 * q);
                    p[q].x *= w2.x;
                    p[q].y *= w2.y;
                }
                const float2 k2 = __bfloat1622float2(*(const __nv_bfloat162*)(kp + s * S::KLD + 4 * q));
                a0 = fmaf(p[q].x, k2.x, a0);
                a1 = fmaf(p[q].y, k2.y, a1);
            }
            a0 += a1;
            a0 += __shfl_xor_sync(0xffffffffu, a0, 16);
            // (a token's columns behind it are zeros, each written once)
            if (first) dst[ti >= i ? ti - i : WR_P + ti - i] = ti >= i ? a0 : 0.0f;
        }
    }
    // ---- scores between pieces: the pair's two warps take the earlier pieces in turn
    for (int b = hf; b < pa; b += 2) {
        const float* g = pa - b == 1 ? nullptr : tab + (b == 1 ? 5 : pa == 2 ? 4 : 6) * DP;
        float acc[2][4] = {};
#pragma unroll 2
        for (int k = 0; k < DP / 16; k++) {
            uint32_t ar[KB_SPLIT][4], bf[KB_SPLIT][4];
            const int row = b * 16 + (lane & 7) + (lane >> 4) * 8, col = k * 16 + ((lane >> 3) & 1) * 8;
#pragma unroll
            for (int i = 0; i < KB_SPLIT; i++)
                ldsm_x4(smem_u32(kw + i * S::KPLANE + row * S::KLD + col), bf[i][0], bf[i][1], bf[i][2], bf[i][3]);
            wr_frag(rh + t0 * S::RLD, S::RLD, nullptr, 0, k * 16, g, lane, ar);
            wr_mma6(acc, ar, bf);
        }
#pragma unroll
        for (int u = 0; u < 2; u++) {
            float* p = sc + (t0 + (lane >> 2)) * WR_SLD + b * 16 + u * 8 + (lane & 3) * 2;
            *(float2*)p = make_float2(acc[u][0], acc[u][1]);
            *(float2*)(p + 8 * WR_SLD) = make_float2(acc[u][2], acc[u][3]);
        }
    }
    // the state's columns, 64 channels at a time, on their way meanwhile
    constexpr int NS = WR_E * 16 / WR_THREADS;
    const bool s4 = (vec & 4) && ne == WR_E;
    float4 sv[NS];
    auto s_load = [&](int jb) {
#pragma unroll
        for (int i = 0; i < NS; i++) {
            const int idx = threadIdx.x + i * WR_THREADS, e = idx >> 4, j = jb + (idx & 15) * 4;
            sv[i] = j < d ? *(const float4*)(S0 + (size_t)e * d + j) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
    };
    if (s4) s_load(0);
    __syncthreads();
    // ---- the run's own tokens: a piece of keys at a time, scores times values
    float o[4][4] = {};
    for (int b = 0; b <= pa; b++) {
        uint32_t ps[KB_SPLIT][4];
        wr_frag(sc + t0 * WR_SLD, WR_SLD, b == pa ? sc2 + t0 * (WR_P + 2) : nullptr, WR_P + 2, b * 16, nullptr, lane, ps);
#pragma unroll
        for (int dp2 = 0; dp2 < 2; dp2++) {
            uint32_t bf[4];
            ldsm_x4_t(smem_u32(vs + (b * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * WR_LD + hf * 32 + dp2 * 16 + (lane >> 4) * 8),
                      bf[0], bf[1], bf[2], bf[3]);
#pragma unroll
            for (int i = KB_SPLIT - 1; i >= 0; i--)
#pragma unroll
                for (int u = 0; u < 2; u++) mma_bf16(o[2 * dp2 + u], ps[i], bf[2 * u], bf[2 * u + 1]);
        }
    }
    // ---- the state's share (the decayed keys' place is free)
#pragma unroll 1
    for (int jb = 0; jb < DP; jb += 64) {
        if (jb > 0) __syncthreads();                   // (the tile before has been read)
        if (s4) {
#pragma unroll
            for (int i = 0; i < NS; i++) {
                const int idx = threadIdx.x + i * WR_THREADS, e = idx >> 4, c = (idx & 15) * 4;
                uint32_t p[KB_SPLIT], q[KB_SPLIT];
                split_pack_bf16(sv[i].x, sv[i].y, p);
                split_pack_bf16(sv[i].z, sv[i].w, q);
#pragma unroll
                for (int u = 0; u < KB_SPLIT; u++) *(uint2*)(ss + u * S::SPLANE + e * WR_LD + c) = make_uint2(p[u], q[u]);
            }
            if (jb + 64 < DP) s_load(jb + 64);
        } else
            for (int idx = threadIdx.x; idx < WR_E * 32; idx += WR_THREADS) {
                const int e = idx >> 5, c = (idx & 31) * 2, j = jb + c;
                float x = 0.0f, y = 0.0f;
                if (e < ne) {
                    if (j < d) x = S0[(size_t)e * d + j];
                    if (j + 1 < d) y = S0[(size_t)e * d + j + 1];
                }
                wr_put_split(ss, S::SPLANE, e * WR_LD + c, x, y);
            }
        __syncthreads();
#pragma unroll 2
        for (int k = 0; k < (DP - jb < 64 ? DP - jb : 64) / 16; k++) {
            uint32_t ar[KB_SPLIT][4];
            wr_frag(rh + t0 * S::RLD, S::RLD, nullptr, 0, jb + k * 16, pa ? tab + (pa - 1) * DP : nullptr, lane, ar);
#pragma unroll
            for (int np = 0; np < 2; np++) {
                const int row = hf * 32 + np * 16 + (lane & 7) + (lane >> 4) * 8, col = k * 16 + ((lane >> 3) & 1) * 8;
                uint32_t bf[KB_SPLIT][4];
#pragma unroll
                for (int i = 0; i < KB_SPLIT; i++)
                    ldsm_x4(smem_u32(ss + i * S::SPLANE + row * WR_LD + col), bf[i][0], bf[i][1], bf[i][2], bf[i][3]);
                wr_mma6(*(float(*)[2][4])(o + 2 * np), ar, bf);
            }
        }
    }
#pragma unroll
    for (int n = 0; n < 4; n++) {
        const int c = hf * 32 + n * 8 + (lane & 3) * 2;
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int t = t0 + (lane >> 2) + half * 8;
            if (t >= r.n) continue;
            float* p = a.out + (size_t)(r.r0 + t) * a.ldo + (size_t)h * dv + e0 + c;
            if (c + 1 < ne && (vec & 2)) *(float2*)p = make_float2(o[n][2 * half], o[n][2 * half + 1]);
            else {
                if (c < ne) p[0] = o[n][2 * half];
                if (c + 1 < ne) p[1] = o[n][2 * half + 1];
            }
        }
    }
}

#define WK_PARAMS                                                                                                      \
    int dtype, const void *r, const void *k, const void *v, int n_planes, long long plane_stride, int ld, const float *z, \
        int ldz, const void *low, int low_planes, long long low_stride, int ld_low, const void *w2, int w2dtype, int rank, \
        const float *w0, const float *u, int B, int H, int d, int dv, const int *q_start, const int *slot, float *state, \
        long long state_stride, float *out, int ldo

static WkvArgs wk_args(WK_PARAMS) {
    WkvArgs a;
    a.r = r; a.k = k; a.v = v; a.n_planes = n_planes; a.plane_stride = (size_t)plane_stride; a.ld = ld;
    a.z = z; a.ldz = ldz; a.low = low; a.low_planes = low_planes; a.low_stride = (size_t)low_stride; a.ld_low = ld_low;
    a.w2 = w2; a.rank = rank; a.w0 = w0; a.u = u; a.B = B; a.H = H; a.d = d; a.dv = dv; a.q_start = q_start; a.slot = slot;
    a.state = state; a.state_stride = (size_t)state_stride; a.out = out; a.ldo = ldo;
    return a;
}
#define WK_PASS                                                                                                        \
    dtype, r, k, v, n_planes, plane_stride, ld, z, ldz, low, low_planes, low_stride, ld_low, w2, w2dtype, rank, w0, u, B, H, d, \
        dv, q_start, slot, state, state_stride, out, ldo

// the recurrence token by token; r, k, v in one dtype (float, planes allowed, or bf16), the decay's exponent either finished
// (z) or as the low-rank projection of the same dtype with W2
extern "C" int kb_wkv_scan(WK_PARAMS, cudaStream_t st) {
    if (B <= 0) return 0;
    if (H <= 0 || d <= 0 || dv <= 0 || d > 256 || (!z && (!low || !w2 || rank < 1 || rank > 512))) return (int)cudaErrorInvalidValue;
    const WkvArgs a = wk_args(WK_PASS);
    // four columns a warp where that still leaves a block or more an SM
    const int nc = d <= 128 && (long long)B * H * ((dv + 4 * WK_COLS - 1) / (4 * WK_COLS)) >= 148 ? 4 : 1;
    const int cols = WK_COLS * nc;
    const dim3 grid(B * H, (dv + cols - 1) / cols);
    const size_t sm = (size_t)WK_STAGE * (3 * d + cols + (z ? 0 : rank)) * sizeof(float);
#define WK_GO1(T, TW, DPL, NC)                                                                                         \
    do {                                                                                                               \
        if (sm > 48 * 1024)                                                                                            \
            cudaFuncSetAttribute(k_wkv_scan<T, TW, DPL, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);    \
        kb_launch(k_wkv_scan<T, TW, DPL, NC>, grid, 32 * WK_COLS, sm, st, a);                                          \
    } while (0)
#define WK_GO(T, TW)                                                                                                   \
    do {                                                                                                               \
        if (d <= 64) { if (nc == 4) WK_GO1(T, TW, 2, 4); else WK_GO1(T, TW, 2, 1); }                                   \
        else if (d <= 128) { if (nc == 4) WK_GO1(T, TW, 4, 4); else WK_GO1(T, TW, 4, 1); }                             \
        else WK_GO1(T, TW, 8, 1);                                                                                      \
    } while (0)
    if (dtype == KB_F32) {
        if (z || w2dtype == KB_F32) WK_GO(float, float); else WK_GO(float, bf16);
    } else {
        if (z || w2dtype == KB_F32) WK_GO(bf16, float); else WK_GO(bf16, bf16);
    }
#undef WK_GO
#undef WK_GO1
    KB_LAUNCH_RET();
}

extern "C" int kb_wkv_run() { return WR_C; }

// the same over long prompts, a sequence's runs of WR_C tokens side by side: r, k, v as bf16 rows, z finished, d <= 128.
// scratch: part [runs][H][dv][d] floats, keep [runs][H][d] floats with runs = T / WR_C + B
extern "C" int kb_wkv_runs(WK_PARAMS, int T, float* part, float* keep, cudaStream_t st) {
    if (B <= 0 || T <= 0) return 0;
    if (H <= 0 || d <= 0 || dv <= 0 || d > 128 || dtype != KB_BF16 || n_planes != 1 || !z || B > 65535 || H > 65535)
        return (int)cudaErrorInvalidValue;
    const WkvArgs a = wk_args(WK_PASS);
    const int runs = T / WR_C + B;
    const bool rows16 = ((uintptr_t)r | (uintptr_t)k | (uintptr_t)v) % 16 == 0 && ld % 8 == 0 && d % 8 == 0 && dv % 8 == 0;
    const bool v4 = d % 4 == 0 && (uintptr_t)state % 16 == 0 && state_stride % 4 == 0 && (uintptr_t)part % 16 == 0 &&
                    (uintptr_t)keep % 16 == 0;
    const int vec = (rows16 ? 1 : 0) | ((uintptr_t)out % 8 == 0 && ldo % 2 == 0 && dv % 2 == 0 ? 2 : 0) |
                    (v4 && (uintptr_t)z % 16 == 0 && ldz % 4 == 0 && (uintptr_t)w0 % 16 == 0 ? 4 : 0);
    const dim3 grid(runs, H, (dv + WR_E - 1) / WR_E);
    const int n_el = dv * d;
#define WR_GO(DP)                                                                                                      \
    do {                                                                                                               \
        static char tag;                                                                                               \
        if (kb_first_use(&tag)) {                                                                                      \
            cudaFuncSetAttribute(k_wkv_state<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, WrSmem<DP>::STATE);     \
            cudaFuncSetAttribute(k_wkv_out<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, WrSmem<DP>::OUT);         \
        }                                                                                                              \
        kb_launch(k_wkv_state<DP>, grid, WR_THREADS, WrSmem<DP>::STATE, st, a, part, keep, vec);                       \
        if (v4) kb_launch(k_wkv_prefix<4>, dim3((n_el / 4 + 255) / 256, H, B), 256, 0, st, a, part, (const float*)keep); \
        else kb_launch(k_wkv_prefix<1>, dim3((n_el + 255) / 256, H, B), 256, 0, st, a, part, (const float*)keep);      \
        kb_launch(k_wkv_out<DP>, grid, WR_THREADS, WrSmem<DP>::OUT, st, a, (const float*)part, vec);                   \
    } while (0)
    switch ((d + 15) / 16) {
        case 1: WR_GO(16); break;
        case 2: WR_GO(32); break;
        case 3: WR_GO(48); break;
        case 4: WR_GO(64); break;
        case 5: WR_GO(80); break;
        case 6: WR_GO(96); break;
        case 7: WR_GO(112); break;
        default: WR_GO(128); break;
    }
#undef WR_GO
    KB_LAUNCH_RET();
}
