// Recurrences whose state is a matrix per head under ONE decay per head and token, and the norms that follow them:
//
//     S_t = a_t S_(t-1) + w_t k_t v_t^T,      o_t = S_t^T q_t
//
// Two mixers are of this kind and differ in where a_t and w_t come from and in what happens to o_t:
//   SS_MLSTM  matrix memory with exponential gates kept in range by a running maximum m (zero at the start): log input
//             gate i = cap tanh(z_i / cap), log forget gate f = -softplus(-cap tanh(z_f / cap)), m_t = max(f + m_(t-1), i),
//             a = exp(f + m_(t-1) - m_t), w = exp(i - m_t). The state has one more column, the normaliser n (the same
//             recurrence with v = 1); the output is o / (max(|n . q|, exp(-m)) + 1e-6).
//   SS_MAMBA  state-space duality: dt = softplus(z + dt_bias), a = exp(-exp(A_log) dt), w = dt; q, k, v are C, B (one pair
//             per group of heads) and x; the output is o + D x.
// Both take their tokens as rows in bf16 or as 32-bit planes that are summed in order; everything else is 32-bit.
//   k_gated_scan    token by token, for single tokens, short steps and the true 32-bit path: a warp per state column
//   k_scan_gates    for long prompts: the gates of all tokens, with the running maxima by a scan over max-plus pairs
//   k_chunk_state   for long prompts: what every run of SS_C tokens adds to the state, all runs side by side
//   k_chunk_prefix  the states at the starts of the runs, in order
//   k_chunk_out     the outputs of every run from the state at its start and from its own tokens
//   k_scan_norm     matrix memory: division, RMS norm per head, gains, sigmoid gate; state space: silu gate, RMS norm per
//                   group, gains
// A run's products run on the tensor cores: q, k, v are bf16 there, and every 32-bit operand (the state, the values times
// their decayed weights, the weighted scores) enters as a sum of three bf16 numbers, so that the products carry 24 bits.
// Rows past a sequence's end in its last run count as tokens with w = 0, a = 1. Rows of a step that belong to no sequence
// (padding of a recorded step) are not touched.
#include "sm100.cuh"
#include "mma_sync.cuh"
#include "runs.cuh"
#include <math.h>

#define SS_MLSTM 0
#define SS_MAMBA 1
#define SS_DEN_EPS 1e-6f

struct SsArgs {
    const void* src;            // q, k, v: columns oq + (h / per) d, ok + (h / per) d, ov + h dv
    int n_planes;
    size_t plane_stride;
    int ld, oq, ok, ov, per;
    const void* gsrc;           // the gates' projections: columns og0 + h (and og1 + h)
    int g_planes;
    size_t g_plane_stride;
    int ldg, og0, og1;
    const float* p0;            // bias of the input gate [H]; dt_bias [H]
    const float* p1;            // bias of the forget gate [H]; A_log [H]
    const float* p2;            // -; D [H]
    float cap, qscale;
    int B, H, d, dv;
    const int* q_start;
    const int* slot;
    float* state;               // [slots][H][rows][d], rows = dv (+ 1: the normaliser)
    size_t state_stride;
    float* m_state;             // [slots][H]: the running maximum before the step (SS_MLSTM)
    size_t m_stride;
    float* out;                 // [T][ldo]
    int ldo;
    float* nq;                  // [T][H]: n . q (SS_MLSTM)
    float* m_rows;              // [T][H]: the running maximum after the token (SS_MLSTM)
};

template <typename T>
__device__ __forceinline__ float ss_rd(const T* p, int n_planes, size_t plane_stride) {
    float v = kb_to_f<T>(p[0]);
    for (int s = 1; s < n_planes; s++) v += kb_to_f<T>(p[(size_t)s * plane_stride]);
    return v;
}
__device__ __forceinline__ float ss_softplus(float z) { return log1pf(expf(-fabsf(z))) + fmaxf(z, 0.0f); }
__device__ __forceinline__ float ss_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
// where the result is rounded to bf16 anyway: the fast exponential and division (a few units of 2^-23)
__device__ __forceinline__ float ss_sigmoid_fast(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }

// the two numbers a token's gates are made of: (i, f) of the matrix memory, (dt, log decay) of the state space
template <typename T, int MODE>
__device__ __forceinline__ void ss_gate(const SsArgs& a, int row, int h, float& g0, float& g1) {
    const T* src = (const T*)a.gsrc + (size_t)row * a.ldg;
    const float z0 = ss_rd<T>(src + a.og0 + h, a.g_planes, a.g_plane_stride) + a.p0[h];
    if (MODE == SS_MLSTM) {
        const float z1 = ss_rd<T>(src + a.og1 + h, a.g_planes, a.g_plane_stride) + a.p1[h];
        g0 = a.cap * tanhf(z0 / a.cap);
        g1 = -ss_softplus(-a.cap * tanhf(z1 / a.cap));
    } else {
        g0 = ss_softplus(z0);
        g1 = -expf(a.p1[h]) * g0;
    }
}

// ------------------------------------------------------------------------------------------------ token by token
// A block works one (sequence, head) and SS_COLS columns of the state, a warp one column with its d elements over the
// lanes; tokens are staged SS_STAGE at a time.
// (NC of them, neighbours SS_COLS apart, when there are blocks enough: the loads of all of them are in flight together)
#define SS_COLS 8
#define SS_STAGE 16
template <typename T, int MODE, int DPL, int NC>
__global__ void __launch_bounds__(32 * SS_COLS, DPL * NC > 16 ? 2 : 3) k_gated_scan(SsArgs a) {
    extern __shared__ float sm[];
    const int d = a.d, dv = a.dv, H = a.H;
    float* qs = sm;                                   // [SS_STAGE][d]
    float* ks = qs + SS_STAGE * d;                    // [SS_STAGE][d]
    constexpr int COLS = SS_COLS * NC;
    float* vs = ks + SS_STAGE * d;                    // [SS_STAGE][COLS]
    float* g0 = vs + SS_STAGE * COLS;                 // [SS_STAGE]: i, then w
    float* g1 = g0 + SS_STAGE;                        // [SS_STAGE]: f, then a
    float* ms = g1 + SS_STAGE;                        // [SS_STAGE + 1]: running maxima, the one before the stage first
    kb_pdl_launch();
    const int b = blockIdx.x / H, h = blockIdx.x % H, hq = h / a.per;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rows = dv + (MODE == SS_MLSTM ? 1 : 0);
    const int e0 = blockIdx.y * COLS, e = e0 + warp;   // this warp's columns: e, e + SS_COLS, ...
    const int r0 = a.q_start[b], r1 = a.q_start[b + 1];
    const int sl = a.slot[b];
    float* srow = a.state + (size_t)sl * a.state_stride + (size_t)h * rows * d;
    const float D = MODE == SS_MAMBA ? a.p2[h] : 0.0f;
    // The states were left by earlier steps, which are complete before this step's first kernel starts: they are fetched
    // while the kernel before this one still runs.
    float S[NC][DPL];
#pragma unroll
    for (int c = 0; c < NC; c++)
#pragma unroll
        for (int i = 0; i < DPL; i++) {
            const int j = lane + 32 * i, ec = e + c * SS_COLS;
            S[c][i] = (ec < rows && j < d) ? srow[(size_t)ec * d + j] : 0.0f;
        }
    if (MODE == SS_MLSTM && threadIdx.x == 0) ms[SS_STAGE] = a.m_state[(size_t)sl * a.m_stride + h];
    kb_pdl_wait();
    const size_t oq = (size_t)a.oq + (size_t)hq * d, ok = (size_t)a.ok + (size_t)hq * d, ov = (size_t)a.ov + (size_t)h * dv;
    int last_n = SS_STAGE;
    for (int c0 = r0; c0 < r1; c0 += SS_STAGE) {
        const int n = min(SS_STAGE, r1 - c0);
        const T* base = (const T*)a.src + (size_t)c0 * a.ld;
        for (int idx = threadIdx.x; idx < n * d; idx += 32 * SS_COLS) {
            const int t = idx / d, j = idx % d;
            const T* p = base + (size_t)t * a.ld + j;
            qs[idx] = __fmul_rn(ss_rd<T>(p + oq, a.n_planes, a.plane_stride), a.qscale);
            ks[idx] = ss_rd<T>(p + ok, a.n_planes, a.plane_stride);
        }
        for (int idx = threadIdx.x; idx < n * COLS; idx += 32 * SS_COLS) {
            const int t = idx / COLS, c = e0 + idx % COLS;
            vs[idx] = c < dv ? ss_rd<T>(base + (size_t)t * a.ld + ov + c, a.n_planes, a.plane_stride) : 1.0f;
        }
        if (threadIdx.x < n) {
            float u0, u1;
            ss_gate<T, MODE>(a, c0 + threadIdx.x, h, u0, u1);
            g0[threadIdx.x] = u0;
            g1[threadIdx.x] = MODE == SS_MLSTM ? u1 : expf(u1);
        }
        __syncthreads();
        if (MODE == SS_MLSTM) {
            if (threadIdx.x == 0) {
                float m = ms[last_n];
                ms[0] = m;
                for (int t = 0; t < n; t++) {
                    m = fmaxf(g1[t] + m, g0[t]);
                    ms[t + 1] = m;
                }
            }
            __syncthreads();
            if (threadIdx.x < n) {
                const int t = threadIdx.x;
                const float m = ms[t + 1];
                g1[t] = expf(g1[t] + ms[t] - m);
                g0[t] = expf(g0[t] - m);
                if (blockIdx.y == 0) a.m_rows[(size_t)(c0 + t) * H + h] = m;
            }
            last_n = n;
            __syncthreads();
        }
        for (int t = 0; t < n; t++) {
            const float keep = g1[t];
            float v[NC], wv[NC], o[NC];
#pragma unroll
            for (int c = 0; c < NC; c++) {
                v[c] = vs[t * COLS + c * SS_COLS + warp];
                wv[c] = __fmul_rn(g0[t], v[c]);
                o[c] = 0.0f;
            }
#pragma unroll
            for (int i = 0; i < DPL; i++) {
                const int j = lane + 32 * i;
                if (j < d) {
                    const float kv = ks[t * d + j], qv = qs[t * d + j];
#pragma unroll
                    for (int c = 0; c < NC; c++) {
                        S[c][i] = fmaf(kv, wv[c], __fmul_rn(keep, S[c][i]));
                        o[c] = fmaf(S[c][i], qv, o[c]);
                    }
                }
            }
#pragma unroll
            for (int c = 0; c < NC; c++) o[c] = kb_warp_sum(o[c]);
#pragma unroll
            for (int c = 0; c < NC; c++) {
                const int ec = e + c * SS_COLS;
                if (lane == 0 && ec < rows) {
                    if (ec < dv) a.out[(size_t)(c0 + t) * a.ldo + (size_t)h * dv + ec] = fmaf(D, v[c], o[c]);
                    else a.nq[(size_t)(c0 + t) * H + h] = o[c];
                }
            }
        }
        __syncthreads();
    }
    if (r1 > r0) {
#pragma unroll
        for (int c = 0; c < NC; c++)
#pragma unroll
            for (int i = 0; i < DPL; i++) {
                const int j = lane + 32 * i, ec = e + c * SS_COLS;
                if (ec < rows && j < d) srow[(size_t)ec * d + j] = S[c][i];
            }
    }
}

// ------------------------------------------------------------------------------------------------ gates of long prompts
// ld [H][T]: log a; w [H][T]. The running maxima are the scan of the maps m -> max(F + m, M), a token's being (f, i):
// (F1, M1) then (F2, M2) is (F1 + F2, max(F2 + M1, M2)). A block per (head, sequence), SG_T tokens at a time.
#define SG_T 1024
template <typename T, int MODE>
__global__ void __launch_bounds__(SG_T) k_scan_gates(SsArgs a, float* __restrict__ ld, float* __restrict__ w, int Tn) {
    __shared__ float sF[SG_T / 32], sM[SG_T / 32], s_prev[SG_T + 1];
    kb_pdl_launch();
    const int h = blockIdx.x, b = blockIdx.y;
    const int r0 = a.q_start[b], r1 = a.q_start[b + 1];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    kb_pdl_wait();
    float* ldh = ld + (size_t)h * Tn, *wh = w + (size_t)h * Tn;
    if (MODE == SS_MAMBA) {
        // (no order among the tokens: gridDim.z blocks share them)
        for (int t = r0 + blockIdx.z * blockDim.x + threadIdx.x; t < r1; t += blockDim.x * gridDim.z) {
            float dt, l;
            ss_gate<T, MODE>(a, t, h, dt, l);
            ldh[t] = l;
            wh[t] = dt;
        }
        return;
    }
    float m_in = a.m_state[(size_t)a.slot[b] * a.m_stride + h];
    for (int c0 = r0; c0 < r1; c0 += SG_T) {
        const int t = c0 + threadIdx.x;
        float i = -INFINITY, f = 0.0f;
        if (t < r1) ss_gate<T, MODE>(a, t, h, i, f);
        float F = f, M = i;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float F1 = __shfl_up_sync(0xffffffffu, F, o), M1 = __shfl_up_sync(0xffffffffu, M, o);
            if (lane >= o) {
                M = fmaxf(F + M1, M);
                F += F1;
            }
        }
        if (lane == 31) {
            sF[warp] = F;
            sM[warp] = M;
        }
        __syncthreads();
        float m = m_in;                                // before this warp's tokens
        for (int k = 0; k < warp; k++) m = fmaxf(sF[k] + m, sM[k]);
        m = fmaxf(F + m, M);
        s_prev[threadIdx.x + 1] = m;
        if (threadIdx.x == 0) s_prev[0] = m_in;
        __syncthreads();
        if (t < r1) {
            ldh[t] = fminf(f + s_prev[threadIdx.x] - m, 0.0f);
            wh[t] = expf(i - m);
            a.m_rows[(size_t)t * a.H + h] = m;
        }
        m_in = s_prev[SG_T];                            // (only read when there is another tile, which this one fills)
        __syncthreads();
    }
}

// ------------------------------------------------------------------------------------------------ runs of long prompts
#define SS_C 64
#define SS_E 64                 // state columns (values) of a block
#define SS_LD 72                // row of a 64-wide bf16 tile in shared memory
#define SS_THREADS 128

__device__ __forceinline__ KbRun ss_run(const SsArgs& a, int run) { return kb_find_run(a.q_start, a.B, SS_C, run); }
// rows of bf16 from global into a padded tile [SS_C][dst_ld]; columns from d to dp and rows from n on are zero. Whole 16-byte
// words go by asynchronous copies: the caller waits for them (cp_async_wait_all) before its barrier
__device__ __forceinline__ void ss_tile(bf16* dst, int dst_ld, const bf16* src, int ld, int n, int d, int dp, bool vec) {
    if (vec) {
        const int per = dp / 8;
        for (int idx = threadIdx.x; idx < SS_C * per; idx += SS_THREADS) {
            const int t = idx / per, c = (idx % per) * 8;
            const bool ok = t < n && c < d;
            cp_async16(smem_u32(dst + t * dst_ld + c), ok ? (const void*)(src + (size_t)t * ld + c) : (const void*)src, ok);
        }
        return;
    }
    for (int idx = threadIdx.x; idx < SS_C * dp; idx += SS_THREADS) {
        const int t = idx / dp, c = idx % dp;
        dst[t * dst_ld + c] = (t < n && c < d) ? src[(size_t)t * ld + c] : __float2bfloat16_rn(0.0f);
    }
}
// the running sum of the run's log decays, up to and with every token, by the first warp (two tokens a lane)
__device__ __forceinline__ void ss_log_sums(const float* ldh, int n, float* lg) {
    if (threadIdx.x < 32) {
        const int t = 2 * threadIdx.x;
        const float x0 = t < n ? ldh[t] : 0.0f, x1 = t + 1 < n ? ldh[t + 1] : 0.0f;
        float s = x0 + x1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, s, o);
            if (threadIdx.x >= o) s += u;
        }
        const float before = __shfl_up_sync(0xffffffffu, s, 1);
        lg[t] = (threadIdx.x > 0 ? before : 0.0f) + x0;
        lg[t + 1] = s;
    }
}

// part [runs][H][rows][d]: sum over the run's tokens of exp(lg_last - lg_s) w_s v_s k_s^T; lg_end [runs][H]: the sum of the
// run's log decays. grid (runs, H, ceil(dv / SS_E))
template <int MODE>
__global__ void __launch_bounds__(SS_THREADS) k_chunk_state(SsArgs a, const float* KB_STEP_DATA ld, const float* KB_STEP_DATA w,
        int Tn, float* __restrict__ part, float* __restrict__ lg_end, int dp, int vec) {
    extern __shared__ __align__(16) uint8_t sm8[];
    const int kld = dp + 8;
    bf16* vw = (bf16*)sm8;                             // [KB_SPLIT][SS_C][SS_LD]
    bf16* ks = vw + KB_SPLIT * SS_C * SS_LD;           // [SS_C][kld]
    __shared__ float lg[SS_C], wt[SS_C];
    kb_pdl_launch();
    const KbRun r = ss_run(a, blockIdx.x);
    kb_pdl_wait();
    if (r.n <= 0) return;
    const int h = blockIdx.y, e0 = blockIdx.z * SS_E;
    const int d = a.d, dv = a.dv, rows = dv + (MODE == SS_MLSTM ? 1 : 0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bf16* src = (const bf16*)a.src + (size_t)r.r0 * a.ld;
    ss_tile(ks, kld, src + a.ok + (size_t)(h / a.per) * d, a.ld, r.n, d, dp, vec & 1);
    const bf16* vsrc = src + a.ov + (size_t)h * dv + e0;
    // values: 8 neighbours a load, 4 loads a thread in flight
    const bool v8 = (vec & 4) && dv - e0 >= SS_E;
    uint4 vv[4];
    if (v8) {
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int idx = threadIdx.x + i * SS_THREADS, s = idx >> 3, c = (idx & 7) * 8;
            vv[i] = s < r.n ? *(const uint4*)(vsrc + (size_t)s * a.ld + c) : make_uint4(0, 0, 0, 0);
        }
    }
    ss_log_sums(ld + (size_t)h * Tn + r.r0, r.n, lg);
    __syncthreads();
    if (threadIdx.x < SS_C) {
        const int s = threadIdx.x;
        wt[s] = s < r.n ? expf(lg[SS_C - 1] - lg[s]) * w[(size_t)h * Tn + r.r0 + s] : 0.0f;
    }
    if (threadIdx.x == 0 && blockIdx.z == 0) lg_end[(size_t)blockIdx.x * a.H + h] = lg[SS_C - 1];
    __syncthreads();
    if (v8) {
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int idx = threadIdx.x + i * SS_THREADS, s = idx >> 3, c = (idx & 7) * 8;
            const __nv_bfloat162* p = (const __nv_bfloat162*)&vv[i];
            uint32_t sp[KB_SPLIT][4];
#pragma unroll
            for (int k = 0; k < 4; k++) {
                uint32_t q[KB_SPLIT];
                split_pack_bf16(__low2float(p[k]) * wt[s], __high2float(p[k]) * wt[s], q);
#pragma unroll
                for (int u = 0; u < KB_SPLIT; u++) sp[u][k] = q[u];
            }
#pragma unroll
            for (int u = 0; u < KB_SPLIT; u++)
                *(uint4*)(vw + (u * SS_C + s) * SS_LD + c) = make_uint4(sp[u][0], sp[u][1], sp[u][2], sp[u][3]);
        }
    } else {
        for (int idx = threadIdx.x; idx < SS_C * (SS_E / 2); idx += SS_THREADS) {
            const int s = idx / (SS_E / 2), c = (idx % (SS_E / 2)) * 2;
            float x = 0.0f, y = 0.0f;
            if (s < r.n) {
                const bf16* p = vsrc + (size_t)s * a.ld + c;
                if ((vec & 2) && e0 + c + 1 < dv) {
                    const __nv_bfloat162 v2 = *(const __nv_bfloat162*)p;
                    x = __low2float(v2) * wt[s];
                    y = __high2float(v2) * wt[s];
                } else {
                    if (e0 + c < dv) x = __bfloat162float(p[0]) * wt[s];
                    if (e0 + c + 1 < dv) y = __bfloat162float(p[1]) * wt[s];
                }
            }
            uint32_t sp[KB_SPLIT];
            split_pack_bf16(x, y, sp);
#pragma unroll
            for (int i = 0; i < KB_SPLIT; i++) *(uint32_t*)(vw + (i * SS_C + s) * SS_LD + c) = sp[i];
        }
    }
    cp_async_wait_all();
    __syncthreads();
    float* pb = part + ((size_t)blockIdx.x * a.H + h) * rows * d;
    // this warp's 16 columns of the state against all of the keys' elements
    uint32_t av[KB_SPLIT][SS_C / 16][4];
    const int m0 = warp * 16;
    const bool live = e0 + m0 < dv;
    if (live) {
#pragma unroll
        for (int i = 0; i < KB_SPLIT; i++)
#pragma unroll
            for (int k = 0; k < SS_C / 16; k++) {
                const int row = k * 16 + ((lane >> 4) & 1) * 8 + (lane & 7), col = m0 + ((lane >> 3) & 1) * 8;
                ldsm_x4_t(smem_u32(vw + (i * SS_C + row) * SS_LD + col), av[i][k][0], av[i][k][1], av[i][k][2], av[i][k][3]);
            }
        for (int j0 = 0; j0 < dp; j0 += 32) {
            // 32 of the keys' elements at a time (the last 16 of an odd multiple twice, which is not stored): four chains of
            // products that do not wait for one another
            const int j1 = j0 + 16 < dp ? j0 + 16 : j0;
            float acc[4][4] = {};
#pragma unroll
            for (int k = 0; k < SS_C / 16; k++) {
                uint32_t bf[2][4];
                const int row = k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, col = (lane >> 4) * 8;
                ldsm_x4_t(smem_u32(ks + row * kld + j0 + col), bf[0][0], bf[0][1], bf[0][2], bf[0][3]);
                ldsm_x4_t(smem_u32(ks + row * kld + j1 + col), bf[1][0], bf[1][1], bf[1][2], bf[1][3]);
#pragma unroll
                for (int i = KB_SPLIT - 1; i >= 0; i--)
#pragma unroll
                    for (int u = 0; u < 4; u++) mma_bf16(acc[u], av[i][k], bf[u >> 1][(u & 1) * 2], bf[u >> 1][(u & 1) * 2 + 1]);
            }
            const int nu = j1 > j0 ? 4 : 2;
#pragma unroll
            for (int u = 0; u < 4; u++) {
                if (u >= nu) break;
                const int j = j0 + u * 8 + (lane & 3) * 2;
#pragma unroll
                for (int hf = 0; hf < 2; hf++) {
                    const int e = e0 + m0 + (lane >> 2) + hf * 8;
                    if (e >= dv) continue;
                    float* p = pb + (size_t)e * d + j;
                    if (j + 1 < d && !(d & 1)) *(float2*)p = make_float2(acc[u][2 * hf], acc[u][2 * hf + 1]);
                    else {
                        if (j < d) p[0] = acc[u][2 * hf];
                        if (j + 1 < d) p[1] = acc[u][2 * hf + 1];
                    }
                }
            }
        }
    }
    if (MODE == SS_MLSTM && blockIdx.z == 0) {
        for (int j = threadIdx.x; j < d; j += SS_THREADS) {
            float n = 0.0f;
            for (int s = 0; s < r.n; s++) n = fmaf(wt[s], __bfloat162float(ks[s * kld + j]), n);
            pb[(size_t)dv * d + j] = n;
        }
    }
}

// part[run] <- the state at the run's start; the sequence's state <- the state after its last run. A thread per VW
// neighbouring elements of a (sequence, head), four runs' loads in flight. grid (ceil(elements / (256 VW)), H, B)
template <int VW>
__global__ void __launch_bounds__(256) k_chunk_prefix(SsArgs a, float* part, const float* KB_STEP_DATA lg_end, int n_el) {
    kb_pdl_launch();
    const int h = blockIdx.y, b = blockIdx.z;
    const int s0 = a.q_start[b], len = a.q_start[b + 1] - s0;
    const int nr = (len + SS_C - 1) / SS_C, run0 = s0 / SS_C + b;
    const size_t at = ((size_t)blockIdx.x * 256 + threadIdx.x) * VW;
    kb_pdl_wait();
    if (at >= (size_t)n_el || nr <= 0) return;
    float* st = a.state + (size_t)a.slot[b] * a.state_stride + (size_t)h * n_el + at;
    const size_t step = (size_t)a.H * n_el;
    float* p = part + (size_t)run0 * step + (size_t)h * n_el + at;
    const float* le = lg_end + (size_t)run0 * a.H + h;
    typedef typename std::conditional<VW == 4, float4, float>::type V;
    V S = *(const V*)st;
    float* Sf = (float*)&S;
    for (int c0 = 0; c0 < nr; c0 += 4) {
        V x[4];
        float g[4];
#pragma unroll
        for (int k = 0; k < 4; k++)
            if (c0 + k < nr) {
                x[k] = *(const V*)(p + (size_t)(c0 + k) * step);
                g[k] = le[(size_t)(c0 + k) * a.H];
            }
#pragma unroll
        for (int k = 0; k < 4; k++)
            if (c0 + k < nr) {
                *(V*)(p + (size_t)(c0 + k) * step) = S;
                const float keep = expf(g[k]);
                const float* xf = (const float*)&x[k];
#pragma unroll
                for (int i = 0; i < VW; i++) Sf[i] = fmaf(keep, Sf[i], xf[i]);
            }
    }
    *(V*)st = S;
}

// grid (runs, H, ceil(dv / SS_E)); a warp works 16 of the run's tokens against SS_E columns of the state
template <int MODE>
__global__ void __launch_bounds__(SS_THREADS) k_chunk_out(SsArgs a, const float* KB_STEP_DATA ld, const float* KB_STEP_DATA w,
        int Tn, const float* KB_STEP_DATA part, int dp, int vec) {
    extern __shared__ __align__(16) uint8_t sm8[];
    const int kld = dp + 8;
    bf16* qs = (bf16*)sm8;                             // [SS_C][kld]
    bf16* ss = qs + SS_C * kld;                        // [KB_SPLIT][SS_E][SS_LD]: 64 elements of the state's columns; then
    bf16* vs = ss;                                     // [SS_C][SS_LD]
    bf16* ks = vs + SS_C * SS_LD;                      // [SS_C][kld]
    __shared__ float lg[SS_C], wt[SS_C];
    kb_pdl_launch();
    const KbRun r = ss_run(a, blockIdx.x);
    kb_pdl_wait();
    if (r.n <= 0) return;
    const int h = blockIdx.y, e0 = blockIdx.z * SS_E;
    const int d = a.d, dv = a.dv, rows = dv + (MODE == SS_MLSTM ? 1 : 0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bf16* src = (const bf16*)a.src + (size_t)r.r0 * a.ld;
    const int ne = min(SS_E, dv - e0);
    const float* S0 = part + ((size_t)blockIdx.x * a.H + h) * rows * d;
    // the state's columns, 64 elements at a time: four neighbours a load, eight loads a thread in flight, the next 64 on
    // their way while the products of these run
    const bool s4 = (vec & 16) && ne == SS_E;
    float4 sv[8];
    auto s_load = [&](int jb) {
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int idx = threadIdx.x + i * SS_THREADS, e = idx >> 4, j = jb + (idx & 15) * 4;
            sv[i] = j < d ? *(const float4*)(S0 + (size_t)(e0 + e) * d + j) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
    };
    if (s4) s_load(0);
    ss_tile(qs, kld, src + a.oq + (size_t)(h / a.per) * d, a.ld, r.n, d, dp, vec & 1);
    ss_log_sums(ld + (size_t)h * Tn + r.r0, r.n, lg);
    if (threadIdx.x >= 64 && threadIdx.x < 64 + SS_C) {
        const int s = threadIdx.x - 64;
        wt[s] = s < r.n ? w[(size_t)h * Tn + r.r0 + s] : 0.0f;
    }
    const int t0 = warp * 16;
    float o[SS_E / 8][4] = {};
    for (int jb = 0; jb < dp; jb += 64) {
        __syncthreads();                               // (the tile before has been read)
        if (s4) {
#pragma unroll
            for (int i = 0; i < 8; i++) {
                const int idx = threadIdx.x + i * SS_THREADS, e = idx >> 4, c = (idx & 15) * 4;
                uint32_t p[KB_SPLIT], q[KB_SPLIT];
                split_pack_bf16(sv[i].x, sv[i].y, p);
                split_pack_bf16(sv[i].z, sv[i].w, q);
#pragma unroll
                for (int u = 0; u < KB_SPLIT; u++) *(uint2*)(ss + (u * SS_E + e) * SS_LD + c) = make_uint2(p[u], q[u]);
            }
            if (jb + 64 < dp) s_load(jb + 64);
        } else for (int idx = threadIdx.x; idx < SS_E * 32; idx += SS_THREADS) {
            const int e = idx >> 5, c = (idx & 31) * 2, j = jb + c;
            float x = 0.0f, y = 0.0f;
            if (e < ne) {
                const float* p = S0 + (size_t)(e0 + e) * d + j;
                if (j + 1 < d && !(d & 1)) {
                    const float2 v2 = *(const float2*)p;
                    x = v2.x;
                    y = v2.y;
                } else {
                    if (j < d) x = p[0];
                    if (j + 1 < d) y = p[1];
                }
            }
            uint32_t sp[KB_SPLIT];
            split_pack_bf16(x, y, sp);
#pragma unroll
            for (int i = 0; i < KB_SPLIT; i++) *(uint32_t*)(ss + (i * SS_E + e) * SS_LD + c) = sp[i];
        }
        cp_async_wait_all();
        __syncthreads();
        const int kn = min(64, dp - jb) / 16;
        for (int k = 0; k < kn; k++) {
            uint32_t aq[4];
            ldsm_x4(smem_u32(qs + (t0 + (lane & 7) + ((lane >> 3) & 1) * 8) * kld + jb + k * 16 + (lane >> 4) * 8), aq[0],
                    aq[1], aq[2], aq[3]);
#pragma unroll
            for (int np = 0; np < SS_E / 32; np++) {
                // 32 columns at a time: all loads first, then four chains of products
                uint32_t bf[KB_SPLIT][2][4];
                const int row = np * 32 + (lane & 7) + (lane >> 4) * 8, col = k * 16 + ((lane >> 3) & 1) * 8;
#pragma unroll
                for (int i = 0; i < KB_SPLIT; i++)
#pragma unroll
                    for (int u = 0; u < 2; u++)
                        ldsm_x4(smem_u32(ss + (i * SS_E + row + u * 16) * SS_LD + col), bf[i][u][0], bf[i][u][1], bf[i][u][2],
                                bf[i][u][3]);
#pragma unroll
                for (int i = KB_SPLIT - 1; i >= 0; i--)
#pragma unroll
                    for (int u = 0; u < 4; u++)
                        mma_bf16(o[4 * np + u], aq, bf[i][u >> 1][(u & 1) * 2], bf[i][u >> 1][(u & 1) * 2 + 1]);
            }
        }
    }
    __syncthreads();                                   // the state's tile is done with: its place takes keys and values
    ss_tile(ks, kld, src + a.ok + (size_t)(h / a.per) * d, a.ld, r.n, d, dp, vec & 1);
    ss_tile(vs, SS_LD, src + a.ov + (size_t)h * dv + e0, a.ld, r.n, ne, SS_E, (vec & 4) && ne % 8 == 0);
    // the state's share decays from the run's start
    const int ta = t0 + (lane >> 2), tb = ta + 8;
    const float la = lg[ta], lb = lg[tb], fa = expf(la), fb = expf(lb);
#pragma unroll
    for (int n = 0; n < SS_E / 8; n++) {
        o[n][0] *= fa;
        o[n][1] *= fa;
        o[n][2] *= fb;
        o[n][3] *= fb;
    }
    cp_async_wait_all();
    __syncthreads();
    // the run's own tokens, 16 keys at a time: score, decay and weight, sum
    float sa = 0.0f, sb = 0.0f;                        // sums of the weights (the normaliser's share)
    for (int k2 = 0; k2 <= warp; k2++) {
        float sc[2][4] = {}, s1[2][4] = {};
        for (int k = 0; k < dp / 16; k += 2) {
            // two steps at a time, in sums of their own
            const bool two = (k + 1) * 16 < dp;
            uint32_t aq[2][4], bf[2][4];
#pragma unroll
            for (int u = 0; u < 2; u++) {
                const int kk = (u == 0 || two) ? k + u : k;
                ldsm_x4(smem_u32(qs + (t0 + (lane & 7) + ((lane >> 3) & 1) * 8) * kld + kk * 16 + (lane >> 4) * 8), aq[u][0],
                        aq[u][1], aq[u][2], aq[u][3]);
                ldsm_x4(smem_u32(ks + (k2 * 16 + (lane & 7) + (lane >> 4) * 8) * kld + kk * 16 + ((lane >> 3) & 1) * 8),
                        bf[u][0], bf[u][1], bf[u][2], bf[u][3]);
            }
            mma_bf16(sc[0], aq[0], bf[0][0], bf[0][1]);
            mma_bf16(sc[1], aq[0], bf[0][2], bf[0][3]);
            if (two) {
                mma_bf16(s1[0], aq[1], bf[1][0], bf[1][1]);
                mma_bf16(s1[1], aq[1], bf[1][2], bf[1][3]);
            }
        }
#pragma unroll
        for (int u = 0; u < 2; u++)
#pragma unroll
            for (int c = 0; c < 4; c++) sc[u][c] += s1[u][c];
        uint32_t pa[KB_SPLIT][4];
#pragma unroll
        for (int u = 0; u < 2; u++) {
            const int s = k2 * 16 + u * 8 + (lane & 3) * 2;
            const float l0 = lg[s], l1 = lg[s + 1], w0 = wt[s], w1 = wt[s + 1];
            const float p0 = s <= ta ? sc[u][0] * expf(la - l0) * w0 : 0.0f;
            const float p1 = s + 1 <= ta ? sc[u][1] * expf(la - l1) * w1 : 0.0f;
            const float p2 = s <= tb ? sc[u][2] * expf(lb - l0) * w0 : 0.0f;
            const float p3 = s + 1 <= tb ? sc[u][3] * expf(lb - l1) * w1 : 0.0f;
            sa += p0 + p1;
            sb += p2 + p3;
            uint32_t x[KB_SPLIT], y[KB_SPLIT];
            split_pack_bf16(p0, p1, x);
            split_pack_bf16(p2, p3, y);
#pragma unroll
            for (int i = 0; i < KB_SPLIT; i++) {
                pa[i][2 * u] = x[i];
                pa[i][2 * u + 1] = y[i];
            }
        }
#pragma unroll
        for (int dp2 = 0; dp2 < SS_E / 32; dp2++) {
            uint32_t bf[2][4];
#pragma unroll
            for (int u = 0; u < 2; u++)
                ldsm_x4_t(smem_u32(vs + (k2 * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SS_LD + (dp2 * 2 + u) * 16 +
                                   (lane >> 4) * 8), bf[u][0], bf[u][1], bf[u][2], bf[u][3]);
#pragma unroll
            for (int i = KB_SPLIT - 1; i >= 0; i--)
#pragma unroll
                for (int u = 0; u < 4; u++)
                    mma_bf16(o[4 * dp2 + u], pa[i], bf[u >> 1][(u & 1) * 2], bf[u >> 1][(u & 1) * 2 + 1]);
        }
    }
    const float D = MODE == SS_MAMBA ? a.p2[h] : 0.0f;
#pragma unroll
    for (int n = 0; n < SS_E / 8; n++) {
        const int c = n * 8 + (lane & 3) * 2;
#pragma unroll
        for (int hf = 0; hf < 2; hf++) {
            const int t = hf ? tb : ta;
            if (t >= r.n) continue;
            float* p = a.out + (size_t)(r.r0 + t) * a.ldo + (size_t)h * dv + e0 + c;
            float x = o[n][2 * hf] * a.qscale, y = o[n][2 * hf + 1] * a.qscale;
            if (MODE == SS_MAMBA) {
                x = fmaf(D, __bfloat162float(vs[t * SS_LD + c]), x);
                y = fmaf(D, __bfloat162float(vs[t * SS_LD + c + 1]), y);
            }
            if (c + 1 < ne && (vec & 8)) *(float2*)p = make_float2(x, y);
            else {
                if (c < ne) p[0] = x;
                if (c + 1 < ne) p[1] = y;
            }
        }
    }
    if (MODE == SS_MLSTM && blockIdx.z == 0) {
        sa += __shfl_xor_sync(0xffffffffu, sa, 1);
        sa += __shfl_xor_sync(0xffffffffu, sa, 2);
        sb += __shfl_xor_sync(0xffffffffu, sb, 1);
        sb += __shfl_xor_sync(0xffffffffu, sb, 2);
        const float* n0 = S0 + (size_t)dv * d;
        float nr[8];                                   // (d <= 256 here)
#pragma unroll
        for (int k = 0; k < 8; k++) nr[k] = lane + 32 * k < d ? n0[lane + 32 * k] : 0.0f;
#pragma unroll 4
        for (int i = 0; i < 16; i++) {
            const int t = t0 + i;
            float acc = 0.0f;
#pragma unroll
            for (int k = 0; k < 8; k++)
                if (32 * k < d && lane + 32 * k < dp) acc = fmaf(nr[k], __bfloat162float(qs[t * kld + lane + 32 * k]), acc);
            acc = kb_warp_sum(acc);
            const float own = __shfl_sync(0xffffffffu, i < 8 ? sa : sb, (i & 7) * 4);
            if (lane == 0 && t < r.n) a.nq[(size_t)(r.r0 + t) * a.H + h] = (expf(lg[t]) * acc + own) * a.qscale;
        }
    }
}

// ------------------------------------------------------------------------------------------------ norm on the output
// four neighbours, aligned
template <typename TG>
__device__ __forceinline__ void ss_rd4(const TG* p, int n_planes, size_t plane_stride, float* z) {
    for (int s = 0; s < n_planes; s++) {
        float v[4];
        if (sizeof(TG) == 4) {
            const float4 q = *(const float4*)(p + (size_t)s * plane_stride);
            v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
        } else {
            const uint2 q = *(const uint2*)(p + (size_t)s * plane_stride);
            const bf16* qb = (const bf16*)&q;
#pragma unroll
            for (int i = 0; i < 4; i++) v[i] = __bfloat162float(qb[i]);
        }
#pragma unroll
        for (int i = 0; i < 4; i++) z[i] = s == 0 ? v[i] : z[i] + v[i];
    }
}

// A group's n neighbouring elements of a row by TPG threads:
//   SS_MLSTM  u = x / (max(|nq|, exp(-m)) + 1e-6), out = rms(u) * gain * sigmoid(g); a group is a head; the running maximum
//             of a sequence's last row becomes its state
//   SS_MAMBA  u = x * silu(g), out = rms(u) * gain
// VW: neighbouring elements a thread takes at once (4 where everything is aligned); NI > 0: the group in registers, NI times
// four neighbours a thread; NI == 0: in shared memory
template <typename TG, typename TO, int MODE, int TPG, int VW, int NI>
__global__ void __launch_bounds__(256) k_scan_norm(const float* KB_STEP_DATA x, int ldx, int T, int NG, int n,
        const float* __restrict__ w, float eps, const TG* KB_STEP_DATA g, int g_planes, size_t g_plane_stride, int ldg, int og,
        const float* KB_STEP_DATA nq, const float* KB_STEP_DATA m_rows, float* m_state, size_t m_stride,
        const int* __restrict__ pos, const int* __restrict__ seq, const int* __restrict__ slot,
        const int* __restrict__ q_start, TO* __restrict__ out, int ldo) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[8];
    kb_pdl_launch();
    constexpr int GPB = 256 / TPG;
    const int gi = threadIdx.x / TPG, tid = threadIdx.x % TPG;
    const long long item = (long long)blockIdx.x * GPB + gi;
    const bool live = item < (long long)T * NG;
    const int t = live ? (int)(item / NG) : 0, h = live ? (int)(item % NG) : 0;
    kb_pdl_wait();
    float* u = sm + (size_t)gi * ((n + 3) & ~3);
    const float* xr = x + (size_t)t * ldx + (size_t)h * n;
    const TG* gr = g + (size_t)t * ldg + og + (size_t)h * n;
    if constexpr (NI > 0) {
        // the group in registers: every load in flight before the first use
        float4 xv[NI], wv[NI];
        float z[NI][4];
#pragma unroll
        for (int i = 0; i < NI; i++) {
            const int c = (tid + i * TPG) * 4;
            wv[i] = c < n ? *(const float4*)(w + (size_t)h * n + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            xv[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            z[i][0] = z[i][1] = z[i][2] = z[i][3] = 0.0f;
            if (live && c < n) {
                xv[i] = *(const float4*)(xr + c);
                ss_rd4<TG>(gr + c, g_planes, g_plane_stride, z[i]);
            }
        }
        float f = 1.0f;
        if (MODE == SS_MLSTM && live) {
            const float m = m_rows[(size_t)t * NG + h];
            f = 1.0f / (fmaxf(fabsf(nq[(size_t)t * NG + h]), expf(-m)) + SS_DEN_EPS);
            if (tid == 0 && pos[t] >= 0) {
                const int b = seq[t];
                if (t == q_start[b + 1] - 1) m_state[(size_t)slot[b] * m_stride + h] = m;
            }
        }
        float sq = 0.0f;
#pragma unroll
        for (int i = 0; i < NI; i++) {
            float* v = (float*)&xv[i];
#pragma unroll
            for (int k = 0; k < 4; k++) {
                v[k] *= MODE == SS_MLSTM ? f : z[i][k] * (sizeof(TO) == 2 ? ss_sigmoid_fast(z[i][k]) : ss_sigmoid(z[i][k]));
                sq = fmaf(v[k], v[k], sq);
            }
        }
        sq = kb_warp_sum(sq);
        if (TPG > 32) {
            if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
            __syncthreads();
            sq = 0.0f;
#pragma unroll
            for (int k = 0; k < 8; k++) sq += red[k];
        }
        const float rn = 1.0f / sqrtf(sq / (float)n + eps);
#pragma unroll
        for (int i = 0; i < NI; i++) {
            const int c = (tid + i * TPG) * 4;
            if (!live || c >= n) continue;
            const float* v = (const float*)&xv[i], *wf = (const float*)&wv[i];
            float y[4];
#pragma unroll
            for (int k = 0; k < 4; k++) {
                y[k] = __fmul_rn(__fmul_rn(v[k], rn), wf[k]);
                if (MODE == SS_MLSTM) y[k] *= sizeof(TO) == 2 ? ss_sigmoid_fast(z[i][k]) : ss_sigmoid(z[i][k]);
            }
            TO* dst = out + (size_t)t * ldo + (size_t)h * n + c;
            if (sizeof(TO) == 2) {
                *(uint2*)dst = make_uint2(pack_bf16(y[0], y[1]), pack_bf16(y[2], y[3]));
            } else {
#pragma unroll
                for (int k = 0; k < 4; k++) dst[k] = kb_from_f<TO>(y[k]);
            }
        }
        return;
    }
    float f = 1.0f;
    if (MODE == SS_MLSTM && live) {
        const float m = m_rows[(size_t)t * NG + h];
        f = 1.0f / (fmaxf(fabsf(nq[(size_t)t * NG + h]), expf(-m)) + SS_DEN_EPS);
        if (tid == 0 && pos[t] >= 0) {
            const int b = seq[t];
            if (t == q_start[b + 1] - 1) m_state[(size_t)slot[b] * m_stride + h] = m;
        }
    }
    auto gate = [&](int c, float* z) {
        if (VW == 4) ss_rd4<TG>(gr + c, g_planes, g_plane_stride, z);
        else z[0] = ss_rd<TG>(gr + c, g_planes, g_plane_stride);
    };
    float sq = 0.0f;
    if (live) {
        for (int c = tid * VW; c < n; c += TPG * VW) {
            float v[VW], z[VW];
            if (VW == 4) {
                const float4 q = *(const float4*)(xr + c);
                v[0] = q.x;
                if (VW == 4) { v[VW - 3] = q.y; v[VW - 2] = q.z; v[VW - 1] = q.w; }
            } else v[0] = xr[c];
            if (MODE == SS_MAMBA) gate(c, z);
#pragma unroll
            for (int i = 0; i < VW; i++) {
                v[i] = MODE == SS_MLSTM ? v[i] * f : v[i] * (z[i] / (1.0f + expf(-z[i])));
                u[c + i] = v[i];
                sq = fmaf(v[i], v[i], sq);
            }
        }
    }
    sq = kb_warp_sum(sq);
    if (TPG > 32) {
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
        __syncthreads();
        sq = 0.0f;
#pragma unroll
        for (int k = 0; k < 8; k++) sq += red[k];
    }
    if (!live) return;
    const float rn = 1.0f / sqrtf(sq / (float)n + eps);
    for (int c = tid * VW; c < n; c += TPG * VW) {
        float z[VW], y[VW];
        if (MODE == SS_MLSTM) gate(c, z);
#pragma unroll
        for (int i = 0; i < VW; i++) {
            y[i] = __fmul_rn(__fmul_rn(u[c + i], rn), w[(size_t)h * n + c + i]);
            if (MODE == SS_MLSTM) y[i] *= ss_sigmoid(z[i]);
        }
        TO* dst = out + (size_t)t * ldo + (size_t)h * n + c;
        if (VW == 4 && sizeof(TO) == 2) {
            uint2 q;
            q.x = pack_bf16(y[0], y[VW > 1 ? 1 : 0]);
            q.y = pack_bf16(y[VW > 2 ? 2 : 0], y[VW > 3 ? 3 : 0]);
            *(uint2*)dst = q;
        } else {
#pragma unroll
            for (int i = 0; i < VW; i++) dst[i] = kb_from_f<TO>(y[i]);
        }
    }
}

// ------------------------------------------------------------------------------------------------ entry points
static SsArgs ss_args(const void* src, int n_planes, long long plane_stride, int ld, int oq, int ok, int ov, int per,
                      const void* gsrc, int g_planes, long long g_plane_stride, int ldg, int og0, int og1, const float* p0,
                      const float* p1, const float* p2, float cap, float qscale, int B, int H, int d, int dv,
                      const int* q_start, const int* slot, float* state, long long state_stride, float* m_state,
                      long long m_stride, float* out, int ldo, float* nq, float* m_rows) {
    SsArgs a;
    a.src = src; a.n_planes = n_planes; a.plane_stride = (size_t)plane_stride; a.ld = ld;
    a.oq = oq; a.ok = ok; a.ov = ov; a.per = per;
    a.gsrc = gsrc; a.g_planes = g_planes; a.g_plane_stride = (size_t)g_plane_stride; a.ldg = ldg; a.og0 = og0; a.og1 = og1;
    a.p0 = p0; a.p1 = p1; a.p2 = p2; a.cap = cap; a.qscale = qscale;
    a.B = B; a.H = H; a.d = d; a.dv = dv; a.q_start = q_start; a.slot = slot;
    a.state = state; a.state_stride = (size_t)state_stride; a.m_state = m_state; a.m_stride = (size_t)m_stride;
    a.out = out; a.ldo = ldo; a.nq = nq; a.m_rows = m_rows;
    return a;
}

#define SS_PARAMS                                                                                                      \
    int mode, int dtype, const void *src, int n_planes, long long plane_stride, int ld, int oq, int ok, int ov, int per, \
        const void *gsrc, int g_planes, long long g_plane_stride, int ldg, int og0, int og1, const float *p0,          \
        const float *p1, const float *p2, float cap, float qscale, int B, int H, int d, int dv, const int *q_start,    \
        const int *slot, float *state, long long state_stride, float *m_state, long long m_stride, float *out, int ldo, \
        float *nq, float *m_rows
#define SS_PASS                                                                                                        \
    src, n_planes, plane_stride, ld, oq, ok, ov, per, gsrc, g_planes, g_plane_stride, ldg, og0, og1, p0, p1, p2, cap,  \
        qscale, B, H, d, dv, q_start, slot, state, state_stride, m_state, m_stride, out, ldo, nq, m_rows

static bool ss_ok(int mode, int H, int per, int d, int dv, const float* m_state, const float* nq, const float* m_rows) {
    return (mode == SS_MLSTM || mode == SS_MAMBA) && H > 0 && per > 0 && d > 0 && dv > 0 && d <= 512 &&
           (mode == SS_MAMBA || (m_state && nq && m_rows));
}

// the recurrence token by token; q, k, v and the gates in one dtype (float, planes allowed, or bf16)
extern "C" int kb_gated_scan(SS_PARAMS, cudaStream_t st) {
    if (B <= 0) return 0;
    if (!ss_ok(mode, H, per, d, dv, m_state, nq, m_rows)) return (int)cudaErrorInvalidValue;
    const SsArgs a = ss_args(SS_PASS);
    const int rows = dv + (mode == SS_MLSTM ? 1 : 0);
    // four columns a warp where that still leaves a block or more an SM
    const int nc = d <= 128 && (long long)B * H * ((rows + 4 * SS_COLS - 1) / (4 * SS_COLS)) >= 148 ? 4 : 1;
    const int cols = SS_COLS * nc;
    const dim3 grid(B * H, (rows + cols - 1) / cols);
    const size_t sm = (size_t)(2 * SS_STAGE * d + SS_STAGE * cols + 3 * SS_STAGE + 1) * sizeof(float);
#define SS_GO1(T, MODE, DPL, NC)                                                                                       \
    do {                                                                                                               \
        if (sm > 48 * 1024)                                                                                            \
            cudaFuncSetAttribute(k_gated_scan<T, MODE, DPL, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm); \
        kb_launch(k_gated_scan<T, MODE, DPL, NC>, grid, 32 * SS_COLS, sm, st, a);                                      \
    } while (0)
#define SS_GO(T, MODE)                                                                                                 \
    do {                                                                                                               \
        if (d <= 64) { if (nc == 4) SS_GO1(T, MODE, 2, 4); else SS_GO1(T, MODE, 2, 1); }                               \
        else if (d <= 128) { if (nc == 4) SS_GO1(T, MODE, 4, 4); else SS_GO1(T, MODE, 4, 1); }                         \
        else if (d <= 256) SS_GO1(T, MODE, 8, 1);                                                                      \
        else SS_GO1(T, MODE, 16, 1);                                                                                   \
    } while (0)
    if (dtype == KB_F32) {
        if (mode == SS_MLSTM) SS_GO(float, SS_MLSTM); else SS_GO(float, SS_MAMBA);
    } else {
        if (mode == SS_MLSTM) SS_GO(bf16, SS_MLSTM); else SS_GO(bf16, SS_MAMBA);
    }
#undef SS_GO
#undef SS_GO1
    KB_LAUNCH_RET();
}

extern "C" int kb_scan_run() { return SS_C; }

// the same over long prompts, a sequence's runs of SS_C tokens side by side: q, k, v and the gates as bf16 rows, d <= 256.
// scratch: gates [2][H][T] floats, part [runs][H][rows][d] floats, lg_end [runs][H] floats with runs = T / SS_C + B
extern "C" int kb_gated_scan_chunked(SS_PARAMS, int T, float* gates, float* part, float* lg_end, cudaStream_t st) {
    if (B <= 0 || T <= 0) return 0;
    if (!ss_ok(mode, H, per, d, dv, m_state, nq, m_rows) || dtype != KB_BF16 || n_planes != 1 || g_planes != 1 || d > 256 ||
        B > 65535 || H > 65535)
        return (int)cudaErrorInvalidValue;
    const SsArgs a = ss_args(SS_PASS);
    const int rows = dv + (mode == SS_MLSTM ? 1 : 0), dp = (d + 15) / 16 * 16;
    const int runs = T / SS_C + B, ez = (dv + SS_E - 1) / SS_E;
    float* ldg_ = gates, *w = gates + (size_t)H * T;
    const uintptr_t base = (uintptr_t)src;
    // what may be moved in 16-byte words: bit 0 queries and keys, bit 2 values, bit 4 the state; in pairs: bit 1 values, bit 3
    // the output
    const bool rows16 = base % 16 == 0 && ld % 8 == 0;
    const int vec = (rows16 && oq % 8 == 0 && ok % 8 == 0 && d % 8 == 0 ? 1 : 0) |
                    (base % 4 == 0 && ld % 2 == 0 && ov % 2 == 0 && dv % 2 == 0 ? 2 : 0) |
                    (rows16 && ov % 8 == 0 && dv % 8 == 0 ? 4 : 0) |
                    ((uintptr_t)out % 8 == 0 && ldo % 2 == 0 && dv % 2 == 0 ? 8 : 0) |
                    ((uintptr_t)part % 16 == 0 && d % 4 == 0 ? 16 : 0);
    const size_t sm_a = (size_t)(KB_SPLIT * SS_C * SS_LD + SS_C * (dp + 8)) * 2;
    const size_t tile_s = (size_t)KB_SPLIT * SS_E * SS_LD, tile_kv = (size_t)SS_C * SS_LD + (size_t)SS_C * (dp + 8);
    const size_t sm_c = ((size_t)SS_C * (dp + 8) + (tile_s > tile_kv ? tile_s : tile_kv)) * 2;
    const dim3 grid(runs, H, ez);
    const int n_el = rows * d;
    const bool v4 = n_el % 4 == 0 && (uintptr_t)state % 16 == 0 && state_stride % 4 == 0 && (uintptr_t)part % 16 == 0;
#define SS_GO(MODE)                                                                                                    \
    do {                                                                                                               \
        static char tag;                                                                                               \
        if (kb_first_use(&tag)) {                                                                                      \
            cudaFuncSetAttribute(k_chunk_state<MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024);        \
            cudaFuncSetAttribute(k_chunk_out<MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024);          \
        }                                                                                                              \
        kb_launch(k_scan_gates<bf16, MODE>, dim3(H, B, MODE == SS_MAMBA ? 4 : 1), MODE == SS_MAMBA ? 256 : SG_T, 0, st, a, ldg_, w, T);          \
        kb_launch(k_chunk_state<MODE>, grid, SS_THREADS, sm_a, st, a, (const float*)ldg_, (const float*)w, T, part,    \
                  lg_end, dp, vec);                                                                                    \
        if (v4)                                                                                                        \
            kb_launch(k_chunk_prefix<4>, dim3((n_el / 4 + 255) / 256, H, B), 256, 0, st, a, part,                      \
                      (const float*)lg_end, n_el);                                                                     \
        else                                                                                                           \
            kb_launch(k_chunk_prefix<1>, dim3((n_el + 255) / 256, H, B), 256, 0, st, a, part, (const float*)lg_end,    \
                      n_el);                                                                                           \
        kb_launch(k_chunk_out<MODE>, grid, SS_THREADS, sm_c, st, a, (const float*)ldg_, (const float*)w, T,            \
                  (const float*)part, dp, vec);                                                                        \
    } while (0)
    if (mode == SS_MLSTM) SS_GO(SS_MLSTM); else SS_GO(SS_MAMBA);
#undef SS_GO
    KB_LAUNCH_RET();
}

extern "C" int kb_scan_norm(int mode, const float* x, int ldx, int T, int NG, int n, const float* w, float eps,
                            const void* g, int gdtype, int g_planes, long long g_plane_stride, int ldg, int og,
                            const float* nq, const float* m_rows, float* m_state, long long m_stride, const int* pos,
                            const int* seq, const int* slot, const int* q_start, void* out, int odtype, int ldo,
                            cudaStream_t st) {
    if (T <= 0 || NG <= 0) return 0;
    if ((mode == SS_MLSTM && (!nq || !m_rows || !m_state)) || n < 1) return (int)cudaErrorInvalidValue;
    const bool wide = n > 512;
    const size_t sm = (size_t)(wide ? 1 : 8) * ((n + 3) & ~3) * sizeof(float);
    if (sm > 200 * 1024) return (int)cudaErrorInvalidValue;
    const int gpb = wide ? 1 : 8;
    const long long blocks = ((long long)T * NG + gpb - 1) / gpb;
    const int gel = gdtype == KB_F32 ? 4 : 2, oel = odtype == KB_F32 ? 4 : 2;
    const bool v4 = n % 4 == 0 && ldx % 4 == 0 && ldg % 4 == 0 && og % 4 == 0 && g_plane_stride % 4 == 0 && ldo % 4 == 0 &&
                    (uintptr_t)x % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)g % (4 * gel) == 0 && (uintptr_t)out % (4 * oel) == 0;
    // (the register forms need no shared memory)
    const int ni = !v4 ? 0 : (n / 4 + (wide ? 255 : 31)) / (wide ? 256 : 32);
#define SS_N(TG, TO, MODE, TPG, VW, NI)                                                                                \
    do {                                                                                                               \
        if (NI == 0 && sm > 48 * 1024)                                                                                 \
            cudaFuncSetAttribute(k_scan_norm<TG, TO, MODE, TPG, VW, NI>, cudaFuncAttributeMaxDynamicSharedMemorySize,  \
                                 (int)sm);                                                                             \
        kb_launch(k_scan_norm<TG, TO, MODE, TPG, VW, NI>, (unsigned)blocks, 256, NI ? (size_t)0 : sm, st, x, ldx, T,   \
                  NG, n, w, eps, (const TG*)g, g_planes, (size_t)g_plane_stride, ldg, og, nq, m_rows, m_state,         \
                  (size_t)m_stride, pos, seq, slot, q_start, (TO*)out, ldo);                                           \
    } while (0)
#define SS_N3(TG, TO, MODE, TPG)                                                                                       \
    do {                                                                                                               \
        if (ni == 1) SS_N(TG, TO, MODE, TPG, 4, 1);                                                                    \
        else if (ni >= 2 && ni <= 4) SS_N(TG, TO, MODE, TPG, 4, 4);                                                    \
        else if (v4) SS_N(TG, TO, MODE, TPG, 4, 0);                                                                    \
        else SS_N(TG, TO, MODE, TPG, 1, 0);                                                                            \
    } while (0)
#define SS_N2(TG, TO, MODE) do { if (wide) SS_N3(TG, TO, MODE, 256); else SS_N3(TG, TO, MODE, 32); } while (0)
#define SS_N1(TG, TO) do { if (mode == SS_MLSTM) SS_N2(TG, TO, SS_MLSTM); else SS_N2(TG, TO, SS_MAMBA); } while (0)
    if (gdtype == KB_F32 && odtype == KB_F32) SS_N1(float, float);
    else if (gdtype == KB_F32 && odtype == KB_BF16) SS_N1(float, bf16);
    else if (gdtype == KB_BF16 && odtype == KB_BF16) SS_N1(bf16, bf16);
    else return (int)cudaErrorInvalidValue;
#undef SS_N1
#undef SS_N2
#undef SS_N3
#undef SS_N
    KB_LAUNCH_RET();
}
