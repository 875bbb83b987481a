// Time mixing with a decay per key channel (the WKV recurrence of RWKV-6). Per head, with a bonus u for the current token:
//
//     o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t,      S_t = diag(w_t) S_(t-1) + k_t v_t^T
//
// where w_t = exp(-exp(z_t + w0)), z_t a low-rank projection W2 tanh(.) of the token. Rows arrive in bf16 or in 32-bit (as
// planes that are summed in order); everything else is 32-bit.
//   k_token_mix   the inputs of the projections: every stream's own mix of a row and the row before it
//   k_tanh_rows   tanh of the low-rank projection's rows
//   k_wkv_scan    token by token, for single tokens, short steps and the true 32-bit path: a warp per state column
// The state is kept per cache slot as [H][dv][d]. Rows of a step that belong to no sequence (padding of a recorded step) are
// not touched; their mixes are zeros.
#include "common.cuh"
#include <math.h>

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
    for (int s = 0; s < n; s++) {
        const float* m = mu + (size_t)s * E + c;
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
    const bool vec = E % v == 0 && ldo % v == 0 && (uintptr_t)y % (v * el) == 0 && (uintptr_t)out % (v * el) == 0;
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
template <typename T>
__global__ void __launch_bounds__(256) k_tanh_rows(const T* KB_STEP_DATA a, int lda, T* __restrict__ out, int N, long long n) {
    kb_pdl_launch();
    kb_pdl_wait();
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i >= n) return;
    out[i] = kb_from_f<T>(tanhf(kb_to_f<T>(a[(i / N) * lda + i % N])));
}

extern "C" int kb_tanh_rows(const void* a, int dtype, int lda, void* out, int T, int N, cudaStream_t st) {
    const long long n = (long long)T * N;
    if (n <= 0) return 0;
    const unsigned grid = (unsigned)((n + 255) / 256);
    if (dtype == KB_F32) kb_launch(k_tanh_rows<float>, grid, 256, 0, st, (const float*)a, lda, (float*)out, N, n);
    else kb_launch(k_tanh_rows<bf16>, grid, 256, 0, st, (const bf16*)a, lda, (bf16*)out, N, n);
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

template <typename T>
__device__ __forceinline__ float wk_rd(const T* p, int n_planes, size_t plane_stride) {
    float v = kb_to_f<T>(p[0]);
    for (int s = 1; s < n_planes; s++) v += kb_to_f<T>(p[(size_t)s * plane_stride]);
    return v;
}
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
            float z;
            if (a.z != nullptr) z = a.z[(size_t)(c0 + t) * a.ldz + ok + j];
            else {
                const TW* w = (const TW*)a.w2 + (ok + j) * a.rank;
                z = 0.0f;
                for (int q = 0; q < a.rank; q++) z = fmaf(lo[t * a.rank + q], kb_to_f<TW>(w[q]), z);
            }
            ws[idx] = wk_decay(z + a.w0[ok + j]);
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

#define WK_PARAMS                                                                                                      \
    int dtype, const void *r, const void *k, const void *v, int n_planes, long long plane_stride, int ld, const float *z, \
        int ldz, const void *low, int low_planes, long long low_stride, int ld_low, const void *w2, int w2dtype, int rank, \
        const float *w0, const float *u, int B, int H, int d, int dv, const int *q_start, const int *slot, float *state, \
        long long state_stride, float *out, int ldo

// the recurrence token by token; r, k, v in one dtype (float, planes allowed, or bf16), the decay's exponent either finished
// (z) or as the low-rank projection of the same dtype with W2
extern "C" int kb_wkv_scan(WK_PARAMS, cudaStream_t st) {
    if (B <= 0) return 0;
    if (H <= 0 || d <= 0 || dv <= 0 || d > 256 || (!z && (!low || !w2 || rank < 1 || rank > 512))) return (int)cudaErrorInvalidValue;
    WkvArgs a;
    a.r = r; a.k = k; a.v = v; a.n_planes = n_planes; a.plane_stride = (size_t)plane_stride; a.ld = ld;
    a.z = z; a.ldz = ldz; a.low = low; a.low_planes = low_planes; a.low_stride = (size_t)low_stride; a.ld_low = ld_low;
    a.w2 = w2; a.rank = rank; a.w0 = w0; a.u = u; a.B = B; a.H = H; a.d = d; a.dv = dv; a.q_start = q_start; a.slot = slot;
    a.state = state; a.state_stride = (size_t)state_stride; a.out = out; a.ldo = ldo;
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
