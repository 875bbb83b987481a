// Shared helpers of the kernel library: storage types, the status word, launch checks.
//
// Every entry point is extern "C", takes raw device pointers and a stream, and returns the cudaError_t of its
// launch as an int. Kernels never trap: an index that is out of range (a token id beyond the table, a page that is
// not mapped) sets a bit in the caller's status word and the access is skipped, so the context stays usable and
// the host can raise an error after the step.
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <stdint.h>

#define KB_F32 0
#define KB_BF16 1

#define KB_PAGE 64                 // positions per cache page

// status bits
#define KB_ST_BAD_TOKEN 1
#define KB_ST_BAD_PAGE 2
#define KB_ST_WAIT_TIMEOUT 4
#define KB_ST_BAD_ROW 8

typedef __nv_bfloat16 bf16;

template <typename T> __device__ __forceinline__ float kb_to_f(T v);
template <> __device__ __forceinline__ float kb_to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float kb_to_f<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T kb_from_f(float v);
template <> __device__ __forceinline__ float kb_from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 kb_from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float kb_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float kb_warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// where a sequence's keys and values live: pool of pages [page][2][n_kv][KB_PAGE][head_dim] for one cache entry,
// and the table that maps (slot, position / KB_PAGE) to a page. one_plane: a position's value is the beginning of its key, a
// page is [n_kv][KB_PAGE][head_dim]
struct KbCacheView {
    void* pool;                 // this cache entry's pages
    const int* table;           // [n_slots][table_stride]
    int table_stride;
    int n_pages;
    int n_kv;
    int head_dim;
    int one_plane;
};

__device__ __forceinline__ size_t kb_kv_offset(const KbCacheView& c, int page, int kv, int head, int p_in_page) {
    const size_t plane = c.one_plane ? (size_t)page : (size_t)page * 2 + kv;
    return ((plane * c.n_kv + head) * KB_PAGE + p_in_page) * (size_t)c.head_dim;
}

// activations of a feed-forward that takes its activation as a parameter
#define KB_ACT_NONE 0
#define KB_ACT_RELU2 1
#define KB_ACT_SILU 2
#define KB_ACT_GELU_TANH 3
__device__ __forceinline__ float kb_act(float z, int act) {
    switch (act) {
        case KB_ACT_RELU2: {
            const float r = fmaxf(z, 0.0f);
            return r * r;
        }
        case KB_ACT_SILU: return z / (1.0f + expf(-z));
        case KB_ACT_GELU_TANH:
            return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
        default: return z;
    }
}

// the gate of a gated feed-forward (act(gate) * up) inside a product's epilogue, with the fast exponential and
// division (their error is far below one bf16 rounding): silu(g) = g / (1 + exp(-g)), and the tanh form of GELU is
// the same shape, gelu_tanh(g) = g / (1 + exp(-2 u)) with u = sqrt(2 / pi) (g + 0.044715 g^3)
__device__ __forceinline__ float kb_gate_act_fast(float g, int act) {
    const float e = act == KB_ACT_GELU_TANH ? -1.5957691216057308f * (g + 0.044715f * g * g * g) : -g;
    return __fdividef(g, 1.0f + __expf(e));
}

// the gated unit a product finishes in its epilogue: which activation, and for the clamped unit its two constants.
// KB_ACT_GLU_CLAMP: g' sigmoid(alpha g') (u' + 1) with g' = min(g, lim), u' = clamp(u, -lim, lim)
#define KB_ACT_GLU_CLAMP 4
// A product without a gated unit may finish its rows instead: out = act(v + bias), `post` the activation's code (-1: the
// rows leave as they are) and `bias` a float per output column (null: none).
struct KbGate {
    int act;
    float lim, alpha;
    int post;
    const float* bias;
};
__device__ __forceinline__ float kb_post_act(float z, int post) {
    if (post == KB_ACT_RELU2) {
        const float r = fmaxf(z, 0.0f);
        return r * r;
    }
    return post == KB_ACT_NONE ? z : kb_gate_act_fast(z, post);
}
// the biases of 32 neighbouring columns, all loads in flight (columns from n_cols on: zero)
__device__ __forceinline__ void kb_post_bias32(float (&b)[32], int col, int n_cols, const KbGate& k) {
    if (k.bias != nullptr && col + 32 <= n_cols && (((uintptr_t)(k.bias + col)) & 15) == 0) {
#pragma unroll
        for (int c = 0; c < 32; c += 4) {
            const float4 v = __ldg((const float4*)(k.bias + col + c));
            b[c] = v.x; b[c + 1] = v.y; b[c + 2] = v.z; b[c + 3] = v.w;
        }
        return;
    }
#pragma unroll
    for (int c = 0; c < 32; c++) b[c] = k.bias != nullptr && col + c < n_cols ? __ldg(k.bias + col + c) : 0.0f;
}
__device__ __forceinline__ void kb_post32(uint32_t (&r)[32], const float (&b)[32], int post) {
    if (post == KB_ACT_RELU2) {
#pragma unroll
        for (int c = 0; c < 32; c++) {
            const float z = fmaxf(__uint_as_float(r[c]) + b[c], 0.0f);
            r[c] = __float_as_uint(z * z);
        }
        return;
    }
#pragma unroll
    for (int c = 0; c < 32; c++) r[c] = __float_as_uint(kb_post_act(__uint_as_float(r[c]) + b[c], post));
}
__device__ __forceinline__ float kb_glu_fast(float g, float u, const KbGate& k) {
    if (k.act == KB_ACT_GLU_CLAMP) {
        g = fminf(g, k.lim);
        u = fminf(fmaxf(u, -k.lim), k.lim) + 1.0f;
        return __fdividef(g, 1.0f + __expf(-k.alpha * g)) * u;
    }
    return kb_gate_act_fast(g, k.act) * u;
}
// (an entry point's activation code: 0, 1 and KB_ACT_SILU all mean silu)
static inline KbGate kb_gate_of(int act, float lim, float alpha) {
    KbGate k;
    k.act = act == KB_ACT_GELU_TANH ? KB_ACT_GELU_TANH : act == KB_ACT_GLU_CLAMP ? KB_ACT_GLU_CLAMP : KB_ACT_SILU;
    k.lim = lim;
    k.alpha = alpha;
    k.post = -1;
    k.bias = nullptr;
    return k;
}

// The first position that the row at position p sees: with a window the last `window` positions, with chunks (counted from
// the sequence's first position) its own chunk's
__device__ __forceinline__ int kb_span_lo(int p, int window, int chunk) {
    int lo = window > 0 && p - window + 1 > 0 ? p - window + 1 : 0;
    if (chunk > 0) lo = max(lo, p / chunk * chunk);
    return lo;
}

// A cap on attention scores, s -> cap tanh(s / cap), for kernels that work in powers of two: kb_cap2 turns a raw product
// q . k into log2(e) cap tanh(scale (q . k) / cap). mode 0: no cap. mode 1: tanh(u) = 1 - 2 / (1 + e^(2u)) with the fast
// exponential and reciprocal (2^-22 of the cap). mode 2: products known to stay within a bound (unit-norm queries and
// keys), where an odd polynomial of degree 11 in the product, made on the host by Chebyshev interpolation, is as exact
// and needs no special function. bounded: the capped scores lie so close to zero that exponentials and their sums cannot
// leave the 32-bit range, so that no running maximum is needed.
struct KbCap {
    int mode, bounded;
    float a;                    // 2 log2(e) scale / cap
    float out2;                 // log2(e) cap
    float k[6];                 // mode 2: s2 = x (k0 + k1 x^2 + ... + k5 x^10)
};
__device__ __forceinline__ float kb_cap2(float x, const KbCap& c) {
    if (c.mode == 2) {
        const float r = x * x;
        float p = c.k[5];
#pragma unroll
        for (int i = 4; i >= 0; i--) p = fmaf(p, r, c.k[i]);
        return p * x;
    }
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * c.a));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(e + 1.0f));
    return c.out2 * fmaf(-2.0f, r, 1.0f);
}
// host: ten floats (mode, bounded, a, out2, k0 .. k5), or null for no cap
static inline KbCap kb_cap_of(const float* h) {
    KbCap c = {};
    if (h) {
        c.mode = (int)h[0];
        c.bounded = (int)h[1];
        c.a = h[2];
        c.out2 = h[3];
        for (int i = 0; i < 6; i++) c.k[i] = h[4 + i];
    }
    return c;
}

#define KB_LAUNCH_RET() return (int)cudaGetLastError()

// Programmatic dependent launch. Every kernel of the library begins with kb_pdl_launch() (when its grid is small,
// the next kernel of the stream may be scheduled as soon as all CTAs of this one have started) and calls
// kb_pdl_wait() before its first
// read of anything an earlier kernel wrote and before its first global write (until then it may only set up
// barriers and tensor memory and fetch weights, which no kernel writes). The wait returns when the whole preceding
// kernel has finished and its writes are visible, so results are those of strictly ordered launches; what is
// gained is that launch latency and prologues overlap the predecessor's tail.
// Before its wait a kernel also reads the step's metadata (positions, lengths, slots, row lists, the page table)
// and cache pages of older positions (a recurrence's token-by-token kernel its states of earlier steps). Callers therefore write those with operations that are complete before the
// step's first kernel starts: the engine brings the page table up to date and then copies the metadata to the
// device (a copy orders fully), and older pages were stored by earlier steps.
__device__ __forceinline__ void kb_pdl_launch_now() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
// Small grids (decode steps) let their successor start at once; large grids (prompt steps) do not: a successor that
// was launched before its predecessor ended was measured to cost a prompt step several microseconds per kernel,
// whether the trigger came at the start of the blocks or after their last loads.
__device__ __forceinline__ void kb_pdl_launch() {
    if (gridDim.x * gridDim.y * gridDim.z <= 1024u) kb_pdl_launch_now();
}
__device__ __forceinline__ void kb_pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
// A kernel parameter that points at what an earlier kernel of the same step wrote (activations, split-K planes,
// partial results, logits) is marked KB_STEP_DATA and is NOT declared __restrict__: for a const __restrict__ pointer the
// compiler may take the data for read-only during the whole kernel and move its loads above the wait (seen with the
// 32-bit product: loads placed right after the wait were issued before it and read what the kernel before had not
// written yet). Weights, tables and the step's metadata are written before the step's first kernel and keep
// __restrict__: they are meant to be read early.
#define KB_STEP_DATA

extern int g_kb_pdl;            // 1: launches carry the programmatic-serialization attribute

#ifdef __cplusplus
#include <utility>
#include <mutex>
#include <unordered_set>
// true the first time it is asked about this kernel on the current device, false ever after: function attributes
// (the shared-memory opt-in, the carve-out) belong to a device, so they are set once per (device, kernel). Safe to
// call from several host threads.
static inline bool kb_first_use(const void* kern) {
    static std::mutex mu;
    static std::unordered_set<uint64_t> seen;
    int dev = 0;
    cudaGetDevice(&dev);
    const uint64_t key = ((uint64_t)(uintptr_t)kern << 8) ^ (uint64_t)(dev & 0xff);
    std::lock_guard<std::mutex> g(mu);
    return seen.insert(key).second;
}
// Every kernel of the library asks for the largest shared-memory partition of the SM, the one its tensor-core
// kernels need: an SM re-partitions L1 and shared memory only when it is idle, so a step whose kernels all want the
// same partition never waits for that, and a kernel launched early can become resident beside its predecessor.
static inline void kb_same_partition(const void* kern) {
    if (kb_first_use(kern))
        cudaFuncSetAttribute(kern, cudaFuncAttributePreferredSharedMemoryCarveout, (int)cudaSharedmemCarveoutMaxShared);
}
template <typename... KArgs, typename... Args>
static inline cudaError_t kb_launch(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st,
                                    Args&&... args) {
    kb_same_partition((const void*)kern);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = g_kb_pdl ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kern, std::forward<Args>(args)...);
}
#endif
