// Attention over a cache of latents: every position holds ONE vector that all query heads share, [latent | rotated key part |
// zeros] of HD elements (a multiple of 64). It is the key of every head, and its first DV elements are the value, so a page
// is stored once, fetched once and read twice: as the K-major operand of Q K^T and as the MN-major operand of P V.
//
//   k_latent_tc      prompt-sized steps (tcgen05). A CTA takes up to 128 rows r = token * G + head of one sequence. S = Q K^T
//                    and O += P V are tcgen05.mma instructions with accumulators in tensor memory, P goes back to tensor
//                    memory as bf16 over the scores it came from, and the exponent's reference moves lazily; the arrangement
//                    is k_attn_tc's. Tiles of KEYS positions (64; 32 for heads whose queries fill most of the shared memory).
//                    Values of more than 256 elements do not fit tensor memory beside the scores: blockIdx.x then also
//                    counts parts of 256 value columns, and every part takes the scores anew.
//   k_latent_decode  single tokens. A CTA takes 16 or 32 heads of one sequence and a stretch of its pages. Four warps: each
//                    scores 16 of a page's 64 positions, the scores meet in shared memory, and each warp then has the whole
//                    page's weights for its quarter of the value columns.
//   k_latent_merge   position splits of a decode step, merged in split order.
//   k_latent_full    prompt-sized steps with every head's keys and values expanded from the latents (a product over all cached
//                    positions of the step's sequences, gathered by k_latent_gather): fewer multiplications per query and key,
//                    worth their making where a step brings a fair share of its sequences' positions. A CTA takes 128 tokens
//                    of one head; its key tile is the head's plain part beside the rotated part that all heads share. The
//                    queries' rotation happens on their way into shared memory, a gate per head on the way out.
// bf16 in and out, 32-bit sums and softmax; every wait is bounded.
#include "sm100.cuh"
#include "mma_sync.cuh"

#define LT_THREADS 192
#define LT_LAZY 8.0f

__device__ __forceinline__ float lt_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void lt_tmem_st32(uint32_t taddr, const uint32_t* r) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
        "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
        ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
          "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]),
          "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]),
          "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
        : "memory");
}
__device__ __forceinline__ void lt_tmem_st16(uint32_t taddr, const uint32_t* r) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
        "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
        ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
          "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
        : "memory");
}
__device__ __forceinline__ void lt_tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// an MN-major operand tile stored as rows of 128 bytes (64 elements of the MN dimension a row, one row per K index), 128-byte
// swizzle: leading byte offset = distance to the next block of 64 MN elements, stride byte offset = 8 K rows (1024)
__device__ __forceinline__ uint64_t lt_desc_mn(uint32_t smem_addr, uint32_t lbo_bytes) {
    uint64_t d = 0;
    d |= (uint64_t)((smem_addr & 0x3FFFFu) >> 4);
    d |= (uint64_t)((lbo_bytes >> 4) & 0x3FFFu) << 16;
    d |= (uint64_t)(1024 >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}

// one tile of a softmax thread's row: scores from tensor memory (t_s, this warp's lanes), probabilities back over them as bf16,
// O (t_o, n_cols columns) rescaled where the row's reference moved, then the tile handed over to the product with the values.
// False: a wait ran out
template <int KEYS>
__device__ __forceinline__ bool lt_softmax_tile(uint32_t t_s, uint32_t t_o, int n_cols, int j, int key0, int p_row,
        float scale_log2e, float& m_ref, float& l, uint32_t b_pv_done, uint32_t b_p_ready, int lane, int* status) {
    tc_fence_after();
    uint32_t sv[KEYS];
#pragma unroll
    for (int c = 0; c < KEYS; c += 32) tmem_ld_32x32(t_s + c, sv + c);
    tmem_ld_wait();
    tc_fence_before();
    __syncwarp();
    float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
    if (key0 + KEYS - 1 <= p_row) {
#pragma unroll
        for (int c = 0; c < KEYS; c++) mx4[c & 3] = fmaxf(mx4[c & 3], __uint_as_float(sv[c]));
    } else {
#pragma unroll
        for (int c = 0; c < KEYS; c++) {
            const float s = key0 + c <= p_row ? __uint_as_float(sv[c]) : -INFINITY;
            sv[c] = __float_as_uint(s);
            mx4[c & 3] = fmaxf(mx4[c & 3], s);
        }
    }
    const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * scale_log2e;
    const bool grow = mx > m_ref + LT_LAZY || (m_ref == -INFINITY && mx > -INFINITY);
    float f = 1.0f;
    if (grow) {
        f = m_ref == -INFINITY ? 0.0f : lt_exp2(m_ref - mx);
        m_ref = mx;
        l *= f;
    }
    // P V of tile j - 1 done means: O holds tiles 0..j-1. A rescale of O waits for that here, otherwise the wait comes
    // just before this tile's P is handed over (once per tile, in order)
    const bool rescale = __any_sync(0xffffffffu, grow) && j > 0;
    if (rescale) {
        if (!mbar_wait(b_pv_done, (uint32_t)(j - 1) & 1u, status)) return false;
        __syncwarp();
        tc_fence_after();
#pragma unroll 1
        for (int c0 = 0; c0 < n_cols; c0 += 32) {
            uint32_t ov[32];
            tmem_ld_32x32(t_o + c0, ov);
            tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < 32; c++) ov[c] = __float_as_uint(__uint_as_float(ov[c]) * f);
            lt_tmem_st32(t_o + c0, ov);
        }
        lt_tmem_st_wait();
    }
    const float nmr = m_ref == -INFINITY ? 0.0f : -m_ref;
    float sum[4] = {0.f, 0.f, 0.f, 0.f};
    uint32_t pv[KEYS / 2];
#pragma unroll
    for (int c = 0; c < KEYS; c += 2) {
        const float p0 = lt_exp2(fmaf(__uint_as_float(sv[c]), scale_log2e, nmr));
        const float p1 = lt_exp2(fmaf(__uint_as_float(sv[c + 1]), scale_log2e, nmr));
        sum[(c >> 1) & 3] += p0 + p1;
        pv[c >> 1] = pack_bf16(p0, p1);
    }
    l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
    if (KEYS == 64) lt_tmem_st32(t_s, pv);
    else lt_tmem_st16(t_s, pv);
    lt_tmem_st_wait();
    if (j > 0 && !rescale) {
        if (!mbar_wait(b_pv_done, (uint32_t)(j - 1) & 1u, status)) return false;
    }
    tc_fence_before();
    __syncwarp();
    if (lane == 0) mbar_arrive(b_p_ready);
    return true;
}

template <int HD, int KEYS, int STAGES>
struct LtSmem {
    static constexpr int Q_BYTES = 128 * HD * 2, TILE_BYTES = KEYS * HD * 2;
    static constexpr int BARS = Q_BYTES + STAGES * TILE_BYTES;
    static constexpr int TOTAL = BARS + (2 * STAGES + 4) * 8 + 16 + 1024;
    static_assert(TOTAL <= 227 * 1024, "shared memory of a CTA");
};

// grid (head groups x value parts, tiles, sequences); dv_part: value columns of a part (a multiple of 16, at most 256)
template <int HD, int KEYS, int STAGES>
__global__ void __launch_bounds__(LT_THREADS, 2 * LtSmem<HD, KEYS, STAGES>::TOTAL <= 226 * 1024 ? 2 : 1)
        k_latent_tc(const __grid_constant__ CUtensorMap map, const bf16* KB_STEP_DATA q, int ldq, bf16* __restrict__ out, int ldo,
        int dv, int dv_part, int n_parts, const int* __restrict__ slot, const int* __restrict__ q_start,
        const int* __restrict__ kv_len, int G, float scale_log2e, const int* __restrict__ table, int table_stride, int n_pages,
        uint32_t tmem_cols, int* status) {
    using L = LtSmem<HD, KEYS, STAGES>;
    constexpr int BOX = KEYS * 128;                  // bytes of a 64-column box of a tile
    constexpr int PP = KB_PAGE / KEYS;               // tiles of a page
    extern __shared__ __align__(128) uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const uint32_t sbase = smem_u32(smem);
    const uint32_t s_q = sbase, s_kv = s_q + L::Q_BYTES;
    const uint32_t b_full = sbase + L::BARS, b_empty = b_full + STAGES * 8, b_s_full = b_empty + STAGES * 8;
    const uint32_t b_p_ready = b_s_full + 16, b_pv_done = b_p_ready + 8;
    volatile uint32_t* tmem_slot = (volatile uint32_t*)(smem + L::BARS + (2 * STAGES + 4) * 8);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int b = blockIdx.z, hg = blockIdx.x / n_parts, part = blockIdx.x % n_parts;
    const int c_lo = part * dv_part, n_cols = min(dv_part, (dv - c_lo + 15) / 16 * 16);

    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; s++) {
            mbar_init(b_full + s * 8, 1);
            mbar_init(b_empty + s * 8, 1);
        }
        for (int i = 0; i < 2; i++) mbar_init(b_s_full + i * 8, 1);
        mbar_init(b_p_ready, 4);
        mbar_init(b_pv_done, 1);
        mbar_fence_init();
        tma_prefetch_desc(&map);
    }
    if (warp == 5) {
        tmem_alloc(smem_u32((const void*)tmem_slot), tmem_cols);
        tmem_relinquish();
    }
    kb_pdl_wait();                       // Q and the newest latents come from earlier kernels
    const int qs0 = q_start[b], qlen = q_start[b + 1] - qs0, kvl = kv_len[b];
    const int pos0 = kvl - qlen;
    const int TOK = 128 / G;                         // whole tokens per CTA
    const int n_tiles = (qlen + TOK - 1) / TOK;
    const bool active = (int)blockIdx.y < n_tiles;   // uniform over the CTA
    const int tile = n_tiles - 1 - (int)blockIdx.y;  // the longest tiles first
    const int tok0 = tile * TOK;
    const int ntok = active ? min(TOK, qlen - tok0) : 0;
    const int nrows = ntok * G;
    const int n_iter = active ? (pos0 + tok0 + ntok - 1) / KEYS + 1 : 0;

    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    const uint32_t t_s = tmem, t_o = tmem + 2 * KEYS;

    // ---- Q into shared memory: blocks of [128 rows][64 columns], rows of 128 bytes, 128-byte swizzle
    if (warp != 4) {
        if (active) {
            constexpr int QT = LT_THREADS - 32, QV = 128 * (HD / 8), QN = 8;
            const int qt = warp < 4 ? (int)threadIdx.x : (int)threadIdx.x - 32;
#pragma unroll 1
            for (int e0 = 0; e0 < QV; e0 += QT * QN) {
                uint4 v[QN];
#pragma unroll
                for (int i = 0; i < QN; i++) {
                    const int e = e0 + qt + i * QT, r = e / (HD / 8), c = e % (HD / 8);
                    v[i] = make_uint4(0, 0, 0, 0);
                    if (e < QV && r < nrows)
                        v[i] = *(const uint4*)(q + (size_t)(qs0 + tok0 + r / G) * ldq + (size_t)(hg * G + r % G) * HD + c * 8);
                }
#pragma unroll
                for (int i = 0; i < QN; i++) {
                    const int e = e0 + qt + i * QT, r = e / (HD / 8), c = e % (HD / 8);
                    if (e < QV) *(uint4*)(smem + (c >> 3) * 16384 + r * 128 + (((c & 7) ^ (r & 7)) << 4)) = v[i];
                }
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        }
        asm volatile("bar.sync 1, %0;" ::"n"(LT_THREADS - 32) : "memory");
    }

    if (warp == 4) {
        // ------------------------------------------------------------ TMA producer
        if (lane == 0) {
            const int* trow = table + (size_t)slot[b] * table_stride;
            for (int i = 0; i < n_iter; i++) {
                const int s = i % STAGES;
                if (!mbar_wait(b_empty + s * 8, ((uint32_t)(i / STAGES) & 1u) ^ 1u, status)) break;
                int page = trow[i / PP];
                if (page < 0 || page >= n_pages) {
                    atomicOr(status, KB_ST_BAD_PAGE);
                    page = 0;
                }
                const int row = page * KB_PAGE + i % PP * KEYS;
                const uint32_t dst = s_kv + s * L::TILE_BYTES;
                mbar_expect_tx(b_full + s * 8, L::TILE_BYTES);
#pragma unroll
                for (int h = 0; h < HD / 64; h++) tma_load_2d(dst + h * BOX, &map, h * 64, row, b_full + s * 8);
            }
        }
    } else if (warp == 5) {
        // ------------------------------------------------------------ MMA issuer
        if (lane == 0 && n_iter > 0) {
            constexpr uint32_t idesc_s = umma_idesc_bf16(128, KEYS);                // Q K^T: both K-major
            const uint32_t idesc_o = umma_idesc_bf16(128, n_cols) | (1u << 16);     // P V: the values are MN-major
            bool ok = true;
            auto issue_s = [&](int j) {
                const uint32_t kt = s_kv + (j % STAGES) * L::TILE_BYTES;
                const uint32_t d = t_s + (uint32_t)(j & 1) * KEYS;
#pragma unroll
                for (int k = 0; k < HD / 16; k++)
                    umma_bf16(d, umma_desc_sw128(s_q + (k >> 2) * 16384 + (k & 3) * 32),
                              umma_desc_sw128(kt + (k >> 2) * BOX + (k & 3) * 32), idesc_s, k > 0 ? 1u : 0u);
                umma_commit(b_s_full + (j & 1) * 8);
            };
            ok = mbar_wait(b_full, 0, status);
            if (ok) {
                tc_fence_after();
                issue_s(0);
            }
            for (int j = 0; j < n_iter && ok; j++) {
                if (j + 1 < n_iter) {
                    const int s1 = (j + 1) % STAGES;
                    if (!(ok = mbar_wait(b_full + s1 * 8, (uint32_t)((j + 1) / STAGES) & 1u, status))) break;
                    // (the scores' buffer holds P of tile j - 1, whose product was issued before this one: the tensor pipe
                    // runs them in order)
                    tc_fence_after();
                    issue_s(j + 1);
                }
                if (!(ok = mbar_wait(b_p_ready, (uint32_t)j & 1u, status))) break;
                tc_fence_after();
                const uint32_t vt = s_kv + (j % STAGES) * L::TILE_BYTES + (c_lo >> 6) * BOX;
#pragma unroll
                for (int k = 0; k < KEYS / 16; k++)
                    umma_bf16_ts(t_o, t_s + (uint32_t)(j & 1) * KEYS + k * 8, lt_desc_mn(vt + k * 2048, BOX), idesc_o,
                                 (j > 0 || k > 0) ? 1u : 0u);
                umma_commit(b_pv_done);                           // O holds tiles 0..j
                umma_commit(b_empty + (j % STAGES) * 8);          // the tile has been read as keys and as values
            }
        }
    } else if (n_iter > 0) {
        // ------------------------------------------------------------ softmax: thread = row = TMEM lane
        const int r = warp * 32 + lane;
        const bool row_ok = r < nrows;
        const int p_row = row_ok ? pos0 + tok0 + r / G : 0x3fffffff;       // (padding rows see every key: no masked branch)
        const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
        float m_ref = -INFINITY, l = 0.0f;
        bool ok = true;
        for (int j = 0; j < n_iter && ok; j++) {
            const int bsel = j & 1;
            if (!(ok = mbar_wait(b_s_full + bsel * 8, (uint32_t)(j >> 1) & 1u, status))) break;
            __syncwarp();
            ok = lt_softmax_tile<KEYS>(t_s + lane_base + bsel * KEYS, t_o + lane_base, n_cols, j, j * KEYS, p_row, scale_log2e, m_ref,
                                       l, b_pv_done, b_p_ready, lane, status);
        }
        if (ok) ok = mbar_wait(b_pv_done, (uint32_t)(n_iter - 1) & 1u, status);
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
            tc_fence_after();
            const float inv = l > 0.0f ? 1.0f / l : 0.0f;
            bf16* dst = out + (size_t)(qs0 + tok0 + (row_ok ? r / G : 0)) * ldo + (size_t)(hg * G + (row_ok ? r % G : 0)) * dv + c_lo;
            const int n_out = min(n_cols, dv - c_lo);
            const bool v16 = dv % 8 == 0;
#pragma unroll 1
            for (int c0 = 0; c0 < n_cols; c0 += 32) {
                uint32_t ov[32];
                tmem_ld_32x32(t_o + lane_base + c0, ov);
                tmem_ld_wait();
                if (!row_ok) continue;
#pragma unroll
                for (int c = 0; c < 32; c += 8) {
                    uint32_t h[4];
#pragma unroll
                    for (int k = 0; k < 4; k++)
                        h[k] = pack_bf16(__uint_as_float(ov[c + 2 * k]) * inv, __uint_as_float(ov[c + 2 * k + 1]) * inv);
                    if (v16 && c0 + c + 8 <= n_out) {
                        *(uint4*)(dst + c0 + c) = make_uint4(h[0], h[1], h[2], h[3]);
                    } else {
                        const bf16* hb = (const bf16*)h;
#pragma unroll
                        for (int k = 0; k < 8; k++)
                            if (c0 + c + k < n_out) dst[c0 + c + k] = hb[k];
                    }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 5) {
        tc_fence_after();
        tmem_dealloc(tmem, tmem_cols);
    }
}

// ------------------------------------------------------------------------------------------------ expanded keys and values
// the cached latents and rotated parts of the step's sequences, one after another: row sum(kv_len[0 .. b)) + p of lat [N][kr] and
// rotk [N][rot]. A warp a row; 16-byte words
__global__ void __launch_bounds__(256) k_latent_gather(const bf16* KB_STEP_DATA pool, int hd, int kr, int rot,
        const int* __restrict__ slot, const int* __restrict__ kv_len, int B, const int* __restrict__ table, int table_stride,
        int n_pages, bf16* __restrict__ lat, bf16* __restrict__ rotk, int N, int* status) {
    kb_pdl_launch();
    kb_pdl_wait();
    const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= N) return;
    int b = 0, p = row;
    while (b + 1 < B && p >= kv_len[b]) p -= kv_len[b++];
    const int page = p < kv_len[b] ? table[(size_t)slot[b] * table_stride + p / KB_PAGE] : -1;
    const bool ok = page >= 0 && page < n_pages;
    if (!ok && lane == 0) atomicOr(status, KB_ST_BAD_PAGE);
    const uint4* src = (const uint4*)(pool + ((size_t)(ok ? page : 0) * KB_PAGE + p % KB_PAGE) * hd);
    for (int c = lane; c < (kr + rot) / 8; c += 32) {
        const uint4 v = ok ? src[c] : make_uint4(0, 0, 0, 0);
        if (c * 8 < kr) *(uint4*)(lat + (size_t)row * kr + c * 8) = v;
        else *(uint4*)(rotk + (size_t)row * rot + c * 8 - kr) = v;
    }
}

template <int KBX, int VBX>
struct LfSmem {
    static constexpr int QB = KBX + 1;
    static constexpr int Q_BYTES = QB * 16384, K_BYTES = QB * 8192, V_BYTES = VBX * 8192;
    static constexpr int V_OFF = Q_BYTES + 2 * K_BYTES, BARS = V_OFF + V_BYTES;
    static constexpr int TOTAL = BARS + 96 + 896;      // (the base is 128-byte aligned and moves up to the next 1024)
};
struct LfArgs {
    const bf16* q;              // rows [T][ldq]: heads of [d | rot]
    int ldq, d, rot, dv, n_heads;
    const float2* angles;       // [T][rot / 2]: cosine and sine of the row's angles
    float mult;
    int half;                   // pairs (i, i + rot / 2) instead of neighbours
    const bf16* gate;           // rows [T][ldg], one number a head, or null
    int ldg;
    bf16* out;                  // rows [T][ldo]: heads of dv
    int ldo;
    const int* q_start;
    const int* kv_len;
    float scale_log2e;
    int* status;
};

// kvmap: [N][n_heads d keys | n_heads dv values]; rotmap: [N][rot]. grid (heads, tiles of 128 tokens, sequences)
template <int KBX, int VBX>
__global__ void __launch_bounds__(LT_THREADS, 2) k_latent_full(const __grid_constant__ CUtensorMap kvmap,
        const __grid_constant__ CUtensorMap rotmap, LfArgs a) {
    using L = LfSmem<KBX, VBX>;
    constexpr int QB = L::QB;
    extern __shared__ __align__(128) uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const uint32_t sbase = smem_u32(smem);
    const uint32_t s_q = sbase, s_k = s_q + L::Q_BYTES, s_v = sbase + L::V_OFF;
    const uint32_t b_k_full = sbase + L::BARS, b_k_empty = b_k_full + 16, b_v_full = b_k_empty + 16, b_v_empty = b_v_full + 8;
    const uint32_t b_s_full = b_v_empty + 8, b_p_ready = b_s_full + 16, b_pv_done = b_p_ready + 8;
    volatile uint32_t* tmem_slot = (volatile uint32_t*)(smem + L::BARS + 80);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x, b = blockIdx.z;
    const int n_cols = (a.dv + 15) / 16 * 16;
    if (threadIdx.x == 0) {
        for (int i = 0; i < 2; i++) {
            mbar_init(b_k_full + i * 8, 1);
            mbar_init(b_k_empty + i * 8, 1);
            mbar_init(b_s_full + i * 8, 1);
        }
        mbar_init(b_v_full, 1);
        mbar_init(b_v_empty, 1);
        mbar_init(b_p_ready, 4);
        mbar_init(b_pv_done, 1);
        mbar_fence_init();
        tma_prefetch_desc(&kvmap);
        tma_prefetch_desc(&rotmap);
    }
    if (warp == 5) {
        tmem_alloc(smem_u32((const void*)tmem_slot), 256);
        tmem_relinquish();
    }
    kb_pdl_wait();
    const int qs0 = a.q_start[b], qlen = a.q_start[b + 1] - qs0, kvl = a.kv_len[b];
    int kv0 = 0;                                     // the sequence's first row among the expanded ones
    for (int i = 0; i < b; i++) kv0 += a.kv_len[i];
    const int pos0 = kvl - qlen;
    const int n_tiles = (qlen + 127) / 128;
    const bool active = (int)blockIdx.y < n_tiles;
    const int tok0 = (n_tiles - 1 - (int)blockIdx.y) * 128;          // the longest tiles first
    const int nrows = active ? min(128, qlen - tok0) : 0;
    const int n_iter = active ? (pos0 + tok0 + nrows - 1) / 64 + 1 : 0;
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    const uint32_t t_s = tmem, t_o = tmem + 128;

    if (warp != 4) {
        if (active) {
            constexpr int QT = LT_THREADS - 32, QV = 128 * QB * 8, QN = 8;
            const int qt = warp < 4 ? (int)threadIdx.x : (int)threadIdx.x - 32;
            const int rh = a.rot / 2;
#pragma unroll 1
            for (int e0 = 0; e0 < QV; e0 += QT * QN) {
                uint4 v[QN], w[QN];
#pragma unroll
                for (int i = 0; i < QN; i++) {
                    const int e = e0 + qt + i * QT, r = e / (QB * 8), c = e % (QB * 8);
                    v[i] = w[i] = make_uint4(0, 0, 0, 0);
                    if (e < QV && r < nrows) {
                        const bf16* row = a.q + (size_t)(qs0 + tok0 + r) * a.ldq + (size_t)h * (a.d + a.rot);
                        const int x = (c - KBX * 8) * 8;             // (rotated part)
                        if (c < KBX * 8) {
                            if (c * 8 < a.d) v[i] = *(const uint4*)(row + c * 8);
                        } else if (x < a.rot) {
                            v[i] = *(const uint4*)(row + a.d + x);
                            if (a.half) w[i] = *(const uint4*)(row + a.d + (x < rh ? x + rh : x - rh));
                        }
                    }
                }
#pragma unroll
                for (int i = 0; i < QN; i++) {
                    const int e = e0 + qt + i * QT, r = e / (QB * 8), c = e % (QB * 8);
                    if (e >= QV) continue;
                    const int x = (c - KBX * 8) * 8;
                    if (c >= KBX * 8 && x < a.rot && r < nrows) {
                        const float2* an = a.angles + (size_t)(qs0 + tok0 + r) * rh;
                        const bf16* vb = (const bf16*)&v[i], *wb = (const bf16*)&w[i];
                        float y[8];
                        if (a.half) {
                            const bool lo = x < rh;
#pragma unroll
                            for (int k = 0; k < 8; k++) {
                                const float2 cs = an[(lo ? x : x - rh) + k];
                                const float m = __bfloat162float(vb[k]) * (cs.x * a.mult), o = __bfloat162float(wb[k]) * (cs.y * a.mult);
                                y[k] = lo ? m - o : m + o;
                            }
                        } else {
#pragma unroll
                            for (int k = 0; k < 8; k += 2) {
                                const float2 cs = an[(x + k) / 2];
                                const float u0 = __bfloat162float(vb[k]), u1 = __bfloat162float(vb[k + 1]);
                                const float cc = cs.x * a.mult, sn = cs.y * a.mult;
                                y[k] = u0 * cc - u1 * sn;
                                y[k + 1] = u1 * cc + u0 * sn;
                            }
                        }
                        v[i] = make_uint4(pack_bf16(y[0], y[1]), pack_bf16(y[2], y[3]), pack_bf16(y[4], y[5]), pack_bf16(y[6], y[7]));
                    }
                    *(uint4*)(smem + (c >> 3) * 16384 + r * 128 + (((c & 7) ^ (r & 7)) << 4)) = v[i];
                }
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        }
        asm volatile("bar.sync 1, %0;" ::"n"(LT_THREADS - 32) : "memory");
    }

    if (warp == 4) {
        // ------------------------------------------------------------ TMA producer: two streams, one thread polls both
        if (lane == 0 && n_iter > 0) {
            int ik = 0, iv = 0, spins = 0;
            uint64_t t0 = 0;
            while (iv < n_iter) {
                bool moved = false;
                if (ik < n_iter && mbar_poll(b_k_empty + (ik & 1) * 8, ((uint32_t)(ik >> 1) & 1u) ^ 1u)) {
                    const uint32_t dst = s_k + (ik & 1) * L::K_BYTES, bar = b_k_full + (ik & 1) * 8;
                    mbar_expect_tx(bar, L::K_BYTES);
#pragma unroll
                    for (int c = 0; c < KBX; c++) tma_load_2d(dst + c * 8192, &kvmap, h * a.d + c * 64, kv0 + ik * 64, bar);
                    tma_load_2d(dst + KBX * 8192, &rotmap, 0, kv0 + ik * 64, bar);
                    ik++;
                    moved = true;
                }
                if (iv < ik && mbar_poll(b_v_empty, ((uint32_t)iv & 1u) ^ 1u)) {
                    mbar_expect_tx(b_v_full, L::V_BYTES);
#pragma unroll
                    for (int c = 0; c < VBX; c++)
                        tma_load_2d(s_v + c * 8192, &kvmap, a.n_heads * a.d + h * a.dv + c * 64, kv0 + iv * 64, b_v_full);
                    iv++;
                    moved = true;
                }
                if (moved) {
                    spins = 0;
                    continue;
                }
                __nanosleep(100);
                if (++spins >= 256) {
                    if (spins == 256) t0 = kb_globaltimer();
                    else if ((spins & 255) == 0 && kb_globaltimer() - t0 > KB_WAIT_NS) {
                        atomicOr(a.status, KB_ST_WAIT_TIMEOUT);
                        break;
                    }
                }
            }
        }
    } else if (warp == 5) {
        // ------------------------------------------------------------ MMA issuer
        if (lane == 0 && n_iter > 0) {
            constexpr uint32_t idesc_s = umma_idesc_bf16(128, 64);
            const uint32_t idesc_o = umma_idesc_bf16(128, n_cols) | (1u << 16);
            bool ok = true;
            auto issue_s = [&](int j) {
                const uint32_t kt = s_k + (j & 1) * L::K_BYTES, d = t_s + (uint32_t)(j & 1) * 64;
#pragma unroll
                for (int k = 0; k < QB * 4; k++)
                    umma_bf16(d, umma_desc_sw128(s_q + (k >> 2) * 16384 + (k & 3) * 32),
                              umma_desc_sw128(kt + (k >> 2) * 8192 + (k & 3) * 32), idesc_s, k > 0 ? 1u : 0u);
                umma_commit(b_s_full + (j & 1) * 8);
                umma_commit(b_k_empty + (j & 1) * 8);
            };
            ok = mbar_wait(b_k_full, 0, a.status);
            if (ok) {
                tc_fence_after();
                issue_s(0);
            }
            for (int j = 0; j < n_iter && ok; j++) {
                if (j + 1 < n_iter) {
                    if (!(ok = mbar_wait(b_k_full + ((j + 1) & 1) * 8, (uint32_t)((j + 1) >> 1) & 1u, a.status))) break;
                    tc_fence_after();
                    issue_s(j + 1);
                }
                if (!(ok = mbar_wait(b_p_ready, (uint32_t)j & 1u, a.status))) break;
                if (!(ok = mbar_wait(b_v_full, (uint32_t)j & 1u, a.status))) break;
                tc_fence_after();
#pragma unroll
                for (int k = 0; k < 4; k++)
                    umma_bf16_ts(t_o, t_s + (uint32_t)(j & 1) * 64 + k * 8, lt_desc_mn(s_v + k * 2048, 8192), idesc_o,
                                 (j > 0 || k > 0) ? 1u : 0u);
                umma_commit(b_pv_done);
                umma_commit(b_v_empty);
            }
        }
    } else if (n_iter > 0) {
        // ------------------------------------------------------------ softmax: thread = token = TMEM lane
        const int r = warp * 32 + lane;
        const bool row_ok = r < nrows;
        const int p_row = row_ok ? pos0 + tok0 + r : 0x3fffffff;
        const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
        float m_ref = -INFINITY, l = 0.0f;
        bool ok = true;
        for (int j = 0; j < n_iter && ok; j++) {
            if (!(ok = mbar_wait(b_s_full + (j & 1) * 8, (uint32_t)(j >> 1) & 1u, a.status))) break;
            __syncwarp();
            ok = lt_softmax_tile<64>(t_s + lane_base + (j & 1) * 64, t_o + lane_base, n_cols, j, j * 64, p_row, a.scale_log2e,
                                     m_ref, l, b_pv_done, b_p_ready, lane, a.status);
        }
        if (ok) ok = mbar_wait(b_pv_done, (uint32_t)(n_iter - 1) & 1u, a.status);
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
            tc_fence_after();
            const size_t t = (size_t)(qs0 + tok0 + (row_ok ? r : 0));
            float inv = l > 0.0f ? 1.0f / l : 0.0f;
            if (a.gate != nullptr) inv *= 1.0f / (1.0f + expf(-__bfloat162float(a.gate[t * a.ldg + h])));
            bf16* dst = a.out + t * a.ldo + (size_t)h * a.dv;
#pragma unroll 1
            for (int c0 = 0; c0 < n_cols; c0 += 32) {
                uint32_t ov[32];
                tmem_ld_32x32(t_o + lane_base + c0, ov);
                tmem_ld_wait();
                if (!row_ok) continue;
#pragma unroll
                for (int c = 0; c < 32; c += 8)
                    if (c0 + c < a.dv)
                        *(uint4*)(dst + c0 + c) =
                            make_uint4(pack_bf16(__uint_as_float(ov[c]) * inv, __uint_as_float(ov[c + 1]) * inv),
                                       pack_bf16(__uint_as_float(ov[c + 2]) * inv, __uint_as_float(ov[c + 3]) * inv),
                                       pack_bf16(__uint_as_float(ov[c + 4]) * inv, __uint_as_float(ov[c + 5]) * inv),
                                       pack_bf16(__uint_as_float(ov[c + 6]) * inv, __uint_as_float(ov[c + 7]) * inv));
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 5) {
        tc_fence_after();
        tmem_dealloc(tmem, 256);
    }
}

// ------------------------------------------------------------------------------------------------ single tokens
#define LD_THREADS 160          // warps 0-3: products and softmax, warp 4: TMA producer
#define LD_SLD 72               // row of the score tile (floats): fragment reads meet no bank conflicts
#define LD_EARLY 2              // pages of older positions requested before the programmatic wait

// byte offset of (row, 16-byte piece) in a [64 rows][HD] tile stored as HD / 64 swizzled boxes of [64][128 bytes]
__device__ __forceinline__ uint32_t ld_off(int row, int piece) {
    return (uint32_t)((piece >> 3) * 8192 + row * 128 + (((piece & 7) ^ (row & 7)) << 4));
}

template <int HD, int MT, int STAGES>
struct LdSmem {
    static constexpr int TILE_BYTES = 64 * HD * 2, QLD = HD + 8;
    static constexpr int Q_OFF = STAGES * TILE_BYTES, S_OFF = Q_OFF + MT * 16 * QLD * 2;
    static constexpr int BAR_OFF = S_OFF + 2 * MT * 16 * LD_SLD * 4;
    static constexpr int TOTAL = BAR_OFF + 2 * STAGES * 8 + 16 + 1024;
    static_assert(TOTAL <= 227 * 1024, "shared memory of a CTA");
};

// grid (splits, head tiles of 16 MT, sequences)
template <int HD, int MT, int STAGES>
__global__ void __launch_bounds__(LD_THREADS, 2 * LdSmem<HD, MT, STAGES>::TOTAL <= 226 * 1024 ? 2 : 1)
        k_latent_decode(const __grid_constant__ CUtensorMap map, const bf16* KB_STEP_DATA q, int ldq, bf16* __restrict__ out,
        int ldo, int dv, float* __restrict__ part_o, float* __restrict__ part_ml, const int* __restrict__ slot,
        const int* __restrict__ q_start, const int* __restrict__ kv_len, int nh, float scale_log2e,
        const int* __restrict__ table, int table_stride, int n_pages, int* status) {
    using L = LdSmem<HD, MT, STAGES>;
    constexpr int TPW = HD / 64;                     // 16-column tiles of the values a warp may have
    extern __shared__ __align__(128) uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const uint32_t sbase = smem_u32(smem);
    const uint32_t b_full = sbase + L::BAR_OFF, b_empty = b_full + STAGES * 8;
    bf16* qs = (bf16*)(smem + L::Q_OFF);
    float* ss = (float*)(smem + L::S_OFF);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int b = blockIdx.z, h0 = blockIdx.y * 16 * MT;
    kb_pdl_launch_now();
    const int qs0 = q_start[b], kvl = kv_len[b];
    const int last = (kvl - 1) / KB_PAGE, total = last + 1;
    const int per = (total + (int)gridDim.x - 1) / (int)gridDim.x;
    const int it_lo = (int)blockIdx.x * per, n_iter = min(total, it_lo + per) - it_lo;      // (may be <= 0: an empty split)
    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; s++) {
            mbar_init(b_full + s * 8, 1);
            mbar_init(b_empty + s * 8, 4);
        }
        mbar_fence_init();
    }
    __syncthreads();
    if (warp == 4) {
        // ---------------------------------------------------------------- producer
        if (lane == 0 && n_iter > 0) {
            tma_prefetch_desc(&map);
            const int* trow = table + (size_t)slot[b] * table_stride;
            bool waited = false;
            for (int i = 0; i < n_iter; i++) {
                const int s = i % STAGES;
                // (older pages were stored by earlier steps; the newest position's comes from the kernel before)
                if (!waited && (i >= LD_EARLY || it_lo + i == last)) {
                    kb_pdl_wait();
                    waited = true;
                }
                if (!mbar_wait(b_empty + s * 8, ((uint32_t)(i / STAGES) & 1u) ^ 1u, status)) break;
                int page = trow[it_lo + i];
                if (page < 0 || page >= n_pages) {
                    if (!waited) kb_pdl_wait();              // the status word is shared with earlier kernels
                    waited = true;
                    atomicOr(status, KB_ST_BAD_PAGE);
                    page = 0;
                }
                mbar_expect_tx(b_full + s * 8, L::TILE_BYTES);
#pragma unroll
                for (int h = 0; h < HD / 64; h++)
                    tma_load_2d(sbase + s * L::TILE_BYTES + h * 8192, &map, h * 64, page * KB_PAGE, b_full + s * 8);
            }
        }
        return;
    }
    // -------------------------------------------------------------------- products and softmax
    kb_pdl_wait();
    {
        constexpr int QV = MT * 16 * (HD / 8), QN = QV / 128 < 6 ? QV / 128 : 6;         // (loads in flight a thread)
#pragma unroll 1
        for (int e0 = 0; e0 < QV; e0 += 128 * QN) {
            uint4 v[QN];
#pragma unroll
            for (int i = 0; i < QN; i++) {
                const int e = e0 + threadIdx.x + i * 128, r = e / (HD / 8), c = e % (HD / 8);
                v[i] = make_uint4(0, 0, 0, 0);
                if (e < QV && h0 + r < nh) v[i] = *(const uint4*)(q + (size_t)qs0 * ldq + (size_t)(h0 + r) * HD + c * 8);
            }
#pragma unroll
            for (int i = 0; i < QN; i++) {
                const int e = e0 + threadIdx.x + i * 128, r = e / (HD / 8), c = e % (HD / 8);
                if (e < QV) *(uint4*)(qs + r * L::QLD + c * 8) = v[i];
            }
        }
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    float o[MT][TPW][2][4];
    float m_a[MT], m_b[MT], l_a[MT], l_b[MT];
#pragma unroll
    for (int m = 0; m < MT; m++) {
        m_a[m] = m_b[m] = -INFINITY;
        l_a[m] = l_b[m] = 0.0f;
#pragma unroll
        for (int t = 0; t < TPW; t++)
#pragma unroll
            for (int u = 0; u < 2; u++)
#pragma unroll
                for (int c = 0; c < 4; c++) o[m][t][u][c] = 0.0f;
    }
    const int kw0 = warp * 16;                       // this warp's positions of a page
    for (int i = 0; i < n_iter; i++) {
        const int s = i % STAGES;
        const bool ok = mbar_wait(b_full + s * 8, (uint32_t)(i / STAGES) & 1u, status);
        const uint32_t kt = sbase + s * L::TILE_BYTES;
        float* sb = ss + (i & 1) * MT * 16 * LD_SLD;
        if (ok) {
            float sc[MT][2][4];
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int u = 0; u < 2; u++)
#pragma unroll
                    for (int c = 0; c < 4; c++) sc[m][u][c] = 0.0f;
#pragma unroll 4
            for (int k = 0; k < HD / 16; k++) {
                uint32_t kf[4];
                ldsm_x4(kt + ld_off(kw0 + (lane & 7) + (lane >> 4) * 8, k * 2 + ((lane >> 3) & 1)), kf[0], kf[1], kf[2], kf[3]);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    uint32_t qf[4];
                    ldsm_x4(smem_u32(qs + (m * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * L::QLD + k * 16 + (lane >> 4) * 8), qf[0],
                            qf[1], qf[2], qf[3]);
                    mma_bf16(sc[m][0], qf, kf[0], kf[1]);
                    mma_bf16(sc[m][1], qf, kf[2], kf[3]);
                }
            }
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int u = 0; u < 2; u++) {
                    float* p = sb + (m * 16 + (lane >> 2)) * LD_SLD + kw0 + u * 8 + (lane & 3) * 2;
                    *(float2*)p = make_float2(sc[m][u][0], sc[m][u][1]);
                    *(float2*)(p + 8 * LD_SLD) = make_float2(sc[m][u][2], sc[m][u][3]);
                }
        }
        // the four warps go on together or not at all. One barrier a page is enough: the scores have two buffers
        uint32_t any_bad;
        asm volatile("{\n .reg .pred p, q;\n setp.ne.u32 p, %1, 0;\n bar.red.or.pred q, 1, 128, p;\n selp.u32 %0, 1, 0, q;\n}"
                     : "=r"(any_bad) : "r"(ok ? 0u : 1u) : "memory");
        if (any_bad) break;
        const int key0 = (it_lo + i) * KB_PAGE;
        const bool whole = key0 + KB_PAGE <= kvl;
        uint32_t pf[MT][4][4];
#pragma unroll
        for (int m = 0; m < MT; m++) {
            float v[4][8];                           // [16 positions][rows a, b of fragment words 0..3]
            float xa = -INFINITY, xb = -INFINITY;
#pragma unroll
            for (int k = 0; k < 4; k++)
#pragma unroll
                for (int w = 0; w < 4; w++) {
                    const int c = k * 16 + (w >> 1) * 8 + (lane & 3) * 2;
                    const float2 x = *(const float2*)(sb + (m * 16 + (lane >> 2) + (w & 1) * 8) * LD_SLD + c);
                    const float x0 = whole || key0 + c < kvl ? x.x * scale_log2e : -INFINITY;
                    const float x1 = whole || key0 + c + 1 < kvl ? x.y * scale_log2e : -INFINITY;
                    v[k][2 * w] = x0;
                    v[k][2 * w + 1] = x1;
                    if (w & 1) xb = fmaxf(xb, fmaxf(x0, x1));
                    else xa = fmaxf(xa, fmaxf(x0, x1));
                }
            xa = fmaxf(xa, __shfl_xor_sync(0xffffffffu, xa, 1));
            xa = fmaxf(xa, __shfl_xor_sync(0xffffffffu, xa, 2));
            xb = fmaxf(xb, __shfl_xor_sync(0xffffffffu, xb, 1));
            xb = fmaxf(xb, __shfl_xor_sync(0xffffffffu, xb, 2));
            const float na = fmaxf(m_a[m], xa), nb = fmaxf(m_b[m], xb);       // (a page has at least one visible position)
            const float fa = exp2f(m_a[m] - na), fb = exp2f(m_b[m] - nb);
            m_a[m] = na;
            m_b[m] = nb;
            float sa = 0.0f, sm_b = 0.0f;
#pragma unroll
            for (int k = 0; k < 4; k++)
#pragma unroll
                for (int w = 0; w < 4; w++) {
                    const float u = w & 1 ? nb : na;
                    const float p0 = exp2f(v[k][2 * w] - u), p1 = exp2f(v[k][2 * w + 1] - u);
                    if (w & 1) sm_b += p0 + p1;
                    else sa += p0 + p1;
                    pf[m][k][w] = pack_bf16(p0, p1);
                }
            l_a[m] = l_a[m] * fa + sa;
            l_b[m] = l_b[m] * fb + sm_b;
            if (__any_sync(0xffffffffu, fa != 1.0f || fb != 1.0f)) {
#pragma unroll
                for (int t = 0; t < TPW; t++)
#pragma unroll
                    for (int u = 0; u < 2; u++) {
                        o[m][t][u][0] *= fa;
                        o[m][t][u][1] *= fa;
                        o[m][t][u][2] *= fb;
                        o[m][t][u][3] *= fb;
                    }
            }
        }
#pragma unroll
        for (int t = 0; t < TPW; t++) {
            const int c16 = warp + 4 * t;
            if (c16 * 16 < dv) {
#pragma unroll
                for (int k = 0; k < 4; k++) {
                    uint32_t vf[4];
                    ldsm_x4_t(kt + ld_off(k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, c16 * 2 + (lane >> 4)), vf[0], vf[1], vf[2],
                              vf[3]);
#pragma unroll
                    for (int m = 0; m < MT; m++) {
                        mma_bf16(o[m][t][0], pf[m][k], vf[0], vf[1]);
                        mma_bf16(o[m][t][1], pf[m][k], vf[2], vf[3]);
                    }
                }
            }
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(b_empty + s * 8);
    }
    const int n_splits = gridDim.x, split = blockIdx.x;
#pragma unroll
    for (int m = 0; m < MT; m++) {
        l_a[m] += __shfl_xor_sync(0xffffffffu, l_a[m], 1);
        l_a[m] += __shfl_xor_sync(0xffffffffu, l_a[m], 2);
        l_b[m] += __shfl_xor_sync(0xffffffffu, l_b[m], 1);
        l_b[m] += __shfl_xor_sync(0xffffffffu, l_b[m], 2);
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int h = h0 + m * 16 + (lane >> 2) + half * 8;
            if (h >= nh) continue;
            const float l = half ? l_b[m] : l_a[m];
            const float inv = n_splits > 1 ? 1.0f : l > 0.0f ? 1.0f / l : 0.0f;
            const size_t pi = ((size_t)b * nh + h) * n_splits + split;
#pragma unroll
            for (int t = 0; t < TPW; t++)
#pragma unroll
                for (int u = 0; u < 2; u++)
#pragma unroll
                    for (int e = 0; e < 2; e++) {
                        const int c = (warp + 4 * t) * 16 + u * 8 + (lane & 3) * 2 + e;
                        if (c >= dv) continue;
                        const float v = o[m][t][u][half * 2 + e] * inv;
                        if (n_splits > 1) part_o[pi * dv + c] = v;
                        else out[(size_t)qs0 * ldo + (size_t)h * dv + c] = __float2bfloat16_rn(v);
                    }
            if (n_splits > 1 && warp == 0 && (lane & 3) == 0) {
                part_ml[pi * 2] = half ? m_b[m] : m_a[m];
                part_ml[pi * 2 + 1] = l;
            }
        }
    }
}

// out = sum_s 2^(m_s - M) o_s / sum_s 2^(m_s - M) l_s, in split order. grid (heads, sequences, value columns / 128)
__global__ void __launch_bounds__(128) k_latent_merge(const float* KB_STEP_DATA part_o, const float* KB_STEP_DATA part_ml,
        int n_splits, int dv, bf16* __restrict__ out, int ldo, const int* __restrict__ q_start, int nh) {
    __shared__ float sf[64];
    __shared__ float s_l;
    kb_pdl_launch();
    const int h = blockIdx.x, b = blockIdx.y, c = blockIdx.z * 128 + threadIdx.x;
    const size_t base = ((size_t)b * nh + h) * n_splits;
    kb_pdl_wait();
    float v[16];
#pragma unroll
    for (int j = 0; j < 16; j++) v[j] = (c < dv && j < n_splits) ? part_o[(base + j) * dv + c] : 0.0f;
    if (threadIdx.x < 32) {
        const int i0 = threadIdx.x, i1 = threadIdx.x + 32;
        const float m0 = i0 < n_splits ? part_ml[(base + i0) * 2] : -INFINITY;
        const float m1 = i1 < n_splits ? part_ml[(base + i1) * 2] : -INFINITY;
        const float M = kb_warp_max(fmaxf(m0, m1));
        const float U = M == -INFINITY ? 0.0f : M;
        const float f0 = exp2f(m0 - U), f1 = exp2f(m1 - U);
        sf[i0] = f0;
        sf[i1] = f1;
        const float l = kb_warp_sum((i0 < n_splits ? f0 * part_ml[(base + i0) * 2 + 1] : 0.0f) +
                                    (i1 < n_splits ? f1 * part_ml[(base + i1) * 2 + 1] : 0.0f));
        if (threadIdx.x == 0) s_l = l > 0.0f ? 1.0f / l : 0.0f;
    }
    __syncthreads();
    if (c >= dv) return;
    float o = 0.0f;
#pragma unroll
    for (int j = 0; j < 16; j++)
        if (j < n_splits) o = fmaf(sf[j], v[j], o);
    for (int j = 16; j < n_splits; j++) o = fmaf(sf[j], part_o[(base + j) * dv + c], o);
    out[(size_t)q_start[b] * ldo + (size_t)h * dv + c] = __float2bfloat16_rn(o * s_l);
}

// ------------------------------------------------------------------------------------------------ entry points
template <int HD, int KEYS, int STAGES>
static int launch_latent_tc(const CUtensorMap& map, const void* q, int ldq, void* out, int ldo, int dv, const int* slot,
                            const int* q_start, const int* kv_len, int B, int nh, int G, float scale, const int* table,
                            int table_stride, int n_pages, int grid_x, int* status, cudaStream_t st) {
    using L = LtSmem<HD, KEYS, STAGES>;
    auto kern = k_latent_tc<HD, KEYS, STAGES>;
    static char once_tag;
    if (kb_first_use(&once_tag)) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             L::TOTAL > 118 * 1024 ? L::TOTAL : 118 * 1024);
        if (e != cudaSuccess) return (int)e;
    }
    const int dv_part = dv > 256 ? 256 : (dv + 15) / 16 * 16, parts = (dv + dv_part - 1) / dv_part;
    const uint32_t cols = 2 * KEYS + (dv_part + 31) / 32 * 32 <= 256 ? 256 : 512;
    // (a CTA that holds all of an SM's tensor memory has the SM to itself)
    constexpr int ALONE = 118 * 1024;
    const int sm = cols == 512 && L::TOTAL < ALONE ? ALONE : L::TOTAL;
    dim3 grid(nh / G * parts, grid_x, B);
    cudaError_t e = kb_launch(kern, grid, LT_THREADS, sm, st, map, (const bf16*)q, ldq, (bf16*)out, ldo, dv, dv_part, parts,
                              slot, q_start, kv_len, G, scale * 1.4426950408889634f, table, table_stride, n_pages, cols, status);
    return (int)e;
}

// pool: pages [n_pages][64][hd] of the cached vectors; q rows [nh][hd], out rows [nh][dv] (dv <= hd). G: heads a CTA takes
// together (nh % G == 0, at most 128); grid_x = ceil(longest q_len / (128 / G))
extern "C" int kb_latent_tc(const void* q, int ldq, void* out, int ldo, int dv, const int* slot, const int* q_start,
                            const int* kv_len, int B, int nh, int G, int hd, float scale, void* pool, const int* table,
                            int table_stride, int n_pages, int grid_x, int* status, cudaStream_t st) {
    if (B <= 0 || grid_x <= 0) return 0;
    if (G < 1 || G > 128 || nh % G || dv < 1 || dv > hd || grid_x > 65535 || B > 65535 || ldq % 8 || ldo % 8 ||
        ((uintptr_t)q & 15) || ((uintptr_t)out & 15) || !(scale > 0.0f))
        return (int)cudaErrorInvalidValue;
    CUtensorMap map;
    int rc = kb_make_map_bf16(&map, pool, (uint64_t)n_pages * KB_PAGE, hd, hd, hd > 256 ? 32 : 64);
    if (rc) return rc;
#define LT_GO(HD, KEYS, ST)                                                                                            \
    return launch_latent_tc<HD, KEYS, ST>(map, q, ldq, out, ldo, dv, slot, q_start, kv_len, B, nh, G, scale, table,     \
                                          table_stride, n_pages, grid_x, status, st)
    switch (hd) {
        case 64: LT_GO(64, 64, 4);
        case 128: LT_GO(128, 64, 4);
        case 192: LT_GO(192, 64, 2);
        case 256: LT_GO(256, 64, 3);
        case 320: LT_GO(320, 32, 4);
        case 576: LT_GO(576, 32, 2);
        default: return (int)cudaErrorInvalidValue;
    }
#undef LT_GO
}

extern "C" int kb_latent_gather(const void* pool, int hd, int kr, int rot, const int* slot, const int* kv_len, int B,
                                const int* table, int table_stride, int n_pages, void* lat, void* rotk, int N, int* status,
                                cudaStream_t st) {
    if (N <= 0) return 0;
    if (hd % 8 || kr % 8 || rot % 8 || kr + rot > hd || B < 1) return (int)cudaErrorInvalidValue;
    kb_launch(k_latent_gather, (N + 7) / 8, 256, 0, st, (const bf16*)pool, hd, kr, rot, slot, kv_len, B, table, table_stride,
              n_pages, (bf16*)lat, (bf16*)rotk, N, status);
    KB_LAUNCH_RET();
}

template <int KBX, int VBX>
static int launch_latent_full(const CUtensorMap& kv, const CUtensorMap& rot, const LfArgs& a, int grid_x, int B, cudaStream_t st) {
    using L = LfSmem<KBX, VBX>;
    static char once_tag;
    if (kb_first_use(&once_tag)) {
        cudaError_t e = cudaFuncSetAttribute(k_latent_full<KBX, VBX>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
        if (e != cudaSuccess) return (int)e;
    }
    return (int)kb_launch(k_latent_full<KBX, VBX>, dim3(a.n_heads, grid_x, B), LT_THREADS, L::TOTAL, st, kv, rot, a);
}

// q rows of nh heads [d | rot]; kv rows [N][nh d keys | nh dv values] and rotk rows [N][rot] of the step's sequences one after
// another (kv_len[b] rows each); angles [T][rot / 2] (cosine, sine); gate: rows of one number a head, or null. d, rot, dv
// multiples of 8 (half pairing: rot of 16), d and dv at most 128, rot at most 64; grid_x = ceil(longest q_len / 128)
extern "C" int kb_latent_full(const void* q, int ldq, int d, int rot, int dv, int nh, const void* kv, int ldkv, const void* rotk,
                              int N, const float* angles, float mult, int half, const void* gate, int ldg, void* out, int ldo,
                              const int* q_start, const int* kv_len, int B, float scale, int grid_x, int* status,
                              cudaStream_t st) {
    if (B <= 0 || grid_x <= 0) return 0;
    if (d < 8 || d % 8 || d > 128 || dv < 8 || dv % 8 || dv > 128 || rot < 8 || rot % 8 || rot > 64 || (half && rot % 16) ||
        ldq % 8 || ldkv % 8 || ldo % 8 || (((uintptr_t)q | (uintptr_t)out) & 15) || N < 1 || grid_x > 65535 || B > 65535 ||
        !(scale > 0.0f) || ((uintptr_t)angles & 7))
        return (int)cudaErrorInvalidValue;
    CUtensorMap kvm, rm;
    int rc = kb_make_map_bf16(&kvm, kv, N, (uint64_t)nh * (d + dv), ldkv, 64);
    if (!rc) rc = kb_make_map_bf16(&rm, rotk, N, rot, rot, 64);
    if (rc) return rc;
    LfArgs a;
    a.q = (const bf16*)q; a.ldq = ldq; a.d = d; a.rot = rot; a.dv = dv; a.n_heads = nh;
    a.angles = (const float2*)angles; a.mult = mult; a.half = half; a.gate = (const bf16*)gate; a.ldg = ldg;
    a.out = (bf16*)out; a.ldo = ldo; a.q_start = q_start; a.kv_len = kv_len; a.scale_log2e = scale * 1.4426950408889634f;
    a.status = status;
    if (d <= 64) return dv <= 64 ? launch_latent_full<1, 1>(kvm, rm, a, grid_x, B, st) : launch_latent_full<1, 2>(kvm, rm, a, grid_x, B, st);
    return dv <= 64 ? launch_latent_full<2, 1>(kvm, rm, a, grid_x, B, st) : launch_latent_full<2, 2>(kvm, rm, a, grid_x, B, st);
}

template <int HD, int MT, int STAGES>
static int launch_latent_decode(const CUtensorMap& map, const void* q, int ldq, void* out, int ldo, int dv, float* part_o,
                                float* part_ml, const int* slot, const int* q_start, const int* kv_len, int B, int nh,
                                float scale, const int* table, int table_stride, int n_pages, int splits, int* status,
                                cudaStream_t st) {
    using L = LdSmem<HD, MT, STAGES>;
    auto kern = k_latent_decode<HD, MT, STAGES>;
    static char once_tag;
    if (kb_first_use(&once_tag)) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
        if (e != cudaSuccess) return (int)e;
    }
    dim3 grid(splits, (nh + 16 * MT - 1) / (16 * MT), B);
    cudaError_t e = kb_launch(kern, grid, LD_THREADS, L::TOTAL, st, map, (const bf16*)q, ldq, (bf16*)out, ldo, dv, part_o, part_ml,
                              slot, q_start, kv_len, nh, scale * 1.4426950408889634f, table, table_stride, n_pages, status);
    return (int)e;
}

// one row per sequence; splits > 1: part_o [B][nh][splits][dv] and part_ml [B][nh][splits][2] are scratch
extern "C" int kb_latent_decode(const void* q, int ldq, void* out, int ldo, int dv, float* part_o, float* part_ml,
                                const int* slot, const int* q_start, const int* kv_len, int B, int nh, int hd, float scale,
                                void* pool, const int* table, int table_stride, int n_pages, int splits, int* status,
                                cudaStream_t st) {
    if (B <= 0) return 0;
    if (splits < 1 || splits > 64 || nh < 1 || dv < 1 || dv > hd || B > 65535 || ldq % 8 || ((uintptr_t)q & 15) ||
        (splits > 1 && (!part_o || !part_ml)))
        return (int)cudaErrorInvalidValue;
    CUtensorMap map;
    int rc = kb_make_map_bf16(&map, pool, (uint64_t)n_pages * KB_PAGE, hd, hd, 64);
    if (rc) return rc;
    const bool two = nh > 16;
#define LD_GO(HD, S1, S2)                                                                                              \
    rc = two ? launch_latent_decode<HD, 2, S2>(map, q, ldq, out, ldo, dv, part_o, part_ml, slot, q_start, kv_len, B, nh, \
                                               scale, table, table_stride, n_pages, splits, status, st)                \
             : launch_latent_decode<HD, 1, S1>(map, q, ldq, out, ldo, dv, part_o, part_ml, slot, q_start, kv_len, B, nh, \
                                               scale, table, table_stride, n_pages, splits, status, st)
    switch (hd) {
        case 64: LD_GO(64, 6, 6); break;
        case 128: LD_GO(128, 5, 4); break;
        case 192: LD_GO(192, 3, 3); break;
        case 256: LD_GO(256, 2, 2); break;
        case 320: LD_GO(320, 4, 3); break;
        case 576: LD_GO(576, 2, 2); break;
        default: return (int)cudaErrorInvalidValue;
    }
#undef LD_GO
    if (rc || splits == 1) return rc;
    kb_launch(k_latent_merge, dim3(nh, B, (dv + 127) / 128), 128, 0, st, (const float*)part_o, (const float*)part_ml, splits, dv,
              (bf16*)out, ldo, q_start, nh);
    KB_LAUNCH_RET();
}
