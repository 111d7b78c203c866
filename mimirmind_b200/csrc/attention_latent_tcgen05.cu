// Latent attention of prompt portions on the tcgen05 tensor cores, with keys and values made in full.
//
// For a single token the up-projections are absorbed into the query and the output (attention_latent_mma.cu): the latent rows
// are read once for all heads.  A portion of a prompt meets every cached row with many tokens, so it pays to make each head's
// plain keys and values once per step (a plain matrix product over the cached latents, 64 tokens and more) and to run
//
//   s_j = (q_plain . k_plain_j + q_turned . k_turned_j) scale,  o = sum_j softmax(s)_j v_j      (dk + dr + dv products a pair
//
// instead of 2 rank + dr).  The turned key part is shared by the heads and is read as it is cached.  A sink (one number per
// head) adds exp(sink_h) to the softmax's denominator.
//
// One CTA per (tile of up to 128 query tokens of one request, head), 128 keys per tile, as attention_tcgen05.cu: two softmax
// groups take the even and the odd key tiles with a maximum, a sum and an O accumulator of their own; S and O in tensor memory,
// P through shared memory.  What differs: keys and values are rows of plain matrices, so one thread fetches them with one copy a
// piece; a key tile is a sequence of 64-wide pieces (the plain part's, then the turned part's) that go through a ring piece by
// piece, and a value tile is two pieces of 64 keys, so that 192-wide keys and 128-wide values fit beside Q and two tiles of P.
// Columns that a piece holds beyond its head's size belong to the next head (or are zero): Q is zero there, and the
// output columns made from them are not written.
// All mbarrier waits are bounded; on a time-out the kernel frees its tensor memory, sets `err` and returns.
#include "tcgen05_attention.cuh"

namespace {

using namespace tc;

constexpr int BM = 128, BN = 128;
constexpr int PIECE_BYTES = 128 * 64 * 2;       // [128 rows x 64 columns] bf16: a piece of Q or of a key tile, half a tile of P
constexpr int VPIECE_BYTES = 64 * 64 * 2;       // [64 keys x 64 columns]: a value piece is VH of these
constexpr int P_BYTES = 2 * PIECE_BYTES;
constexpr int LT_THREADS = 384;                 // K producer warp, Q K^T issuer, 8 softmax warps, V producer warp, P V issuer
constexpr int V_PRODUCER_WARP = 10, PV_ISSUER_WARP = 11, SOFTMAX_WARPS = 8, GROUP_WARPS = 4;
constexpr int MAX_KSTAGES = 6, MAX_VSTAGES = 4;
constexpr int SMEM_MAX = 232448;
constexpr int LT_TMEM_COLS = 512;               // S of the even / odd tiles: columns 0..255; O of the even / odd tiles from 256

struct LtCtl {
    uint64_t q_full;
    uint64_t k_full[MAX_KSTAGES], k_empty[MAX_KSTAGES];
    uint64_t v_full[MAX_VSTAGES], v_empty[MAX_VSTAGES];
    uint64_t s_full[2], s_free[2], p_full[2], pv_done[2];
    uint64_t l_full;
    uint32_t tmem_base;
    int abort_flag;
    float xchg[2][2][128];   // [group][maximum, sum][row]
};

// tiles: int32 [n_tiles, 4] = (first token row, rows in the tile (<= 128), position of the first row, row of the request's key 0)
template <int VH>
__global__ void __launch_bounds__(LT_THREADS, 1)
attention_latent_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmR,
                           const __grid_constant__ CUtensorMap tmV, __nv_bfloat16* __restrict__ out, const int32_t* __restrict__ tiles, int H,
                           int dk, int dv, int plain_pieces, int pieces, int k_stages, int v_stages, float scale_log2,
                           const float* __restrict__ sink, int* __restrict__ err) {
    extern __shared__ __align__(1024) unsigned char smem_raw[];   // 128-byte swizzle wants 1024-byte aligned tiles
    if ((smem_u32(smem_raw) & 1023u) != 0) {
        if (threadIdx.x == 0 && err != nullptr) atomicExch(err, 3);
        return;
    }
    constexpr int DVP = 64 * VH, VSTAGE_BYTES = VH * VPIECE_BYTES;
    unsigned char* sQ = smem_raw;                                // pieces * PIECE_BYTES
    unsigned char* sP = sQ + pieces * PIECE_BYTES;               // 2 * P_BYTES
    unsigned char* sK = sP + 2 * P_BYTES;                        // k_stages * PIECE_BYTES
    unsigned char* sV = sK + k_stages * PIECE_BYTES;             // v_stages * VSTAGE_BYTES
    LtCtl* ctl = reinterpret_cast<LtCtl*>(sV + v_stages * VSTAGE_BYTES);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    volatile int* abort_flag = &ctl->abort_flag;

    // heads fastest, later (longer) tiles first
    const int tile = gridDim.y - 1 - blockIdx.y, h = blockIdx.x;
    const int row0 = tiles[tile * 4 + 0], n_rows = tiles[tile * 4 + 1], pos0 = tiles[tile * 4 + 2], key_row0 = tiles[tile * 4 + 3];
    const int n_tiles_k = (pos0 + n_rows + BN - 1) / BN;

    if (threadIdx.x == 64) {
        prefetch_tensormap(&tmQ);
        prefetch_tensormap(&tmK);
        prefetch_tensormap(&tmR);
        prefetch_tensormap(&tmV);
    }
    if (threadIdx.x == 0) {
        mbar_init(smem_u32(&ctl->q_full), 1);
        for (int s = 0; s < k_stages; ++s) {
            mbar_init(smem_u32(&ctl->k_full[s]), 1);
            mbar_init(smem_u32(&ctl->k_empty[s]), 1);
        }
        for (int s = 0; s < v_stages; ++s) {
            mbar_init(smem_u32(&ctl->v_full[s]), 1);
            mbar_init(smem_u32(&ctl->v_empty[s]), 1);
        }
        for (int b = 0; b < 2; ++b) {
            mbar_init(smem_u32(&ctl->s_full[b]), 1);
            mbar_init(smem_u32(&ctl->s_free[b]), GROUP_WARPS);
            mbar_init(smem_u32(&ctl->p_full[b]), GROUP_WARPS);
            mbar_init(smem_u32(&ctl->pv_done[b]), 1);
        }
        mbar_init(smem_u32(&ctl->l_full), SOFTMAX_WARPS);
        ctl->abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        // Q needs nobody else: its copies go out before the CTA has set itself up
        const uint32_t qbar = smem_u32(&ctl->q_full);
        mbar_expect_tx(qbar, (uint32_t)pieces * PIECE_BYTES);
        for (int p = 0; p < pieces; ++p) tma_load_2d(smem_u32(sQ) + p * PIECE_BYTES, &tmQ, (h * pieces + p) * 64, row0, qbar);
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&ctl->tmem_base)), "r"(LT_TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = ctl->tmem_base;

    if (warp == 0) {
        if (lane == 0) {
            // ---- keys: piece by piece ----
            bool ok = true;
            int s = 0;
            uint32_t round = 0;
            for (int t = 0; t < n_tiles_k && ok; ++t) {
                for (int p = 0; p < pieces; ++p) {
                    if (!mbar_wait(smem_u32(&ctl->k_empty[s]), (round & 1) ^ 1, abort_flag)) { ok = false; break; }
                    const uint32_t full = smem_u32(&ctl->k_full[s]), dst = smem_u32(sK + s * PIECE_BYTES);
                    mbar_expect_tx(full, PIECE_BYTES);
                    if (p < plain_pieces) tma_load_2d(dst, &tmK, h * dk + p * 64, key_row0 + t * BN, full);
                    else tma_load_2d(dst, &tmR, (p - plain_pieces) * 64, key_row0 + t * BN, full);
                    if (++s == k_stages) { s = 0; ++round; }
                }
            }
        }
    } else if (warp == V_PRODUCER_WARP) {
        if (lane == 0) {
            // ---- values: 64 keys at a time ----
            bool ok = true;
            int s = 0;
            uint32_t round = 0;
            for (int t = 0; t < 2 * n_tiles_k && ok; ++t) {
                if (!mbar_wait(smem_u32(&ctl->v_empty[s]), (round & 1) ^ 1, abort_flag)) { ok = false; break; }
                const uint32_t full = smem_u32(&ctl->v_full[s]), dst = smem_u32(sV + s * VSTAGE_BYTES);
                mbar_expect_tx(full, VSTAGE_BYTES);
#pragma unroll
                for (int c = 0; c < VH; ++c) tma_load_2d(dst + c * VPIECE_BYTES, &tmV, h * dv + c * 64, key_row0 + t * 64, full);
                if (++s == v_stages) { s = 0; ++round; }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            // ---- Q K^T issuer ----
            constexpr uint32_t IDESC_QK = idesc_bf16(BM, BN, false);
            const uint32_t q_addr = smem_u32(sQ);
            bool ok = mbar_wait(smem_u32(&ctl->q_full), 0, abort_flag);
            int s = 0;
            uint32_t round = 0;
            for (int t = 0; t < n_tiles_k && ok; ++t) {
                const uint32_t b = t & 1, u = (uint32_t)t >> 1;
                if (!mbar_wait(smem_u32(&ctl->s_free[b]), (u & 1) ^ 1, abort_flag)) { ok = false; break; }
                for (int p = 0; p < pieces; ++p) {
                    if (!mbar_wait(smem_u32(&ctl->k_full[s]), round & 1, abort_flag)) { ok = false; break; }
                    tc_fence_after();
                    const uint32_t k_addr = smem_u32(sK + s * PIECE_BYTES), a_addr = q_addr + p * PIECE_BYTES;
#pragma unroll
                    for (int k = 0; k < 4; ++k)                    // 16 columns = 32 bytes inside the swizzled row
                        umma_bf16(tmem_base + b * 128, smem_desc_sw128(a_addr + k * 32, 16, 1024), smem_desc_sw128(k_addr + k * 32, 16, 1024), IDESC_QK,
                                  (p | k) ? 1u : 0u);
                    umma_commit(smem_u32(&ctl->k_empty[s]));
                    if (++s == k_stages) { s = 0; ++round; }
                }
                if (ok) umma_commit(smem_u32(&ctl->s_full[b]));
            }
        }
    } else if (warp == PV_ISSUER_WARP) {
        if (lane == 0) {
            // ---- P V issuer ----
            constexpr uint32_t IDESC_PV = idesc_bf16(BM, DVP, true);
            bool ok = true;
            int s = 0;
            uint32_t round = 0;
            for (int t = 0; t < n_tiles_k && ok; ++t) {
                const uint32_t b = t & 1, u = (uint32_t)t >> 1;
                if (!mbar_wait(smem_u32(&ctl->p_full[b]), u & 1, abort_flag)) { ok = false; break; }       // P is there, O is rescaled
                for (int hf = 0; hf < 2; ++hf) {
                    if (!mbar_wait(smem_u32(&ctl->v_full[s]), round & 1, abort_flag)) { ok = false; break; }
                    tc_fence_after();
                    const uint32_t p_addr = smem_u32(sP + b * P_BYTES + hf * PIECE_BYTES), v_addr = smem_u32(sV + s * VSTAGE_BYTES);
#pragma unroll
                    for (int k = 0; k < 4; ++k)                    // P: K-major over the keys; V: 16 key rows of 128 bytes further
                        umma_bf16(tmem_base + 256 + b * DVP, smem_desc_sw128(p_addr + k * 32, 16, 1024), smem_desc_sw128(v_addr + k * 16 * 128, VPIECE_BYTES, 1024),
                                  IDESC_PV, (u | (uint32_t)hf | (uint32_t)k) ? 1u : 0u);
                    umma_commit(smem_u32(&ctl->v_empty[s]));
                    if (++s == v_stages) { s = 0; ++round; }
                }
                if (ok) umma_commit(smem_u32(&ctl->pv_done[b]));
            }
        }
    } else {
        // ---- softmax and output: group g (warps 2 + 4g .. 5 + 4g) takes the key tiles of parity g, one thread per row ----
        const int q = warp & 3;                                    // warp w may read tensor-memory lanes 32 (w % 4) .. + 31
        const uint32_t g = (uint32_t)(warp - 2) >> 2;
        const int row = q * 32 + lane, pos = pos0 + row;
        const bool row_valid = row < n_rows;
        const uint32_t lane_addr = tmem_base + ((uint32_t)(q * 32) << 16);
        const uint32_t s_addr = lane_addr + g * 128, o_addr = lane_addr + 256 + g * DVP;
        const SoftmaxBars bars = {smem_u32(&ctl->s_full[g]), smem_u32(&ctl->s_free[g]), smem_u32(&ctl->p_full[g]), smem_u32(&ctl->pv_done[g])};
        float m_ref = -INFINITY, l = 0.0f;
        bool ok = true;
        uint32_t sreg[128];
        for (uint32_t t = g; (int)t < n_tiles_k && ok; t += 2)
            ok = softmax_tile<DVP>(bars, abort_flag, s_addr, o_addr, sP + g * P_BYTES, PIECE_BYTES, row, lane, row_valid, pos, 0, (int)t * BN, t >> 1,
                                   t == g, scale_log2, sreg, m_ref, l);
        // Merge the groups (and the sink, a key without a value): out = (O0 f0 + O1 f1) / (l0 f0 + l1 f1 + fs), f = 2^(m scale - top)
        ctl->xchg[g][0][row] = m_ref;
        ctl->xchg[g][1][row] = l;
        warp_arrive(smem_u32(&ctl->l_full), lane);
        if (ok) ok = mbar_wait(smem_u32(&ctl->l_full), 0, abort_flag);
        const float m0 = ctl->xchg[0][0][row], m1 = ctl->xchg[1][0][row];
        const float l0 = ctl->xchg[0][1][row], l1 = ctl->xchg[1][1][row];
        const float ls = sink ? sink[h] * 1.4426950408889634f : -INFINITY;
        const float top = fmaxf(fmaxf(m0, m1) * scale_log2, ls);
        const float f0 = (m0 == -INFINITY) ? 0.0f : fast_exp2(m0 * scale_log2 - top);
        const float f1 = (m1 == -INFINITY) ? 0.0f : fast_exp2(m1 * scale_log2 - top);
        const float total = l0 * f0 + l1 * f1 + (sink ? fast_exp2(ls - top) : 0.0f);
        const int tiles0 = (n_tiles_k + 1) / 2, tiles1 = n_tiles_k / 2;
        if (ok && tiles0 > 0) ok = mbar_wait(smem_u32(&ctl->pv_done[0]), (uint32_t)(tiles0 - 1) & 1, abort_flag);
        if (ok && tiles1 > 0) ok = mbar_wait(smem_u32(&ctl->pv_done[1]), (uint32_t)(tiles1 - 1) & 1, abort_flag);
        tc_fence_after();
        const float inv = total > 0.0f ? 1.0f / total : 0.0f;
        __nv_bfloat16* orow = out + ((size_t)(row0 + row) * H + h) * dv;
#pragma unroll 1
        for (int c = 0; c < VH; ++c) {                             // group g writes its half of the columns, 32 at a time
            const int col0 = (int)g * (DVP / 2) + c * 32;
            float acc[32];
#pragma unroll
            for (int i = 0; i < 32; ++i) acc[i] = 0.0f;
            if (ok && tiles0 > 0) {                                // uniform over the CTA
                tmem_ld32_nowait(lane_addr + 256 + col0, sreg);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) acc[i] = __uint_as_float(sreg[i]) * f0;
            }
            if (ok && tiles1 > 0) {
                tmem_ld32_nowait(lane_addr + 256 + DVP + col0, sreg);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) acc[i] = fmaf(__uint_as_float(sreg[i]), f1, acc[i]);
            }
            if (ok && row_valid) {
#pragma unroll
                for (int i = 0; i < 32; i += 8)
                    if (col0 + i < dv)
                        *reinterpret_cast<uint4*>(orow + col0 + i) = make_uint4(pack_bf16x2(acc[i] * inv, acc[i + 1] * inv), pack_bf16x2(acc[i + 2] * inv, acc[i + 3] * inv),
                                                                                pack_bf16x2(acc[i + 4] * inv, acc[i + 5] * inv), pack_bf16x2(acc[i + 6] * inv, acc[i + 7] * inv));
            }
        }
    }

    // ---- teardown ----
    if (*abort_flag) {
        for (int i = 0; i < 2000; ++i) __nanosleep(1000);
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (threadIdx.x == 0 && ctl->abort_flag && err != nullptr) atomicExch(err, 2);
    if (warp == 1) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(LT_TMEM_COLS) : "memory");
    }
}

struct LtLayout {
    int plain_pieces, pieces, vh, k_stages, v_stages;
    size_t smem;
};

LtLayout lt_layout(int dk, int dr, int dv) {
    LtLayout a;
    a.plain_pieces = (dk + 63) / 64;
    a.pieces = a.plain_pieces + (dr + 63) / 64;
    a.vh = (dv + 63) / 64;
    a.v_stages = a.vh == 1 ? 4 : 3;
    const long long fixed = (long long)a.pieces * PIECE_BYTES + 2 * P_BYTES + (long long)a.v_stages * a.vh * VPIECE_BYTES + (long long)sizeof(LtCtl);
    const long long left = SMEM_MAX - fixed;
    a.k_stages = left < 0 ? 0 : (int)(left / PIECE_BYTES < MAX_KSTAGES ? left / PIECE_BYTES : MAX_KSTAGES);
    a.smem = (size_t)(fixed + (long long)a.k_stages * PIECE_BYTES);
    return a;
}

template <int VH>
int lt_launch(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tr, const CUtensorMap& tv, void* out, const void* tiles, int n_tiles, int H,
              int dk, int dv, const LtLayout& a, float scale, const void* sink, void* err, cudaStream_t s) {
    static bool configured = false;
    if (!configured) {
        if (cudaFuncSetAttribute(attention_latent_tc_kernel<VH>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX) != cudaSuccess) {
            cudaGetLastError();
            mm_set_last_error("latent attention: cannot reserve shared memory");
            return MM_ERR_LAUNCH;
        }
        configured = true;
    }
    attention_latent_tc_kernel<VH><<<dim3(H, n_tiles), LT_THREADS, a.smem, s>>>(tq, tk, tr, tv, (__nv_bfloat16*)out, (const int32_t*)tiles, H, dk, dv,
                                                                                a.plain_pieces, a.pieces, a.k_stages, a.v_stages, scale * 1.4426950408889634f,
                                                                                (const float*)sink, (int*)err);
    MM_CHECK_LAUNCH();
    return MM_OK;
}

}  // namespace

// Sizes the kernel takes: all multiples of 8 (16-byte copies), at most four 64-wide pieces of a key, values up to 128.
MM_EXPORT int mm_attention_latent_tcgen05_supported(int dk, int dr, int dv) {
    if (dk < 8 || dr < 0 || dv < 8 || dk % 8 || dr % 8 || dv % 8 || dv > 128 || dk > 256 || dr > 256) return 0;
    const LtLayout a = lt_layout(dk, dr, dv);
    return a.pieces <= 4 && a.k_stages >= 3;
}

// Numbers of a query row per head: every part filled up to whole pieces of 64 with zeros.
MM_EXPORT int mm_attention_latent_tcgen05_query_width(int dk, int dr) { return 64 * ((dk + 63) / 64 + (dr + 63) / 64); }

// q [n_tokens, H, query width] bf16 (plain part, zeros, turned part, zeros); kv [key_rows, H dk + H dv] bf16 (every head's plain
// key, then every head's value); turned [key_rows, dr] bf16 (null with dr = 0); out [n_tokens, H dv] bf16: the tiles' rows are
// written.  tiles int32 [n_tiles, 4] = (first token row, rows <= 128, position of the first row, row of the request's key 0), its
// keys in consecutive rows.  sink fp32 [H] or null.  `err`: device int set to 2 when a bounded wait ran out (may be null).
MM_EXPORT int mm_attention_latent_tcgen05(const void* q, const void* kv, const void* turned, void* out, const void* tiles, int n_tiles, int n_tokens,
                                          int key_rows, int H, int dk, int dr, int dv, float scale, const void* sink, void* err, void* stream) {
    MM_REQUIRE(mm_attention_latent_tcgen05_supported(dk, dr, dv), "latent attention (tcgen05): sizes that are multiples of 8, keys of at most four pieces of 64, values up to 128");
    MM_REQUIRE(n_tiles >= 0 && n_tiles <= 65535 && n_tokens > 0 && key_rows > 0 && H > 0 && scale > 0.0f, "latent attention (tcgen05): bad sizes or scale");
    MM_REQUIRE(((uintptr_t)q & 15) == 0 && ((uintptr_t)kv & 15) == 0 && ((uintptr_t)turned & 15) == 0 && ((uintptr_t)out & 15) == 0 && (dr == 0 || turned != nullptr),
               "latent attention (tcgen05): pointers must be 16-byte aligned");
    if (n_tiles == 0) return MM_OK;
    const LtLayout a = lt_layout(dk, dr, dv);
    const long long ld = (long long)H * (dk + dv), qw = (long long)H * a.pieces * 64;
    CUtensorMap tq, tk, tr, tv;
    const __nv_bfloat16* kvp = (const __nv_bfloat16*)kv;
    if (!tc::make_map_bf16(&tq, q, n_tokens, (int)qw, qw, 128) || !tc::make_map_bf16(&tk, kvp, key_rows, H * dk, ld, 128) ||
        !(dr > 0 ? tc::make_map_bf16(&tr, turned, key_rows, dr, dr, 128) : tc::make_map_bf16(&tr, kvp, key_rows, H * dk, ld, 128)) ||
        !tc::make_map_bf16(&tv, kvp + (size_t)H * dk, key_rows, H * dv, ld, 64)) {
        mm_set_last_error("latent attention (tcgen05): cuTensorMapEncodeTiled failed or is not available");
        return MM_ERR_DRIVER;
    }
    cudaStream_t s = (cudaStream_t)stream;
    if (a.vh == 1) return lt_launch<1>(tq, tk, tr, tv, out, tiles, n_tiles, H, dk, dv, a, scale, sink, err, s);
    return lt_launch<2>(tq, tk, tr, tv, out, tiles, n_tiles, H, dk, dv, a, scale, sink, err, s);
}

// Cached latent rows of several requests side by side: row i of request entry e (its rows start at meta[3 e + 1], meta[3 e + 2] of
// them) comes from token i's place in the pages of block-table row meta[3 e]; its first `rank` numbers go to c [rows, rank], the
// rest to turned [rows, wide - rank].  A warp per row, 16 bytes per lane.
__global__ void latent_gather_kernel(const __nv_bfloat16* __restrict__ pages, const int32_t* __restrict__ table, int table_width, int page_size,
                                     const int32_t* __restrict__ meta, int entries, int rows, int wide, int rank, __nv_bfloat16* __restrict__ c,
                                     __nv_bfloat16* __restrict__ turned) {
    const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= rows) return;
    int e = 0;
    while (e + 1 < entries && row >= meta[3 * (e + 1) + 1]) ++e;
    const int key = row - meta[3 * e + 1];
    if (key >= meta[3 * e + 2]) return;
    const int page = table[(size_t)meta[3 * e] * table_width + key / page_size];
    const __nv_bfloat16* src = pages + ((size_t)page * page_size + key % page_size) * wide;
    const int extra = wide - rank;
    for (int i = lane * 8; i < wide; i += 256) {
        const uint4 v = *reinterpret_cast<const uint4*>(src + i);
        if (i < rank) *reinterpret_cast<uint4*>(c + (size_t)row * rank + i) = v;
        else *reinterpret_cast<uint4*>(turned + (size_t)row * extra + i - rank) = v;
    }
}

MM_EXPORT int mm_latent_gather(const void* pages, const void* table, int table_width, int page_size, const void* meta, int entries, int rows, int wide,
                               int rank, void* c, void* turned, void* stream) {
    MM_REQUIRE(entries > 0 && rows >= 0 && page_size > 0 && table_width > 0 && rank > 0 && wide >= rank && rank % 8 == 0 && wide % 8 == 0,
               "latent gather: bad sizes");
    MM_REQUIRE(((uintptr_t)pages & 15) == 0 && ((uintptr_t)c & 15) == 0 && ((uintptr_t)turned & 15) == 0, "latent gather: pointers must be 16-byte aligned");
    if (rows == 0) return MM_OK;
    mm_launch(latent_gather_kernel, dim3(ceil_div(rows, 8)), dim3(256), 0, (cudaStream_t)stream, (const __nv_bfloat16*)pages, (const int32_t*)table, table_width,
              page_size, (const int32_t*)meta, entries, rows, wide, rank, (__nv_bfloat16*)c, (__nv_bfloat16*)turned);
    MM_CHECK_LAUNCH();
    return MM_OK;
}
