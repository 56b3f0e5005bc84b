// Blackwell-native causal flash-prefill over the paged KV cache: tcgen05 MMAs for Q.K^T and P.V with S and O in tensor memory,
// K / V pages brought in by TMA.
//
// Reference counterpart: flash_attn_ext_f16 (llama.cpp/ggml/src/ggml-cuda/fattn-mma-f16.cuh:38-104), an FA-2 schedule on
// mma.sync + cp.async with the accumulators in registers - which is also what attention.cu:attn_prefill_kernel is.  This kernel
// is the sm_100a form of the same algorithm:
//
//   CTA = one tile of 128 queries of one query head.  192 threads (320 where four more softmax warps share a row):
//     warp 0      producer   TMA: the Q tile once, then per 128-key tile the K and V rows page by page (the block table gives the
//                            page ids; a page is a contiguous [page_size x D] block, box {64, page_size} of a 2-D map over the cache)
//     warp 1      MMA        one thread issues  S = Q.K^T  (M = 128 queries, N = 128 keys, K = D) into one of two TMEM S buffers,
//                            and  O += P.V  (M = 128, N = D, K = 128 keys) into the TMEM O accumulator.  V stays in its cache
//                            layout [key][D]: it is the *MN-major* B operand (descriptor: 128-byte swizzle atoms of 8 keys x 64
//                            dims, SBO = 1024 B between key groups, LBO = distance between the two 64-dim halves).
//     warps 2-5   softmax    thread r owns query row r: tcgen05.ld of its S row, causal mask on the diagonal tiles, running
//                            max / sum, P = exp2(..) written as fp16 into shared memory in the K-major swizzled layout the
//                            second MMA reads as its A operand.  O is rescaled in TMEM only when a row maximum actually grew
//                            (warp-uniform test), and normalised + stored as fp16 at the end.
//                            (FA_ROWS / FA_TILES: warps 2-5 and 6-9 take 64 keys of every tile each, with a maximum, a sum and an O
//                            accumulator of their own, and join them at the end.)
//   QK^T of tile i+1 is issued before P.V of tile i, so the tensor pipe works on the next scores while the softmax warps are
//   busy; K/V stages form a 2-deep ring.
#pragma once
#include <string.h>

#include "kernels.cuh"
#include "mma.cuh"

namespace dlp {

int make_tmap_2d(CUtensorMap* out, const void* base, int is_bf16, uint64_t rows, uint64_t K, uint64_t ld, uint32_t box_rows);

__device__ __forceinline__ void tmem_st_32x32(uint32_t taddr, const uint32_t (&r)[32]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,"
        "%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};"
        ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
          "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]),
          "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]),
          "r"(r[30]), "r"(r[31])
        : "memory");
}
__device__ __forceinline__ void tc_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// mbarrier wait with a limit: a protocol error ends as an error flag the host reads, not as a GPU that spins forever.  Once the flag is
// up every later wait gives up at once, so the kernel runs to its end, frees its tensor memory and returns (with wrong results).
// Without a flag (FA_PAGED) the kernel traps: an error the host sees as well.
__device__ __forceinline__ void mbar_wait_g(uint64_t* bar, uint32_t parity, int* error) {
    for (unsigned spins = 0; !mbar_try_wait(bar, parity); ++spins) {
        if (error != nullptr && (spins & 1023u) == 1023u && *reinterpret_cast<volatile int*>(error) != 0) return;
        if (spins > (1u << 24)) {
            if (error == nullptr) __trap();
            atomicExch(error, 1);
            return;
        }
    }
}

// MN-major operand in the 128-byte-swizzled layout TMA produces for rows of 64 fp16: atoms of 8 rows (1024 B); `lbo_bytes` =
// distance between consecutive 64-element chunks along the MN dimension, SBO = 1024 B between groups of 8 rows along K.
__device__ __forceinline__ uint64_t make_smem_desc_sw128_mn(uint32_t smem_addr, uint32_t lbo_bytes) {
    uint64_t d = 0;
    d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
    d |= (uint64_t)((lbo_bytes >> 4) & 0x3FFF) << 16;
    d |= (uint64_t)(1024 >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
// kind::f16 instruction descriptor with an MN-major B operand (bit 16)
__host__ __device__ constexpr uint32_t make_idesc_f16_bmn(int m, int n, int fmt) { return make_idesc_f16(m, n, fmt) | (1u << 16); }

struct FaParams {
    const int* bt_row;      // FA_PAGED: block-table row of the sequence
    void* out;              // [T, ldo] fp16 (FA_PAGED) or bf16
    int T, pos0, Hq, Hkv, page_size, max_pages;
    int ldo;
    // FA_ROWS
    const float* gate;      // [T, ldg] one logit per query head: the head's output is multiplied by its sigmoid (nullptr: not gated)
    int ldg, V;             // V: value size of a head (<= D2; the rest of the tile is padding)
    float scale;
    int* error;             // set when a wait ran into its limit
    int window, keep, chunk;       // (FA_PAGED: none) position i sees key j <= i when i - j < window and (chunk > 0) both are in one chunk, or when j < keep
    // FA_TILES
    const int* tile_row0;   // [grid.x] first query row of a tile, and its rows (consecutive positions of one sequence)
    const int* tile_rows;
    const int* pos;         // [T]
    const int* tok_slot;    // [T] block-table row
    const int* block_table;
    int q_head;             // columns from one query head to the next
    int maps, out_f32;      // maps: query heads take turns over that many key heads of a key / value head;  out is fp32
};
// FA_PAGED: fp16, K / V pages of a [pages][Hkv][page][D] cache, queries scaled in advance, fp16 softmax weights
// FA_ROWS:  bf16, K / V as plain rows [keys][Hkv * D1 | D2], scores scaled in fp32, every softmax weight as two bf16 parts (value and
//           remainder, two MMAs), optional output gate
// FA_TILES: bf16 with the numerics of FA_ROWS, K / V pages of [pages][Hkv][page][<= D1 | <= D2] caches (tensor maps complete narrower heads
//           with zeros), tiles of several sequences, sliding window with kept first keys, chunks: only key tiles that some row sees are read
enum FaMode : int { FA_PAGED = 0, FA_ROWS = 1, FA_TILES = 2 };

template <int D1, int D2, int MODE>
struct FaCfg {
    static constexpr int BM = 128, BN = D1 > 128 ? 64 : 128;      // (wider keys: shorter key tiles)
    static constexpr int KB = D1 / 64, VB = D2 / 64;
    static constexpr int Q_BYTES = BM * D1 * 2;
    static constexpr int K_BYTES = BN * D1 * 2, V_BYTES = BN * D2 * 2;
    static constexpr int P_PARTS = MODE == FA_PAGED ? 1 : 2;
    static constexpr int P_BYTES = BM * BN * 2;      // one part
    static constexpr int HALVES = MODE == FA_PAGED ? 1 : 2;      // groups of four softmax warps; each takes its part of a key tile into an O of its own
    static constexpr int THREADS = 64 + 128 * HALVES;
    static constexpr int STAGES = 2;
    static constexpr int SMEM_BYTES = Q_BYTES + STAGES * (K_BYTES + V_BYTES) + P_PARTS * P_BYTES + 1024 + 256;
    static constexpr int TMEM_COLS = 512;            // S0 [0,128)  S1 [128,256)  O [256, 256 + HALVES * D2)
    static constexpr int O_COL = 256;
};

template <int D1, int D2, int MODE>
__global__ void __launch_bounds__((FaCfg<D1, D2, MODE>::THREADS), 1)
attn_prefill_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                       const __grid_constant__ CUtensorMap tm_v, const FaParams p) {
    using Cfg = FaCfg<D1, D2, MODE>;
    constexpr int BM = Cfg::BM, BN = Cfg::BN, KB = Cfg::KB, VB = Cfg::VB, HALVES = Cfg::HALVES, FMT = MODE == FA_PAGED ? 0 : 1;
    constexpr bool EXACT = MODE != FA_PAGED;                     // fp32 scores times scale, split softmax weights
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* sm_q = smem;                                        // [KB][128 rows][128 B]
    uint8_t* sm_k = sm_q + Cfg::Q_BYTES;                         // [stage][KB][BN rows][128 B]
    uint8_t* sm_v = sm_k + Cfg::STAGES * Cfg::K_BYTES;           // [stage][VB (dim halves)][BN keys][128 B]
    uint8_t* sm_p = sm_v + Cfg::STAGES * Cfg::V_BYTES;           // [part][BN / 64][128 rows][128 B]
    uint64_t* bars = reinterpret_cast<uint64_t*>(sm_p + Cfg::P_PARTS * Cfg::P_BYTES);
    uint64_t* q_full = bars;
    uint64_t* k_full = bars + 1;      // [2]
    uint64_t* v_full = bars + 3;      // [2]
    uint64_t* k_empty = bars + 5;     // [2]
    uint64_t* v_empty = bars + 7;     // [2]
    uint64_t* s_full = bars + 9;      // [2]
    uint64_t* s_free = bars + 11;     // [2]
    uint64_t* p_full = bars + 13;     // [HALVES]
    uint64_t* pv_done = bars + 15;    // [HALVES]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 17);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int qt = gridDim.x - 1 - blockIdx.x;        // heaviest (latest) query tiles first (FA_TILES: in the order of the table)
    const int t0 = MODE == FA_TILES ? p.tile_row0[blockIdx.x] : qt * BM;
    const int rows = MODE == FA_TILES ? p.tile_rows[blockIdx.x] : min(BM, p.T - t0);
    const int pos_t = MODE == FA_TILES ? p.pos[t0] : p.pos0 + t0;      // position of the first row
    const int* bt_row = MODE == FA_TILES ? p.block_table + (size_t)p.tok_slot[t0] * p.max_pages : p.bt_row;
    const int hq = blockIdx.y;
    const int kvh = hq / (p.Hq / p.Hkv);
    const int q_hi = pos_t + rows;                    // keys visible to the last query of this tile
    auto first_key = [&](int pos) { return max(max(0, pos - p.window + 1), p.chunk > 0 ? pos / p.chunk * p.chunk : 0); };
    const int lo_tile = EXACT ? first_key(pos_t) / BN : 0;                       // first key tile the window shows
    const int keep_tiles = EXACT ? min((p.keep + BN - 1) / BN, lo_tile) : 0;      // kept tiles in front of it
    const int n_tiles = keep_tiles + (q_hi + BN - 1) / BN - lo_tile;
    auto key_of = [&](int i) { return (EXACT && i >= keep_tiles ? lo_tile - keep_tiles + i : i) * BN; };

    if (warp == 0 && lane == 0) {
        tma_prefetch_desc(&tm_q);
        tma_prefetch_desc(&tm_k);
        tma_prefetch_desc(&tm_v);
        mbar_init(q_full, 1);
        for (int s = 0; s < 2; ++s) {
            mbar_init(&k_full[s], 1);
            mbar_init(&v_full[s], 1);
            mbar_init(&k_empty[s], 1);
            mbar_init(&v_empty[s], 1);
            mbar_init(&s_full[s], 1);
            mbar_init(&s_free[s], 4 * HALVES);
        }
        for (int h = 0; h < HALVES; ++h) {
            mbar_init(&p_full[h], 4);
            mbar_init(&pv_done[h], 1);
        }
        mbar_fence_init();
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, Cfg::TMEM_COLS);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        // ===== producer =====
        if (lane == 0) {
            mbar_expect_tx(q_full, Cfg::Q_BYTES);
            for (int kb = 0; kb < KB; ++kb) tma_load_2d(sm_q + kb * (BM * 128), &tm_q, q_full, hq * (MODE == FA_TILES ? p.q_head : D1) + kb * 64, t0);
            const int ps = MODE == FA_ROWS ? BN : p.page_size, chunks = BN / ps;
            for (int i = 0; i < n_tiles; ++i) {
                const int s = i & 1;
                const uint32_t ph = (uint32_t)(i >> 1) & 1u;
                const int n0 = key_of(i);
                auto row_of = [&](int pc, bool key) {
                    if (MODE == FA_ROWS) return n0;
                    const int pi = min((n0 + pc * ps) / ps, p.max_pages - 1), head = bt_row[pi] * p.Hkv + kvh;
                    return (MODE == FA_TILES && key ? head * p.maps + hq % p.maps : head) * ps;
                };
                mbar_wait_g(&k_empty[s], ph ^ 1, p.error);
                mbar_expect_tx(&k_full[s], Cfg::K_BYTES);
                for (int pc = 0; pc < chunks; ++pc) {
                    const int row = row_of(pc, true);
                    for (int kb = 0; kb < KB; ++kb)
                        tma_load_2d(sm_k + s * Cfg::K_BYTES + kb * (BN * 128) + pc * (ps * 128), &tm_k, &k_full[s], (MODE == FA_ROWS ? kvh * D1 : 0) + kb * 64, row);
                }
                mbar_wait_g(&v_empty[s], ph ^ 1, p.error);
                mbar_expect_tx(&v_full[s], Cfg::V_BYTES);
                for (int pc = 0; pc < chunks; ++pc) {
                    const int row = row_of(pc, false);
                    for (int kb = 0; kb < VB; ++kb)
                        tma_load_2d(sm_v + s * Cfg::V_BYTES + kb * (BN * 128) + pc * (ps * 128), &tm_v, &v_full[s], (MODE == FA_ROWS ? kvh * D2 : 0) + kb * 64, row);
                }
            }
        }
    } else if (warp == 1) {
        // ===== MMA issuer =====
        if (lane == 0) {
            constexpr uint32_t idesc_s = make_idesc_f16(BM, BN, FMT);
            constexpr uint32_t idesc_o = make_idesc_f16_bmn(BM, D2, FMT);
            auto issue_pv = [&](int j) {
                const int s = j & 1;
                mbar_wait_g(&v_full[s], (uint32_t)(j >> 1) & 1u, p.error);
#pragma unroll
                for (int h = 0; h < HALVES; ++h) {
                    mbar_wait_g(&p_full[h], (uint32_t)j & 1u, p.error);
                    tc_fence_after();
#pragma unroll
                    for (int kk = h * (BN / 16 / HALVES); kk < (h + 1) * (BN / 16 / HALVES); ++kk) {
                        const uint64_t db = make_smem_desc_sw128_mn(smem_u32(sm_v + s * Cfg::V_BYTES + kk * 16 * 128), BN * 128);
#pragma unroll
                        for (int part = 0; part < Cfg::P_PARTS; ++part) {
                            const uint64_t da = make_smem_desc_sw128(smem_u32(sm_p + part * Cfg::P_BYTES + (kk >> 2) * (BM * 128))) + (uint64_t)(2 * (kk & 3));
                            tc_mma_f16(tmem_base + Cfg::O_COL + h * D2, da, db, idesc_o, (j > 0 || kk > h * (BN / 16 / HALVES) || part > 0) ? 1u : 0u);
                        }
                    }
                    tc_commit(&pv_done[h]);
                }
                tc_commit(&v_empty[s]);
            };
            mbar_wait_g(q_full, 0, p.error);
            for (int i = 0; i < n_tiles; ++i) {
                const int s = i & 1;
                const uint32_t ph = (uint32_t)(i >> 1) & 1u;
                mbar_wait_g(&k_full[s], ph, p.error);
                mbar_wait_g(&s_free[s], ph ^ 1, p.error);
                tc_fence_after();
#pragma unroll
                for (int kb = 0; kb < KB; ++kb) {
                    const uint64_t da = make_smem_desc_sw128(smem_u32(sm_q + kb * (BM * 128)));
                    const uint64_t db = make_smem_desc_sw128(smem_u32(sm_k + s * Cfg::K_BYTES + kb * (BN * 128)));
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        tc_mma_f16(tmem_base + s * BN, da + (uint64_t)(2 * k), db + (uint64_t)(2 * k), idesc_s, (kb > 0 || k > 0) ? 1u : 0u);
                }
                tc_commit(&k_empty[s]);
                tc_commit(&s_full[s]);
                if (i > 0) issue_pv(i - 1);       // scores of tile i are on their way while P.V of tile i-1 runs
            }
            issue_pv(n_tiles - 1);
        }
    } else {
        // ===== softmax / correction / epilogue: thread (half, r) <-> query row r, key columns [half * CW, + CW) of every tile =====
        constexpr int CW = BN / HALVES;
        const int q4 = warp & 3;                       // TMEM lane quarter this warp may access
        const int half = (warp - 2) >> 2;              // its own running maximum, sum and O accumulator
        const int r = q4 * 32 + lane;
        const int q_pos = pos_t + r;                   // this query attends to keys 0 .. q_pos
        const int q_first = EXACT ? first_key(q_pos) : 0, q_first_hi = EXACT ? first_key(q_hi - 1) : 0;      // (from its first key on, and the kept ones)
        const uint32_t lane_addr = tmem_base + ((uint32_t)(q4 * 32) << 16);
        const uint32_t o_addr = lane_addr + Cfg::O_COL + half * D2;
        constexpr float LOG2E = 1.4426950408889634f;
        const float c_in = EXACT ? p.scale * LOG2E : 1.f;         // EXACT: scores in units of log 2 from here on
        constexpr float C_EXP = EXACT ? 1.f : LOG2E;
        float m_run = -INFINITY, l_run = 0.f;
        const int sw = r & 7;
        for (int i = 0; i < n_tiles; ++i) {
            const int s = i & 1;
            const int n0 = key_of(i) + half * CW;
            mbar_wait_g(&s_full[s], (uint32_t)(i >> 1) & 1u, p.error);
            tc_fence_after();
            uint32_t sv[CW];
#pragma unroll
            for (int c = 0; c < CW / 32; ++c) tmem_ld_32x32(lane_addr + s * BN + half * CW + c * 32, *reinterpret_cast<uint32_t(*)[32]>(&sv[c * 32]));
            tc_wait_ld();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&s_free[s]);    // the next-but-one score tile may overwrite this buffer
            if (EXACT) {
#pragma unroll
                for (int j = 0; j < CW; ++j) sv[j] = __float_as_uint(__uint_as_float(sv[j]) * c_in);
            }
            if (n0 + CW - 1 > pos_t || (EXACT && q_first_hi > n0 && n0 + CW > p.keep)) {     // some (query, key) pairs are masked
#pragma unroll
                for (int j = 0; j < CW; ++j)
                    if (n0 + j > q_pos || (EXACT && n0 + j < q_first && n0 + j >= p.keep)) sv[j] = __float_as_uint(-INFINITY);
            }
            float mx[4] = {m_run, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int j = 0; j < CW; ++j) mx[j & 3] = fmaxf(mx[j & 3], __uint_as_float(sv[j]));
            const float m_new = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
            const float ms = (m_new == -INFINITY) ? 0.f : m_new * C_EXP;
            const float alpha = (m_run == -INFINITY) ? 0.f : exp2f(m_run * C_EXP - ms);
            float sum[2] = {0.f, 0.f};
            // the weights replace the scores in registers: fp16 pairs in the lower half of sv (FA_PAGED), or fp32 until they are split
#pragma unroll
            for (int j = 0; j < CW; j += 2) {
                const float p0 = exp2f(__uint_as_float(sv[j]) * C_EXP - ms);
                const float p1 = exp2f(__uint_as_float(sv[j + 1]) * C_EXP - ms);
                if (EXACT) {
                    sum[0] += p0;
                    sum[1] += p1;
                    sv[j] = __float_as_uint(p0);
                    sv[j + 1] = __float_as_uint(p1);
                } else {
                    const __half2 h = __floats2half2_rn(p0, p1);
                    const float2 hf = __half22float2(h);             // the sum uses the rounded values the tensor core will see
                    sum[0] += hf.x + hf.y;
                    sv[j / 2] = *reinterpret_cast<const uint32_t*>(&h);
                }
            }
            l_run = l_run * alpha + (sum[0] + sum[1]);
            m_run = m_new;
            if (i > 0) {
                mbar_wait_g(&pv_done[half], (uint32_t)(i - 1) & 1u, p.error);       // P.V of the previous tile has read P and updated O
                tc_fence_after();
                if (__any_sync(0xffffffffu, alpha != 1.f)) {      // a row maximum grew: rescale this warp's 32 rows of O
#pragma unroll 1
                    for (int c = 0; c < D2 / 32; ++c) {
                        uint32_t o[32];
                        tmem_ld_32x32(o_addr + c * 32, o);
                        tc_wait_ld();
#pragma unroll
                        for (int j = 0; j < 32; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
                        tmem_st_32x32(o_addr + c * 32, o);
                    }
                    tc_wait_st();
                }
            }
            // P row -> shared memory, K-major swizzled (16-byte chunk c of 64-key block b lands at chunk c ^ (r & 7))
#pragma unroll
            for (int b = 0; b < (CW + 63) / 64; ++b)
#pragma unroll
                for (int c = 0; c < (CW < 64 ? CW : 64) / 8; ++c) {
                    const int col = half * CW + b * 64 + c * 8;
                    uint8_t* dst = sm_p + (col >> 6) * (BM * 128) + r * 128 + ((((col & 63) >> 3) ^ sw) << 4);
                    if (EXACT) {
                        uint32_t hi[4], lo[4];
#pragma unroll
                        for (int e = 0; e < 4; ++e) split_bf16(__uint_as_float(sv[b * 64 + c * 8 + 2 * e]), __uint_as_float(sv[b * 64 + c * 8 + 2 * e + 1]), hi[e], lo[e]);
                        *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                        *reinterpret_cast<uint4*>(dst + Cfg::P_BYTES) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
                    } else {
                        *reinterpret_cast<uint4*>(dst) = make_uint4(sv[b * 32 + c * 4], sv[b * 32 + c * 4 + 1], sv[b * 32 + c * 4 + 2], sv[b * 32 + c * 4 + 3]);
                    }
                }
            fence_proxy_async();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[half]);
        }
        // epilogue: O / l in the output type; with two halves their accumulators are joined here
        for (int h = 0; h < HALVES; ++h) mbar_wait_g(&pv_done[h], (uint32_t)(n_tiles - 1) & 1u, p.error);
        tc_fence_after();
        float w0 = 1.f, w1 = 0.f;
        if constexpr (HALVES == 2) {
            float2* ml = reinterpret_cast<float2*>(sm_q);       // [half][128 rows]: every score product has read Q
            ml[half * BM + r] = make_float2(m_run, l_run);
            asm volatile("bar.sync 1, 256;" ::: "memory");      // the eight softmax warps
            const float2 a = ml[r], b = ml[BM + r];
            const float m = fmaxf(a.x, b.x);
            w0 = a.x == -INFINITY ? 0.f : exp2f(a.x - m);
            w1 = b.x == -INFINITY ? 0.f : exp2f(b.x - m);
            l_run = a.y * w0 + b.y * w1;
        }
        float inv = l_run > 0.f ? 1.f / l_run : 0.f;
        const int t = t0 + r;
        if (MODE == FA_ROWS && p.gate != nullptr && t < p.T) inv *= 1.f / (1.f + __expf(-p.gate[(size_t)t * p.ldg + hq]));
        w0 *= inv;
        w1 *= inv;
        const bool wide = EXACT && ((p.V | p.ldo) & 7) == 0 && (reinterpret_cast<uintptr_t>(p.out) & 15) == 0;
#pragma unroll 1
        for (int c = half * (D2 / 32 / HALVES); c < (half + 1) * (D2 / 32 / HALVES); ++c) {
            uint32_t o[32];
            tmem_ld_32x32(lane_addr + Cfg::O_COL + c * 32, o);
            if constexpr (HALVES == 2) {
                uint32_t o1[32];
                tmem_ld_32x32(lane_addr + Cfg::O_COL + D2 + c * 32, o1);
                tc_wait_ld();
#pragma unroll
                for (int j = 0; j < 32; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * w0 + __uint_as_float(o1[j]) * w1);
            } else {
                tc_wait_ld();
#pragma unroll
                for (int j = 0; j < 32; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * w0);
            }
            if (MODE == FA_TILES && p.out_f32) {
                float* orow = reinterpret_cast<float*>(p.out) + (size_t)t * p.ldo + (size_t)hq * p.V;
                if (((p.V | p.ldo) & 3) == 0 && (reinterpret_cast<uintptr_t>(p.out) & 15) == 0) {
#pragma unroll
                    for (int j = 0; j < 32; j += 4)
                        if (r < rows && c * 32 + j < p.V) *reinterpret_cast<uint4*>(orow + c * 32 + j) = make_uint4(o[j], o[j + 1], o[j + 2], o[j + 3]);
                } else {
#pragma unroll
                    for (int j = 0; j < 32; ++j)
                        if (r < rows && c * 32 + j < p.V) orow[c * 32 + j] = __uint_as_float(o[j]);
                }
            } else if (EXACT) {
                __nv_bfloat16* orow = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)t * p.ldo + (size_t)hq * p.V;
                if (wide) {
#pragma unroll
                    for (int j = 0; j < 32; j += 8) {
                        uint32_t w[4];
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const __nv_bfloat162 h = __floats2bfloat162_rn(__uint_as_float(o[j + 2 * e]), __uint_as_float(o[j + 2 * e + 1]));
                            w[e] = *reinterpret_cast<const uint32_t*>(&h);
                        }
                        if (r < rows && c * 32 + j < p.V) *reinterpret_cast<uint4*>(orow + c * 32 + j) = make_uint4(w[0], w[1], w[2], w[3]);
                    }
                } else {
#pragma unroll
                    for (int j = 0; j < 32; ++j)
                        if (r < rows && c * 32 + j < p.V) orow[c * 32 + j] = __float2bfloat16_rn(__uint_as_float(o[j]));
                }
            } else if (t < p.T) {
                __half* orow = reinterpret_cast<__half*>(p.out) + (size_t)t * p.ldo + (size_t)hq * D2;
#pragma unroll
                for (int j = 0; j < 32; j += 8) {
                    uint32_t w[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const __half2 h = __floats2half2_rn(__uint_as_float(o[j + 2 * e]), __uint_as_float(o[j + 2 * e + 1]));
                        w[e] = *reinterpret_cast<const uint32_t*>(&h);
                    }
                    *reinterpret_cast<uint4*>(orow + c * 32 + j) = make_uint4(w[0], w[1], w[2], w[3]);
                }
            }
            __syncwarp();
        }
    }
    if (p.error != nullptr && threadIdx.x == 0 && *reinterpret_cast<volatile int*>(p.error) != 0)
        for (int i = 0; i < 1000; ++i) __nanosleep(1000);      // a wait gave up: copies in flight land before the block goes away
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        __syncwarp();
        tmem_dealloc(tmem_base, Cfg::TMEM_COLS);
    }
}

}  // namespace dlp
