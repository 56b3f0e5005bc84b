// tcgen05 / TMEM / TMA GEMM for sm_100a:   Y[T, N] (op)= X[T, K] . W[N, K]^T
//
// Role in the engine: every prefill / batched-decode linear layer (QKV, attn-out, gate/up, down, lm_head).
// The reference runs these through cuBLAS GemmEx or its mma.sync MMQ kernels
// (llama.cpp/ggml/src/ggml-cuda/ggml-cuda.cu:1227-1371, mmq.cuh:3459); this is the Blackwell-native
// replacement: weights are the UMMA "A" operand (M = 128 output features per CTA), tokens are the "B"
// operand (N = BT tokens, 16..256), so small decode batches still fill the 128-lane datapath
// ("swap-AB"), accumulators live in TMEM and the epilogue (fp16/fp32 store, fp32 residual
// accumulate / split-K reduction, SwiGLU over a gate+up accumulator pair) reads them back with
// tcgen05.ld.  Operands arrive through TMA with the 128-byte swizzle; a 3..8 stage mbarrier ring
// decouples the TMA warp from the single MMA-issuing thread.
#pragma once
#include <string.h>

#include "kernels.cuh"

namespace dlp {

constexpr int GEMM_BM = 128;  // output features per CTA (UMMA M)
constexpr int GEMM_BK = 64;   // K elements per pipeline stage (= 128 B of fp16: one swizzle atom)

enum GemmEpilogue : int { EPI_STORE_F16 = 0, EPI_STORE_F32 = 1, EPI_ATOMIC_ADD_F32 = 2, EPI_SWIGLU_F16 = 3,
                          EPI_STORE_BF16 = 4, EPI_RS_PUSH_F32 = 5, EPI_GEGLU_BF16 = 6, EPI_RELU2_BF16 = 7, EPI_SWIGLU_BF16 = 8,
                          EPI_TAIL_BF16 = 9 /* OutTail: fp32, the second part as bf16 */ };
constexpr bool epi_is_gated(int e) { return e == EPI_SWIGLU_F16 || e == EPI_GEGLU_BF16 || e == EPI_SWIGLU_BF16; }   // two accumulators: gate and up

struct GemmParams {
    void* y;       // output [T, ldy]
    int T, N, K;   // tokens, output features, reduction
    int ldy;       // row stride of y in elements
    int epilogue;
    int k_blocks_per_split;
    GemmCollective coll;   // fused all-gather (X side) / reduce-scatter (Y side); zero-initialised = none
    GemmGroup grp;         // grouped (MoE) launch: per-tile expert / row range table built on the device
    // split-K with a deterministic fix-up (any epilogue): every split stores its fp32 partial tile into `ws`, the split that
    // arrives last at the tile's counter adds the partials in split order and runs the epilogue.  nullptr: not used.
    float* ws;
    unsigned* ws_counters;
    OutTail tail;          // EPI_TAIL_BF16
};

template <int BT, int NA>
struct GemmCfg {
    static constexpr int A_BYTES = GEMM_BM * GEMM_BK * 2;
    static constexpr int B_BYTES = BT * GEMM_BK * 2;
    static constexpr int STAGE_BYTES = NA * A_BYTES + B_BYTES;
    static constexpr int STAGES_RAW = (200 * 1024) / STAGE_BYTES;
    static constexpr int STAGES = STAGES_RAW > 8 ? 8 : STAGES_RAW;
    static constexpr int TMEM_COLS_RAW = NA * BT;
    static constexpr int TMEM_COLS = TMEM_COLS_RAW <= 32 ? 32 : TMEM_COLS_RAW <= 64 ? 64 : TMEM_COLS_RAW <= 128 ? 128
                                     : TMEM_COLS_RAW <= 256 ? 256 : 512;
    static constexpr int SMEM_BYTES = STAGES * STAGE_BYTES + 1024 /*align slack*/ + 256 /*barriers*/;
};

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + __expf(-x)); }
// tanh form of gelu: 0.5 (1 + tanh u) is the sigmoid of 2u
__device__ __forceinline__ float gelu_f(float x) { return x / (1.f + __expf(-1.5957691216057308f * (x + 0.044715f * x * x * x))); }

// ---- dequant-fused A operand ---------------------------------------------------------------------------
// For block-quantised weights the four epilogue warps (idle while the accumulator is being built) act as the
// A-operand producer: thread r owns row r of the 128-row tile, decodes that row's 64-element K slice from
// the GGUF blocks straight into shared memory as fp16 - in exactly the layout TMA would have produced
// (128-byte rows, 16-byte chunks XOR-swizzled by row % 8) - then fences the generic-proxy writes towards the
// async proxy and arrives on the stage's "full" barrier.  The tensor core never sees the difference; no
// dequantised copy of the weights ever exists in global memory.
template <int WT>
__device__ __forceinline__ void dequant_row_slice(const QWeight& w, int row, int kc, uint8_t* tile, int r) {
    uint8_t* dst = tile + r * 128;
    const int sw = r & 7;
    if (row >= w.N) {
#pragma unroll
        for (int c = 0; c < 8; ++c) *reinterpret_cast<uint4*>(dst + c * 16) = make_uint4(0, 0, 0, 0);
        return;
    }
    constexpr int NCH = (WT == W_Q6_K) ? 4 : 2;
    int cbase;
    if (WT == W_Q8_0) cbase = kc >> 5;
    else if (WT == W_Q6_K) cbase = (kc >> 8) * 8 + ((kc & 255) >> 7) * 4;
    else cbase = (kc >> 8) * 8 + ((kc & 255) >> 6) * 2;
    QChunk ch[NCH];
#pragma unroll
    for (int i = 0; i < NCH; ++i) load_chunk<WT>(w, row, cbase + i, ch[i]);   // all loads in flight before any math
#pragma unroll
    for (int i = 0; i < NCH; ++i) {
#pragma unroll
        for (int g = 0; g < 2; ++g) {
            const int e0 = ch[i].k[g] - kc;   // 16-aligned element offset inside the 64-wide slice (or outside it)
            if (e0 < 0 || e0 >= 64) continue;
            uint32_t o[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float2 f = __half22float2(ch[i].q[g][j]);
                const __half2 h = __floats2half2_rn(fmaf(ch[i].scale[g], f.x, ch[i].bias[g]), fmaf(ch[i].scale[g], f.y, ch[i].bias[g]));
                o[j] = *reinterpret_cast<const uint32_t*>(&h);
            }
            const int c0 = e0 >> 3;
            *reinterpret_cast<uint4*>(dst + ((c0 ^ sw) << 4)) = make_uint4(o[0], o[1], o[2], o[3]);
            *reinterpret_cast<uint4*>(dst + (((c0 + 1) ^ sw) << 4)) = make_uint4(o[4], o[5], o[6], o[7]);
        }
    }
}

template <int WT>
__device__ __forceinline__ void prefetch_row_slice(const QWeight& w, int row, int kc) {
    if (row >= w.N || kc >= w.K) return;
    if (WT == W_Q8_0) prefetch_l2(w.base + (size_t)row * w.K + kc);
    else if (WT == W_Q4_K) prefetch_l2(w.base + ((size_t)row * (w.K >> 8) + (kc >> 8)) * 144 + 16 + ((kc & 255) >> 6) * 32);
    else if (WT == W_Q5_K) prefetch_l2(w.base + ((size_t)row * (w.K >> 8) + (kc >> 8)) * 176 + 48 + ((kc & 255) >> 6) * 32);
    else if (WT == W_Q6_K) prefetch_l2(w.base + ((size_t)row * (w.K >> 8) + (kc >> 8)) * 128 + ((kc & 255) >> 7) * 64);
}

template <int MODE, int CH>
__device__ __forceinline__ void epi_loop(const GemmParams& p, const uint32_t (&r0)[CH], const uint32_t (&r1)[CH], int tb, int n, int t_end, float bias = 0.f) {
    if (MODE == EPI_RS_PUSH_F32) {
        // GEMM -> reduce-scatter: token t is owned by rank t / rs_rows; our partial for it goes straight into that rank's
        // reduce buffer, slot [our rank][t % rs_rows][n] (NVLink store).  Owner / local row advance incrementally.
        int owner = tb / p.coll.rs_rows;
        int local = tb - owner * p.coll.rs_rows;
        float* dst = p.coll.rs_peer_buf[owner] + ((size_t)p.coll.rs_rank * p.coll.rs_rows + local) * p.N + n;
#pragma unroll
        for (int j = 0; j < CH; ++j) {
            if (tb + j < t_end) *dst = __uint_as_float(r0[j]);
            dst += p.N;
            if (++local == p.coll.rs_rows) {
                local = 0;
                ++owner;
                if (owner < p.coll.rs_tp) dst = p.coll.rs_peer_buf[owner] + (size_t)p.coll.rs_rank * p.coll.rs_rows * p.N + n;
            }
        }
        return;
    }
    if (MODE == EPI_TAIL_BF16) {
        if (n < p.tail.n2) {
            float* dst = reinterpret_cast<float*>(p.y) + (size_t)tb * p.ldy + n;
#pragma unroll
            for (int j = 0; j < CH; ++j, dst += p.ldy)
                if (tb + j < t_end) *dst = __uint_as_float(r0[j]) + bias;
        } else {
            const float pos = p.tail.pos, neg = p.tail.neg;
            __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.tail.out2) + (size_t)tb * p.tail.ldo2 + (n - p.tail.n2);
#pragma unroll
            for (int j = 0; j < CH; ++j, dst += p.tail.ldo2)
                if (tb + j < t_end) *dst = __float2bfloat16_rn(xielu_fast(__uint_as_float(r0[j]) + bias, pos, neg));
        }
        return;
    }
    size_t o = (size_t)tb * p.ldy + n;
#pragma unroll
    for (int j = 0; j < CH; ++j, o += p.ldy) {
        if (tb + j >= t_end) break;
        const float v = __uint_as_float(r0[j]);
        if (MODE == EPI_STORE_F16) reinterpret_cast<__half*>(p.y)[o] = __float2half_rn(v);
        else if (MODE == EPI_STORE_BF16) reinterpret_cast<__nv_bfloat16*>(p.y)[o] = __float2bfloat16_rn(v);
        else if (MODE == EPI_STORE_F32) reinterpret_cast<float*>(p.y)[o] = v;
        else if (MODE == EPI_ATOMIC_ADD_F32) atomicAdd(reinterpret_cast<float*>(p.y) + o, v);
        else if (MODE == EPI_SWIGLU_F16) reinterpret_cast<__half*>(p.y)[o] = __float2half_rn(silu_f(v) * __uint_as_float(r1[j]));
        else if (MODE == EPI_GEGLU_BF16) reinterpret_cast<__nv_bfloat16*>(p.y)[o] = __float2bfloat16_rn(gelu_f(v) * __uint_as_float(r1[j]));
        else if (MODE == EPI_SWIGLU_BF16) reinterpret_cast<__nv_bfloat16*>(p.y)[o] = __float2bfloat16_rn(silu_f(v) * __uint_as_float(r1[j]));
        else if (MODE == EPI_RELU2_BF16) { const float u = fmaxf(v, 0.f); reinterpret_cast<__nv_bfloat16*>(p.y)[o] = __float2bfloat16_rn(u * u); }
    }
}

template <int BT, int NA, int AB_FMT, int WT>
__global__ void __launch_bounds__(192, 1)
gemm_tcgen05_kernel(const __grid_constant__ CUtensorMap tm_w0, const __grid_constant__ CUtensorMap tm_w1,
                    const __grid_constant__ CUtensorMap tm_x, const GemmParams p, const QWeight qw0, const QWeight qw1) {
    constexpr bool QUANT = (WT != W_F16);
    using Cfg = GemmCfg<BT, NA>;
    constexpr int STAGES = Cfg::STAGES;
    extern __shared__ uint8_t smem_raw[];
    // 1024-byte alignment is required by the 128B swizzle atoms
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* smem_a0 = smem;
    uint8_t* smem_a1 = smem + STAGES * Cfg::A_BYTES;  // only when NA == 2
    uint8_t* smem_b = smem + NA * STAGES * Cfg::A_BYTES;
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + STAGES * Cfg::STAGE_BYTES);
    uint64_t* full_bar = bars;
    uint64_t* empty_bar = bars + STAGES;
    uint64_t* tmem_full_bar = bars + 2 * STAGES;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * STAGES + 1);

    const int warp = threadIdx.x >> 5;
    const int lane = threadIdx.x & 31;
    int n0 = blockIdx.x * GEMM_BM;      // first weight row of this tile (A operand)
    int t0 = blockIdx.y * BT;           // first token row (B operand, output row)
    int t_end = p.T;                    // output rows >= t_end are not stored
    const int n_out0 = n0;              // first output column
    if (p.grp.tile_expert != nullptr) {
        // grouped launch: this token tile belongs to one expert; its weight rows sit at expert * rows_per_expert in the stack
        if ((int)blockIdx.y >= *p.grp.n_tiles) return;          // (uniform over the CTA, before any barrier / TMEM allocation)
        n0 += p.grp.tile_expert[blockIdx.y] * p.grp.rows_per_expert;
        t0 = p.grp.tile_row0[blockIdx.y];
        t_end = t0 + p.grp.tile_rows[blockIdx.y];
    }
    const int total_kb = (p.K + GEMM_BK - 1) / GEMM_BK;     // a partial last block is completed with zeros by the tensor maps
    const int kb_begin = blockIdx.z * p.k_blocks_per_split;
    const int kb_end = min(total_kb, kb_begin + p.k_blocks_per_split);
    const int num_kb = kb_end - kb_begin;

    if (warp == 0 && lane == 0) {
        tma_prefetch_desc(&tm_w0);
        if (NA == 2) tma_prefetch_desc(&tm_w1);
        tma_prefetch_desc(&tm_x);
        for (int s = 0; s < STAGES; ++s) {
            mbar_init(&full_bar[s], QUANT ? 5 : 1);   // TMA thread (+ one lane of each of the 4 dequant warps)
            mbar_init(&empty_bar[s], 1);
        }
        mbar_init(tmem_full_bar, 1);
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
        // ===== TMA producer =====
        if (lane == 0) {
            if (p.coll.x_flags != nullptr) {
                // all-gather -> GEMM: the token rows of this tile were pushed into our gather buffer by their owner
                // ranks; wait for exactly those owners, then order the acquired generic-proxy view before the TMA reads
                const int s0 = t0 / p.coll.x_rows_per_src, s1 = min(p.T - 1, t0 + BT - 1) / p.coll.x_rows_per_src;
                const long long c0 = clock64();
                const uint32_t x_epoch = sp_epoch(p.coll.step, p.coll.x_epoch);
                for (int src = s0; src <= s1; ++src) {
                    uint32_t v;
                    do {
                        asm volatile("ld.acquire.sys.global.u32 %0, [%1];" : "=r"(v) : "l"(p.coll.x_flags + src) : "memory");
                        if (clock64() - c0 > (1ll << 34)) { if (p.coll.error) atomicExch(p.coll.error, 1); break; }
                    } while ((int32_t)(v - x_epoch) < 0);
                }
                fence_proxy_async_global();
            }
            int stage = 0;
            uint32_t phase = 0;
            for (int kb = 0; kb < num_kb; ++kb) {
                mbar_wait(&empty_bar[stage], phase ^ 1);
                mbar_expect_tx(&full_bar[stage], QUANT ? Cfg::B_BYTES : Cfg::STAGE_BYTES);
                const int kc = (kb_begin + kb) * GEMM_BK;
                if (!QUANT) {
                    tma_load_2d(smem_a0 + stage * Cfg::A_BYTES, &tm_w0, &full_bar[stage], kc, n0);
                    if (NA == 2) tma_load_2d(smem_a1 + stage * Cfg::A_BYTES, &tm_w1, &full_bar[stage], kc, n0);
                }
                tma_load_2d(smem_b + stage * Cfg::B_BYTES, &tm_x, &full_bar[stage], kc, t0);
                if (++stage == STAGES) { stage = 0; phase ^= 1; }
            }
        }
    } else if (warp == 1) {
        // ===== MMA issuer (one thread) =====
        if (lane == 0) {
            constexpr uint32_t idesc = make_idesc_f16(GEMM_BM, BT, AB_FMT);
            int stage = 0;
            uint32_t phase = 0;
            for (int kb = 0; kb < num_kb; ++kb) {
                mbar_wait(&full_bar[stage], phase);
                tc_fence_after();
                const uint64_t da0 = make_smem_desc_sw128(smem_u32(smem_a0 + stage * Cfg::A_BYTES));
                const uint64_t da1 = make_smem_desc_sw128(smem_u32(smem_a1 + stage * Cfg::A_BYTES));
                const uint64_t db = make_smem_desc_sw128(smem_u32(smem_b + stage * Cfg::B_BYTES));
#pragma unroll
                for (int k = 0; k < GEMM_BK / 16; ++k) {
                    const uint32_t acc = (kb > 0 || k > 0) ? 1u : 0u;
                    // +32 bytes (>>4 = 2) per 16-element K step inside the swizzle atom
                    tc_mma_f16(tmem_base, da0 + (uint64_t)(2 * k), db + (uint64_t)(2 * k), idesc, acc);
                    if (NA == 2) tc_mma_f16(tmem_base + BT, da1 + (uint64_t)(2 * k), db + (uint64_t)(2 * k), idesc, acc);
                }
                tc_commit(&empty_bar[stage]);  // frees this smem slot once the MMAs above have read it
                if (++stage == STAGES) { stage = 0; phase ^= 1; }
            }
            tc_commit(tmem_full_bar);  // accumulator complete
        }
    } else {
        if constexpr (QUANT) {
            // ===== dequant producers (the epilogue warps, before there is anything to drain) =====
            const int r = (warp - 2) * 32 + lane;
            int stage = 0;
            uint32_t phase = 0;
            for (int kb = 0; kb < num_kb; ++kb) {
                const int kc = (kb_begin + kb) * GEMM_BK;
                prefetch_row_slice<WT>(qw0, n0 + r, kc + 4 * GEMM_BK);
                if (NA == 2) prefetch_row_slice<WT>(qw1, n0 + r, kc + 4 * GEMM_BK);
                mbar_wait(&empty_bar[stage], phase ^ 1);
                dequant_row_slice<WT>(qw0, n0 + r, kc, smem_a0 + stage * Cfg::A_BYTES, r);
                if (NA == 2) dequant_row_slice<WT>(qw1, n0 + r, kc, smem_a1 + stage * Cfg::A_BYTES, r);
                fence_proxy_async();   // generic-proxy smem writes -> visible to tcgen05 (async proxy)
                __syncwarp();
                if (lane == 0) mbar_arrive(&full_bar[stage]);
                if (++stage == STAGES) { stage = 0; phase ^= 1; }
            }
        }
        // ===== epilogue: 4 warps, warp%4 selects the TMEM lane quarter =====
        const int q = warp & 3;
        const int n_local = q * 32 + lane;
        const int n = n_out0 + n_local;
        const float bias = p.epilogue == EPI_TAIL_BF16 && p.tail.bias != nullptr && n < p.N ? p.tail.bias[n] : 0.f;      // (requested before the accumulators are there)
        if (num_kb > 0) {
            mbar_wait(tmem_full_bar, 0);
            tc_fence_after();
        }
        const uint32_t lane_addr = tmem_base + ((uint32_t)(q * 32) << 16);
        constexpr int CH = BT >= 32 ? 32 : 16;
        const int S = gridDim.z;
        const bool split_ws = p.ws != nullptr && S > 1;
        const size_t tile = (size_t)blockIdx.y * gridDim.x + blockIdx.x;
        auto load_acc = [&](int c, uint32_t (&r0)[CH], uint32_t (&r1)[CH]) {
            if (num_kb > 0) {
                if constexpr (CH == 32) {
                    tmem_ld_32x32(lane_addr + c * CH, r0);
                    if (NA == 2) tmem_ld_32x32(lane_addr + BT + c * CH, r1);
                } else {
                    tmem_ld_32x16(lane_addr + c * CH, r0);
                    if (NA == 2) tmem_ld_32x16(lane_addr + BT + c * CH, r1);
                }
                tc_wait_ld();
            } else {
#pragma unroll
                for (int j = 0; j < CH; ++j) { r0[j] = 0; r1[j] = 0; }
            }
        };
        auto run_epilogue = [&](int c, const uint32_t (&r0)[CH], const uint32_t (&r1)[CH]) {
            if (n < p.N) {
                // one specialised store loop per epilogue (dispatch hoisted out of the per-element loop: a switch with the
                // reduce-scatter address arithmetic inside it cost 35-50 % of the whole GEMM, see profiles/r1_gemm_ab.txt)
                const int tb = t0 + c * CH;
                switch (p.epilogue) {
                    case EPI_STORE_F16: epi_loop<EPI_STORE_F16, CH>(p, r0, r1, tb, n, t_end); break;
                    case EPI_STORE_BF16: epi_loop<EPI_STORE_BF16, CH>(p, r0, r1, tb, n, t_end); break;
                    case EPI_STORE_F32: epi_loop<EPI_STORE_F32, CH>(p, r0, r1, tb, n, t_end); break;
                    case EPI_ATOMIC_ADD_F32: epi_loop<EPI_ATOMIC_ADD_F32, CH>(p, r0, r1, tb, n, t_end); break;
                    case EPI_SWIGLU_F16: if (NA == 2) epi_loop<EPI_SWIGLU_F16, CH>(p, r0, r1, tb, n, t_end); break;
                    case EPI_GEGLU_BF16: if (NA == 2 && AB_FMT == 1) epi_loop<EPI_GEGLU_BF16, CH>(p, r0, r1, tb, n, t_end); break;
                    case EPI_SWIGLU_BF16: if (NA == 2 && AB_FMT == 1) epi_loop<EPI_SWIGLU_BF16, CH>(p, r0, r1, tb, n, t_end); break;
                    case EPI_RELU2_BF16: if (NA == 1 && AB_FMT == 1) epi_loop<EPI_RELU2_BF16, CH>(p, r0, r1, tb, n, t_end); break;
                    case EPI_TAIL_BF16: if (NA == 1 && AB_FMT == 1) epi_loop<EPI_TAIL_BF16, CH>(p, r0, r1, tb, n, t_end, bias); break;
                    case EPI_RS_PUSH_F32: epi_loop<EPI_RS_PUSH_F32, CH>(p, r0, r1, tb, n, t_end); break;
                }
            }
        };
        if (!split_ws) {
#pragma unroll 1
            for (int c = 0; c < BT / CH; ++c) {
                if (t0 + c * CH >= t_end) break;  // warp-uniform
                uint32_t r0[CH], r1[CH];
                load_acc(c, r0, r1);
                run_epilogue(c, r0, r1);
            }
        } else {
            // partial tile -> workspace [tile][split][accumulator][token][128 features] (128 consecutive floats per store round)
            __shared__ int s_last;
            float* wsp = p.ws + ((tile * S + blockIdx.z) * NA) * (size_t)BT * GEMM_BM;
#pragma unroll 1
            for (int c = 0; c < BT / CH; ++c) {
                if (t0 + c * CH >= t_end) break;
                uint32_t r0[CH], r1[CH];
                load_acc(c, r0, r1);
#pragma unroll
                for (int j = 0; j < CH; ++j) {
                    __stcg(wsp + (size_t)(c * CH + j) * GEMM_BM + n_local, __uint_as_float(r0[j]));
                    if (NA == 2) __stcg(wsp + (size_t)(BT + c * CH + j) * GEMM_BM + n_local, __uint_as_float(r1[j]));
                }
            }
            __threadfence();
            asm volatile("bar.sync 1, 128;" ::: "memory");
            if (threadIdx.x == 64) s_last = (atomicAdd(p.ws_counters + tile, 1u) == (unsigned)(S - 1)) ? 1 : 0;
            asm volatile("bar.sync 1, 128;" ::: "memory");
            if (s_last) {
                __threadfence();
                const float* base = p.ws + (tile * S * NA) * (size_t)BT * GEMM_BM;
#pragma unroll 1
                for (int c = 0; c < BT / CH; ++c) {
                    if (t0 + c * CH >= t_end) break;
                    uint32_t r0[CH], r1[CH];
#pragma unroll
                    for (int j = 0; j < CH; ++j) {
                        float a0 = 0.f, a1 = 0.f;
                        for (int z = 0; z < S; ++z) {      // fixed order: the result does not depend on which split finished last
                            const float* pz = base + (size_t)z * NA * BT * GEMM_BM;
                            a0 += __ldcg(pz + (size_t)(c * CH + j) * GEMM_BM + n_local);
                            if (NA == 2) a1 += __ldcg(pz + (size_t)(BT + c * CH + j) * GEMM_BM + n_local);
                        }
                        r0[j] = __float_as_uint(a0);
                        r1[j] = __float_as_uint(a1);
                    }
                    run_epilogue(c, r0, r1);
                }
                if (threadIdx.x == 64) p.ws_counters[tile] = 0;    // ready for the next launch
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        __syncwarp();
        tmem_dealloc(tmem_base, Cfg::TMEM_COLS);
    }
    if (p.epilogue == EPI_RS_PUSH_F32 && threadIdx.x == 64) {
        // every CTA's stores are ordered before its counter bump; the last CTA publishes this rank's epoch to all peers
        __threadfence_system();
        const unsigned total = gridDim.x * gridDim.y * gridDim.z;
        if (atomicAdd(p.coll.rs_done, 1u) == total - 1) {
            *p.coll.rs_done = 0;
            __threadfence_system();
            for (int pr = 0; pr < p.coll.rs_tp; ++pr)
                asm volatile("st.release.sys.global.u32 [%0], %1;" ::"l"(p.coll.rs_peer_flags[pr] + p.coll.rs_rank), "r"(sp_epoch(p.coll.step, p.coll.rs_epoch)) : "memory");
        }
    }
}

// ---------------------------------------------------------------------------------------------
// host side

// 2-D K-major tensor map: dims {K, rows}, row stride ld elements, box {64, box_rows}, 128B swizzle.
int make_tmap_2d(CUtensorMap* out, const void* base, int is_bf16, uint64_t rows, uint64_t K, uint64_t ld, uint32_t box_rows);

template <int BT, int NA, int AB_FMT, int WT = W_F16>
static int launch_gemm(const CUtensorMap& tw0, const CUtensorMap& tw1, const CUtensorMap& tx, const GemmParams& p,
                       int splits, cudaStream_t stream, const QWeight& qw0 = QWeight(), const QWeight& qw1 = QWeight()) {
    using Cfg = GemmCfg<BT, NA>;
    auto kern = gemm_tcgen05_kernel<BT, NA, AB_FMT, WT>;
    if (first_use_on_device((const void*)kern))
        DLP_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM_BYTES));
    dim3 grid((p.N + GEMM_BM - 1) / GEMM_BM, p.grp.tile_expert ? p.grp.max_tiles : (p.T + BT - 1) / BT, splits);
    kern<<<grid, 192, Cfg::SMEM_BYTES, stream>>>(tw0, tw1, tx, p, qw0, qw1);
    DLP_LAUNCH_CHECK();
    return 0;
}

// Split-K through the workspace for the epilogues that cannot reduce across CTAs themselves: skinny problems (decode batches,
// narrow tensor-parallel shards) have fewer 128-row tiles than the machine has SMs, and a CTA per tile streams its weight rows at
// a fraction of the HBM rate.  Workspace layout: 4096 tile counters (zero-initialised by the owner, self-resetting), then
// [tile][split][accumulator][BT][128] fp32 partials.
constexpr size_t GEMM_WS_COUNTERS = 4096;
static int auto_split_ws(int epilogue, int split_k, long tiles, int total_kb, int na, int bt, void* ws, size_t ws_bytes, GemmParams& p) {
    // Measured (profiles/r2_gemm_splitk_ab.txt): the fix-up pays for token tiles up to 32 (decode batches: +19 % at B = 8); for
    // prefill-sized tiles the serial reload of 128 x 256 partials costs more than the idle SMs (54 k -> 29 k tok/s at pp512), and
    // the residual-add epilogue reduces across CTAs with atomics at no extra cost.
    if (split_k > 0 || ws == nullptr || tiles <= 0 || tiles > (long)GEMM_WS_COUNTERS || bt > 32 || epilogue == EPI_ATOMIC_ADD_F32) return 1;
    static int enabled = -1;
    if (enabled < 0) { const char* e = getenv("DLP_GEMM_SPLITK"); enabled = (e && e[0] == '0') ? 0 : 1; }
    if (!enabled) return 1;
    int s = sm_count() / (int)tiles;
    if (s > 8) s = 8;
    while (s > 1 && total_kb / s < 4) --s;
    const size_t per = (size_t)na * bt * GEMM_BM * sizeof(float);
    while (s > 1 && GEMM_WS_COUNTERS * 4 + (size_t)tiles * s * per > ws_bytes) --s;
    if (s <= 1) return 1;
    p.ws_counters = reinterpret_cast<unsigned*>(ws);
    p.ws = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(ws) + GEMM_WS_COUNTERS * 4);
    return s;
}

}  // namespace dlp
