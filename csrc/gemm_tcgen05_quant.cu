// tcgen05 GEMM with the block-quant decode fused into the A-operand producer (kernel: gemm_tcgen05.cuh).
#include "gemm_tcgen05.cuh"

namespace dlp {

// Y[T,N] (op)= X[T,K] . dequant(W)[N,K]^T with the block-quant decode fused into the A-operand producer.
int gemm_quant(const QWeight& w0, const QWeight* w1, int wtype, const void* x, int ldx, void* y, int ldy, int T, int epilogue,
               int split_k, cudaStream_t stream, const GemmCollective* coll, const GemmGroup* grp, void* ws, size_t ws_bytes) {
    // grouped: w0 / w1 describe the stack of all experts (w0.N = n_expert * rows_per_expert); one expert's width tiles the grid
    const int N = grp ? grp->rows_per_expert : w0.N, K = w0.K;
    DLP_REQUIRE(T > 0 && N > 0 && K > 0 && K % 256 == 0, "gemm_quant: bad problem T=%d N=%d K=%d", T, N, K);
    DLP_REQUIRE(grp == nullptr || (grp->tile_expert && grp->tile_row0 && grp->tile_rows && grp->n_tiles && grp->max_tiles > 0 && split_k <= 1 &&
                                   epilogue != EPI_RS_PUSH_F32 && epilogue != EPI_ATOMIC_ADD_F32 && w0.N == grp->rows_per_expert * grp->n_expert),
                "gemm_quant: bad grouped descriptor");
    const int na = (epilogue == EPI_SWIGLU_F16) ? 2 : 1;
    DLP_REQUIRE(na == 1 || w1 != nullptr, "gemm_quant: SwiGLU epilogue needs the up-projection weight");
    const int total_kb = K / GEMM_BK;
    int splits = split_k;
    if (splits <= 0) {
        splits = 1;
        if (epilogue == EPI_ATOMIC_ADD_F32) {
            const int bt_guess = T <= 16 ? 16 : T <= 32 ? 32 : T <= 64 ? 64 : T <= 128 ? 128 : 256;
            const long tiles = (long)((N + GEMM_BM - 1) / GEMM_BM) * ((T + bt_guess - 1) / bt_guess);
            const int sms = sm_count();
            while (tiles * splits * 2 <= sms && total_kb / (splits * 2) >= 8) splits *= 2;
        }
    }
    DLP_REQUIRE(splits == 1 || epilogue == EPI_ATOMIC_ADD_F32, "gemm_quant: split-K needs the atomic-add epilogue or a workspace");
    if (splits > total_kb) splits = total_kb;
    GemmParams p;
    memset(&p, 0, sizeof(p));
    if (coll) p.coll = *coll;
    DLP_REQUIRE(epilogue != EPI_RS_PUSH_F32 || (coll && coll->rs_rows > 0 && coll->rs_done && coll->rs_tp >= 1 && coll->rs_tp <= 8 && splits == 1),
                "gemm: the reduce-scatter epilogue needs a collective descriptor and no atomic split-K");
    p.y = y; p.T = T; p.N = N; p.K = K; p.ldy = ldy; p.epilogue = epilogue;
    if (grp) p.grp = *grp;
    const int bt = grp ? grp->bt : (T <= 16 ? 16 : T <= 32 ? 32 : T <= 64 ? 64 : T <= 128 ? 128 : 256);
    if (splits == 1)
        splits = auto_split_ws(epilogue, split_k, (long)((N + GEMM_BM - 1) / GEMM_BM) * (grp ? grp->max_tiles : (T + bt - 1) / bt), total_kb, na, bt,
                               ws, ws_bytes, p);
    p.k_blocks_per_split = (total_kb + splits - 1) / splits;
    splits = (total_kb + p.k_blocks_per_split - 1) / p.k_blocks_per_split;
    if (splits == 1) { p.ws = nullptr; p.ws_counters = nullptr; }
    CUtensorMap tx;
    int rc;
    if ((rc = make_tmap_2d(&tx, x, 0, T, K, ldx, bt))) return rc;
    const QWeight up = w1 ? *w1 : QWeight();
#define DLP_QG_BT(WT_, BT_)                                                                                   \
    case BT_:                                                                                                 \
        return na == 2 ? launch_gemm<BT_, 2, 0, WT_>(tx, tx, tx, p, splits, stream, w0, up)                   \
                       : launch_gemm<BT_, 1, 0, WT_>(tx, tx, tx, p, splits, stream, w0, up);
#define DLP_QG_TYPE(WT_)                                                                                      \
    case WT_:                                                                                                 \
        switch (bt) { DLP_QG_BT(WT_, 16) DLP_QG_BT(WT_, 32) DLP_QG_BT(WT_, 64) DLP_QG_BT(WT_, 128) DLP_QG_BT(WT_, 256) } \
        break;
    switch (wtype) {
        DLP_QG_TYPE(W_Q8_0)
        DLP_QG_TYPE(W_Q4_K)
        DLP_QG_TYPE(W_Q5_K)
        DLP_QG_TYPE(W_Q6_K)
    }
#undef DLP_QG_TYPE
#undef DLP_QG_BT
    DLP_REQUIRE(false, "gemm_quant: unsupported weight type %d", wtype);
}

}  // namespace dlp
