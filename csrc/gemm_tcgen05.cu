// tcgen05 GEMM, dense fp16 / bf16 operands (kernel: gemm_tcgen05.cuh).
#include "gemm_tcgen05.cuh"

namespace dlp {

typedef CUresult (*PFN_encodeTiled)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                    const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                    CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static PFN_encodeTiled get_encode_fn() {
    static PFN_encodeTiled fn = nullptr;
    if (!fn) {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult qres;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &qres) == cudaSuccess &&
            qres == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<PFN_encodeTiled>(p);
    }
    return fn;
}

// 2-D K-major tensor map: dims {K, rows}, row stride ld elements, box {64, box_rows}, 128B swizzle.
int make_tmap_2d(CUtensorMap* out, const void* base, int is_bf16, uint64_t rows, uint64_t K, uint64_t ld, uint32_t box_rows) {
    PFN_encodeTiled enc = get_encode_fn();
    DLP_REQUIRE(enc != nullptr, "cuTensorMapEncodeTiled entry point unavailable (no CUDA driver?)");
    DLP_REQUIRE((reinterpret_cast<uintptr_t>(base) & 15) == 0, "TMA base pointer must be 16-byte aligned");
    DLP_REQUIRE((ld * 2) % 16 == 0, "TMA row stride must be a multiple of 16 bytes (ld=%llu)", (unsigned long long)ld);
    cuuint64_t dims[2] = {K, rows};
    cuuint64_t strides[1] = {ld * 2};
    cuuint32_t box[2] = {GEMM_BK, box_rows};
    cuuint32_t estr[2] = {1, 1};
    CUresult r = enc(out, is_bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 2,
                     const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                     CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    DLP_REQUIRE(r == CUDA_SUCCESS, "cuTensorMapEncodeTiled failed with CUresult %d", (int)r);
    return 0;
}

// Y[T,N] (op)= X[T,K] . W0[N,K]^T  (and W1 for SwiGLU).  X/W are fp16 (is_bf16=0) or bf16 (is_bf16=1).
int gemm_f16(const void* w0, const void* w1, int ldw, const void* x, int ldx, void* y, int ldy, int T, int N, int K,
             int epilogue, int is_bf16, int split_k, cudaStream_t stream, const GemmCollective* coll, const GemmGroup* grp, void* ws,
             size_t ws_bytes, const OutTail* tail) {
    // grouped: N = output features of ONE expert, w0/w1 = stacks of all experts (rows_total = what the tensor map must cover)
    DLP_REQUIRE(T > 0 && N > 0 && K > 0, "gemm: empty problem T=%d N=%d K=%d", T, N, K);
    DLP_REQUIRE(grp == nullptr || (grp->tile_expert && grp->tile_row0 && grp->tile_rows && grp->n_tiles && grp->max_tiles > 0 && split_k <= 1 &&
                                   epilogue != EPI_RS_PUSH_F32 && epilogue != EPI_ATOMIC_ADD_F32), "gemm: bad grouped descriptor");
    if (grp && split_k == 1) { ws = nullptr; ws_bytes = 0; }
    DLP_REQUIRE(K % 8 == 0, "gemm: K=%d must be a multiple of 8", K);
    const int na = epi_is_gated(epilogue) ? 2 : 1;
    DLP_REQUIRE(na == 1 || w1 != nullptr, "gemm: a gated epilogue needs the up-projection weight");
    DLP_REQUIRE((epilogue != EPI_GEGLU_BF16 && epilogue != EPI_SWIGLU_BF16 && epilogue != EPI_RELU2_BF16 && epilogue != EPI_TAIL_BF16) || is_bf16, "gemm: the bf16 epilogues are built for bf16 operands");
    const int total_kb = (K + GEMM_BK - 1) / GEMM_BK;
    int splits = split_k;
    if (splits <= 0) {  // auto: fill the machine when the epilogue can reduce across CTAs
        splits = 1;
        if (epilogue == EPI_ATOMIC_ADD_F32) {
            const int bt_guess = T <= 16 ? 16 : T <= 32 ? 32 : T <= 64 ? 64 : T <= 128 ? 128 : 256;
            const long tiles = (long)((N + GEMM_BM - 1) / GEMM_BM) * ((T + bt_guess - 1) / bt_guess);
            const int sms = sm_count();
            while (tiles * splits * 2 <= sms && total_kb / (splits * 2) >= 8) splits *= 2;
        }
    }
    DLP_REQUIRE(splits == 1 || epilogue == EPI_ATOMIC_ADD_F32, "gemm: split-K needs the atomic-add epilogue or a workspace");
    if (splits > total_kb) splits = total_kb;
    GemmParams p;
    memset(&p, 0, sizeof(p));
    if (coll) p.coll = *coll;
    DLP_REQUIRE((epilogue == EPI_TAIL_BF16) == (tail != nullptr) && (!tail || grp == nullptr), "gemm: what follows the sums and the epilogue do not fit");
    if (tail) p.tail = *tail;
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

    DLP_REQUIRE(bt == 16 || bt == 32 || bt == 64 || bt == 128 || bt == 256, "gemm: token tile %d", bt);
    const uint64_t w_rows = grp ? (uint64_t)grp->rows_per_expert * grp->n_expert : (uint64_t)N;   // grouped: the map spans the whole stack
    CUtensorMap tw0, tw1, tx;
    int rc;
    if ((rc = make_tmap_2d(&tw0, w0, is_bf16, w_rows, K, ldw, GEMM_BM))) return rc;
    tw1 = tw0;
    if (na == 2 && (rc = make_tmap_2d(&tw1, w1, is_bf16, w_rows, K, ldw, GEMM_BM))) return rc;
    if ((rc = make_tmap_2d(&tx, x, is_bf16, T, K, ldx, bt))) return rc;

#ifdef DLP_LAYERS_ONLY      // the library of the layer-list models holds the bf16 form only
    DLP_REQUIRE(is_bf16, "gemm: fp16 operands are not part of this build");
#define DLP_GEMM_CASE(BT_)                                                                         \
    case BT_:                                                                                      \
        if (na == 2) return launch_gemm<BT_, 2, 1>(tw0, tw1, tx, p, splits, stream);               \
        return launch_gemm<BT_, 1, 1>(tw0, tw1, tx, p, splits, stream);
#else
#define DLP_GEMM_CASE(BT_)                                                                         \
    case BT_:                                                                                      \
        if (na == 2) return is_bf16 ? launch_gemm<BT_, 2, 1>(tw0, tw1, tx, p, splits, stream)      \
                                    : launch_gemm<BT_, 2, 0>(tw0, tw1, tx, p, splits, stream);     \
        return is_bf16 ? launch_gemm<BT_, 1, 1>(tw0, tw1, tx, p, splits, stream)                   \
                       : launch_gemm<BT_, 1, 0>(tw0, tw1, tx, p, splits, stream);
#endif
    switch (bt) {
        DLP_GEMM_CASE(16)
        DLP_GEMM_CASE(32)
        DLP_GEMM_CASE(64)
        DLP_GEMM_CASE(128)
        DLP_GEMM_CASE(256)
    }
#undef DLP_GEMM_CASE
    return -1;
}

}  // namespace dlp
