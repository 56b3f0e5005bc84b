// Flash-prefill over the paged fp16 cache (kernel: attention_tc.cuh).
#include "attention_tc.cuh"

namespace dlp {

template <int D>
static int launch_fa(const __half* q, const __half* kc, const __half* vc, const FaParams& p, int n_pages, cudaStream_t s) {
    using Cfg = FaCfg<D, D, FA_PAGED>;
    CUtensorMap tq, tk, tv;
    int rc;
    if ((rc = make_tmap_2d(&tq, q, 0, (uint64_t)p.T, (uint64_t)p.Hq * D, (uint64_t)p.Hq * D, Cfg::BM))) return rc;
    const uint64_t rows = (uint64_t)n_pages * p.Hkv * p.page_size;
    if ((rc = make_tmap_2d(&tk, kc, 0, rows, D, D, (uint32_t)p.page_size))) return rc;
    if ((rc = make_tmap_2d(&tv, vc, 0, rows, D, D, (uint32_t)p.page_size))) return rc;
    auto kern = attn_prefill_tc_kernel<D, D, FA_PAGED>;
    if (first_use_on_device((const void*)kern))
        DLP_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM_BYTES));
    dim3 grid((p.T + Cfg::BM - 1) / Cfg::BM, p.Hq);
    kern<<<grid, Cfg::THREADS, Cfg::SMEM_BYTES, s>>>(tq, tk, tv, p);
    DLP_LAUNCH_CHECK();
    return 0;
}

int attn_prefill_tc(const __half* q, const __half* kc, const __half* vc, const int* bt_row, __half* out, int T, int pos0, int Hq, int Hkv,
                    int D, int page_size, int n_pages, int max_pages, cudaStream_t s) {
    DLP_REQUIRE(T > 0 && Hq % Hkv == 0 && n_pages > 0 && max_pages > 0, "attn_prefill_tc: bad shape");
    DLP_REQUIRE(page_size % 8 == 0 && page_size <= 128 && 128 % page_size == 0, "attn_prefill_tc: page size %d (multiple of 8 that divides 128)", page_size);
    FaParams p;
    memset(&p, 0, sizeof(p));
    p.bt_row = bt_row; p.out = out; p.T = T; p.pos0 = pos0; p.Hq = Hq; p.Hkv = Hkv; p.page_size = page_size; p.max_pages = max_pages;
    p.ldo = Hq * D;
    if (D == 128) return launch_fa<128>(q, kc, vc, p, n_pages, s);
    if (D == 64) return launch_fa<64>(q, kc, vc, p, n_pages, s);
    DLP_REQUIRE(false, "attn_prefill_tc: head dim %d unsupported (64, 128)", D);
}

}  // namespace dlp
