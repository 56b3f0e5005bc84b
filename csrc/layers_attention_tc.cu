// Prompt portions of latent attention with keys and values expanded per head: the tcgen05 flash kernel of attention_tc.cuh on plain
// bf16 rows, and the row kernels that prepare them.
#include "attention_tc.cuh"
#include "layers.cuh"

namespace dlp {

__device__ int g_rows_error;     // a wait of the flash kernel ran into its limit since the library was loaded

int* flash_error_flag() {
    int* p = nullptr;
    const cudaError_t e = cudaGetSymbolAddress((void**)&p, g_rows_error);
    if (e != cudaSuccess) set_error("flash_error_flag: %s", cudaGetErrorString(e));
    return e == cudaSuccess ? p : nullptr;
}

// latent rows 0 .. S-1 of one request, out of its pages
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint4* cache, const int* bt, int page, int chunks, uint4* out) {
    pdl_wait();
    const int key = blockIdx.x;
    const uint4* src = cache + ((size_t)bt[key / page] * page + key % page) * chunks;
    for (int i = threadIdx.x; i < chunks; i += 128) out[(size_t)key * chunks + i] = src[i];
    pdl_launch_dependents();
}
// query columns of the projection -> bf16 rows with every head padded to Dp
__global__ void __launch_bounds__(256) head_rows_kernel(const float* x, int ldx, int D, int Dp, int H, __nv_bfloat16* out) {
    pdl_wait();
    const int t = blockIdx.x;
    for (int i = threadIdx.x; i < H * Dp; i += 256) {
        const int h = i / Dp, d = i - h * Dp;
        out[(size_t)t * H * Dp + i] = __float2bfloat16_rn(d < D ? x[(size_t)t * ldx + h * D + d] : 0.f);
    }
    pdl_launch_dependents();
}

int latent_gather(const void* cache, const int* bt, int page, int Rc, void* out, int S, cudaStream_t s) {
    DLP_REQUIRE(cache && bt && out && page > 0 && Rc % 8 == 0 && S > 0, "latent_gather: bad argument");
    DLP_CHECK_CUDA(launch_pdl(latent_gather_kernel, dim3(S), dim3(128), 0, s, (const uint4*)cache, bt, page, Rc / 8, (uint4*)out));
    return 0;
}
int head_rows(const float* x, int ldx, int D, int Dp, int H, void* out, int T, cudaStream_t s) {
    DLP_REQUIRE(x && out && D > 0 && Dp >= D && H > 0 && T > 0, "head_rows: bad argument");
    DLP_CHECK_CUDA(launch_pdl(head_rows_kernel, dim3(T), dim3(256), 0, s, x, ldx, D, Dp, H, (__nv_bfloat16*)out));
    return 0;
}

template <int D1, int D2>
static int launch_rows(const void* q, const void* k, const void* v, int ldkv, int S, FaParams p, cudaStream_t s) {
    using Cfg = FaCfg<D1, D2, FA_ROWS>;
    static_assert(Cfg::SMEM_BYTES <= 227 * 1024, "flash staging");
    CUtensorMap tq, tk, tv;
    int rc;
    if ((rc = make_tmap_2d(&tq, q, 1, (uint64_t)p.T, (uint64_t)p.Hq * D1, (uint64_t)p.Hq * D1, Cfg::BM))) return rc;
    if ((rc = make_tmap_2d(&tk, k, 1, (uint64_t)S, (uint64_t)p.Hkv * D1, (uint64_t)ldkv, Cfg::BN))) return rc;
    if ((rc = make_tmap_2d(&tv, v, 1, (uint64_t)S, (uint64_t)p.Hkv * D2, (uint64_t)ldkv, Cfg::BN))) return rc;
    auto kern = attn_prefill_tc_kernel<D1, D2, FA_ROWS>;
    if (first_use_on_device((const void*)kern)) DLP_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM_BYTES));
    kern<<<dim3((p.T + Cfg::BM - 1) / Cfg::BM, p.Hq), Cfg::THREADS, Cfg::SMEM_BYTES, s>>>(tq, tk, tv, p);
    DLP_LAUNCH_CHECK();
    return 0;
}

// q [T, H * Dp], kv rows [S, ldkv]: k at column 0 (H * Dp), v at column H * Dp (H * Vp); queries are rows pos0 .. pos0 + T - 1 of them and see the `window` rows up to their own
int rows_attention(const void* q, const void* kv, int ldkv, int S, int T, int pos0, int H, int Dp, int Vp, int V, int window, float scale, const float* gate, int ldg, void* out,
                   int ldo, cudaStream_t s) {
    DLP_REQUIRE(q && kv && out && T > 0 && pos0 >= 0 && S >= pos0 + T && H > 0 && V <= Vp && window >= 1, "rows_attention: bad argument");
    FaParams p;
    memset(&p, 0, sizeof(p));
    p.out = out; p.T = T; p.pos0 = pos0; p.Hq = H; p.Hkv = H; p.page_size = 128; p.max_pages = 1; p.ldo = ldo; p.gate = gate; p.ldg = ldg; p.V = V; p.scale = scale; p.window = window;
    if ((p.error = flash_error_flag()) == nullptr) return -1;
    const void* v = (const uint8_t*)kv + (size_t)H * Dp * 2;
    if (Dp == 64 && Vp == 64) return launch_rows<64, 64>(q, kv, v, ldkv, S, p, s);
    if (Dp == 64 && Vp == 128) return launch_rows<64, 128>(q, kv, v, ldkv, S, p, s);
    if (Dp == 128 && Vp == 64) return launch_rows<128, 64>(q, kv, v, ldkv, S, p, s);
    if (Dp == 128 && Vp == 128) return launch_rows<128, 128>(q, kv, v, ldkv, S, p, s);
    if (Dp == 192 && Vp == 64) return launch_rows<192, 64>(q, kv, v, ldkv, S, p, s);
    if (Dp == 192 && Vp == 128) return launch_rows<192, 128>(q, kv, v, ldkv, S, p, s);
    DLP_REQUIRE(false, "rows_attention: head sizes %d / %d", Dp, Vp);
}
// 0, or 1 when a wait of a flash kernel gave up since the last call (synchronises)
int rows_attention_error(int* flag) {
    DLP_CHECK_CUDA(cudaMemcpyFromSymbol(flag, g_rows_error, sizeof(int)));
    if (*flag) {
        const int zero = 0;
        DLP_CHECK_CUDA(cudaMemcpyToSymbol(g_rows_error, &zero, sizeof(int)));
    }
    return 0;
}

}  // namespace dlp
