// Token mixers with a state of their own, and the small row kernels around them.
//
//   embed_rows           token rows of the embedding table -> fp32 residual stream
//   latent_write         latent of latent attention: RMS norm, then the paged latent cache
//   hgrn2_scan           gated linear recurrence over the tokens of every segment (prompt portions and decode steps alike): the fp32
//                        state lives in registers for the whole segment
#include "layers.cuh"

namespace dlp {

template <typename WT> __device__ __forceinline__ float ld_w(const WT* p) { return (float)*p; }

template <typename WT>
__global__ void __launch_bounds__(256) embed_rows_kernel(const WT* table, int ld, const int* ids, float* h, int E, int vocab) {
    pdl_wait();
    const int t = blockIdx.x;
    const int id = min(max(ids[t], 0), vocab - 1);
    for (int k = threadIdx.x; k < E; k += 256) h[(size_t)t * E + k] = ld_w(table + (size_t)id * ld + k);
    pdl_launch_dependents();
}
int embed_rows(const void* table, int ld, const int* ids, float* h, int E, int T, int vocab, int f32, cudaStream_t s) {
    DLP_REQUIRE(table && ids && h && E > 0 && T > 0 && ld >= E, "embed_rows: bad argument");
    if (f32) DLP_CHECK_CUDA(launch_pdl(embed_rows_kernel<float>, dim3(T), dim3(256), 0, s, (const float*)table, ld, ids, h, E, vocab));
    else DLP_CHECK_CUDA(launch_pdl(embed_rows_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, s, (const __nv_bfloat16*)table, ld, ids, h, E, vocab));
    return 0;
}

template <typename WT>
__global__ void __launch_bounds__(128) latent_write_kernel(const float* proj, int ldp, const float* w, float eps, int R, int Rc, const int* slot, WT* cache) {
    __shared__ float red[32];
    pdl_wait();
    const int t = blockIdx.x;
    const float* x = proj + (size_t)t * ldp;
    float a = 0.f;
    for (int k = threadIdx.x; k < R; k += 128) a = fmaf(x[k], x[k], a);
    const float rs = 1.f / sqrtf(block_sum(a, red) / (float)R + eps);
    const int sl = slot[t];
    if (sl >= 0)
        for (int k = threadIdx.x; k < Rc; k += 128) cache[(size_t)sl * Rc + k] = (WT)(k < R ? x[k] * rs * w[k] : 0.f);
    pdl_launch_dependents();
}
int latent_write(const float* proj, int ldp, const float* w, float eps, int R, int Rc, const int* slot, void* cache, int T, int f32, cudaStream_t s) {
    DLP_REQUIRE(proj && w && slot && cache && R > 0 && Rc >= R && T > 0, "latent_write: bad argument");
    if (f32) DLP_CHECK_CUDA(launch_pdl(latent_write_kernel<float>, dim3(T), dim3(128), 0, s, proj, ldp, w, eps, R, Rc, slot, (float*)cache));
    else DLP_CHECK_CUDA(launch_pdl(latent_write_kernel<__nv_bfloat16>, dim3(T), dim3(128), 0, s, proj, ldp, w, eps, R, Rc, slot, (__nv_bfloat16*)cache));
    return 0;
}

// ---- HGRN2 -------------------------------------------------------------------------------------------------------
//   f = l + (1 - l) sigmoid(z),  S <- diag(f) S + (1 - f) v^T,  o = S^T silu(q)
// (gate: hgrn2_gate in layers.cuh)

// One CTA = one (segment, head, slice of 128 / RG value columns); a thread keeps RPT state rows of one column.  Tokens are staged
// CT at a time; a row group's values sit RPT + 4 floats apart so that the RG groups of a warp read different banks.
template <int RG, int RPT>
__global__ void __launch_bounds__(128) hgrn2_scan_kernel(const Hgrn2Args a) {
    constexpr int COLS = 128 / RG, ROWS = RG * RPT, CT = 2048 / ROWS > 16 ? 16 : (2048 / ROWS < 2 ? 2 : 2048 / ROWS), GS = RPT + 4;
    extern __shared__ __align__(16) float hg_smem[];
    float* sq = hg_smem;                        // [CT][RG * GS]
    float* sf = sq + CT * RG * GS;
    float* sk = sf + CT * RG * GS;
    float* sv = sk + CT * RG * GS;              // [CT][COLS]
    const int tid = threadIdx.x, rg = tid % RG, col = tid / RG;
    const int seg = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * COLS;
    const int HD = a.H * a.D;
    pdl_wait();
    const int lo = a.seg[2 * seg], hi = a.seg[2 * seg + 1];
    if (lo >= hi) return;
    float S[RPT];
    float* st = a.state + (((size_t)a.seg_slot[seg] * a.H + h) * a.D + rg * RPT) * a.V + v0 + col;
    const bool col_ok = v0 + col < a.V;
    const bool fresh = a.pos[lo] == 0;
#pragma unroll
    for (int i = 0; i < RPT; ++i) S[i] = (!fresh && col_ok && rg * RPT + i < a.D) ? st[(size_t)i * a.V] : 0.f;
    for (int t0 = lo; t0 < hi; t0 += CT) {
        const int n = min(CT, hi - t0);
        __syncthreads();
        for (int i = tid; i < n * ROWS; i += 128) {
            const int t = i / ROWS, d = i - t * ROWS, o = t * RG * GS + (d / RPT) * GS + d % RPT;
            float q = 0.f, f = 1.f, k = 0.f;
            if (d < a.D) {
                const float* p = a.proj + (size_t)(t0 + t) * a.ldp + h * a.D + d;
                q = silu_exact(p[0]);
                hgrn2_gate(p[HD] + a.fbias[h * a.D + d], a.lower[h * a.D + d], f, k);
            }
            sq[o] = q;
            sf[o] = f;
            sk[o] = k;
        }
        for (int i = tid; i < n * COLS; i += 128) {
            const int t = i / COLS, c = i - t * COLS;
            sv[i] = v0 + c < a.V ? a.proj[(size_t)(t0 + t) * a.ldp + 2 * HD + h * a.V + v0 + c] : 0.f;
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float v = sv[t * COLS + col];
            const float4* q4 = reinterpret_cast<const float4*>(sq + t * RG * GS + rg * GS);
            const float4* f4 = reinterpret_cast<const float4*>(sf + t * RG * GS + rg * GS);
            const float4* k4 = reinterpret_cast<const float4*>(sk + t * RG * GS + rg * GS);
            float o0 = 0.f, o1 = 0.f;
#pragma unroll
            for (int i = 0; i < RPT / 4; ++i) {
                const float4 q = q4[i], f = f4[i], k = k4[i];
                S[4 * i] = fmaf(f.x, S[4 * i], k.x * v);
                S[4 * i + 1] = fmaf(f.y, S[4 * i + 1], k.y * v);
                S[4 * i + 2] = fmaf(f.z, S[4 * i + 2], k.z * v);
                S[4 * i + 3] = fmaf(f.w, S[4 * i + 3], k.w * v);
                o0 = fmaf(q.x, S[4 * i], o0);
                o1 = fmaf(q.y, S[4 * i + 1], o1);
                o0 = fmaf(q.z, S[4 * i + 2], o0);
                o1 = fmaf(q.w, S[4 * i + 3], o1);
            }
            float o = o0 + o1;
#pragma unroll
            for (int x = 1; x < RG; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
            if (rg == 0 && col_ok) a.out[(size_t)(t0 + t) * a.ldo + h * a.V + v0 + col] = o;
        }
    }
    pdl_launch_dependents();
#pragma unroll
    for (int i = 0; i < RPT; ++i)
        if (col_ok && rg * RPT + i < a.D) st[(size_t)i * a.V] = S[i];
}

template <int RG, int RPT>
static int launch_scan(const Hgrn2Args& a, cudaStream_t s) {
    constexpr int COLS = 128 / RG, ROWS = RG * RPT, CT = 2048 / ROWS > 16 ? 16 : (2048 / ROWS < 2 ? 2 : 2048 / ROWS);
    constexpr size_t smem = (size_t)CT * (3 * RG * (RPT + 4) + COLS) * 4;
    static_assert(smem <= 48 * 1024, "scan staging");
    DLP_CHECK_CUDA(launch_pdl(hgrn2_scan_kernel<RG, RPT>, dim3((a.V + COLS - 1) / COLS, a.H, a.n_seg), dim3(128), smem, s, a));
    return 0;
}

int hgrn2_scan(const Hgrn2Args& a, cudaStream_t s) {
    DLP_REQUIRE(a.proj && a.fbias && a.lower && a.state && a.seg && a.seg_slot && a.pos && a.out, "hgrn2_scan: null argument");
    DLP_REQUIRE(a.H > 0 && a.D > 0 && a.V > 0 && a.n_seg > 0 && a.n_seg <= 65535, "hgrn2_scan: bad shape");
    if (a.D <= 64) return launch_scan<4, 16>(a, s);
    if (a.D <= 128) return launch_scan<4, 32>(a, s);
    if (a.D <= 256) return launch_scan<8, 32>(a, s);
    DLP_REQUIRE(a.D <= 1024, "hgrn2_scan: %d channels per head (at most 1024)", a.D);
    return launch_scan<16, 64>(a, s);
}

}  // namespace dlp
