// Token mixers with a state of their own, and the small row kernels around them.
//
//   embed_rows           token rows of the embedding table -> fp32 residual stream
//   latent_write         latent of latent attention: RMS norm, then the paged latent cache; rotation of the key part behind it and of the queries
//   hgrn2_scan           gated linear recurrence over the tokens of every segment (layers_scan.cuh)
#include "layers_scan.cuh"

namespace dlp {

template <typename WT> __device__ __forceinline__ float ld_w(const WT* p) { return (float)*p; }

template <typename WT>
__global__ void __launch_bounds__(256) embed_rows_kernel(const WT* table, int ld, const int* ids, float* h, int E, int vocab, float scale) {
    pdl_wait();
    const int t = blockIdx.x;
    const int id = min(max(ids[t], 0), vocab - 1);
    for (int k = threadIdx.x; k < E; k += 256) h[(size_t)t * E + k] = ld_w(table + (size_t)id * ld + k) * scale;
    pdl_launch_dependents();
}
int embed_rows(const void* table, int ld, const int* ids, float* h, int E, int T, int vocab, float scale, int f32, cudaStream_t s) {
    DLP_REQUIRE(table && ids && h && E > 0 && T > 0 && ld >= E, "embed_rows: bad argument");
    if (f32) DLP_CHECK_CUDA(launch_pdl(embed_rows_kernel<float>, dim3(T), dim3(256), 0, s, (const float*)table, ld, ids, h, E, vocab, scale));
    else DLP_CHECK_CUDA(launch_pdl(embed_rows_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, s, (const __nv_bfloat16*)table, ld, ids, h, E, vocab, scale));
    return 0;
}

// x (u, v of pair i) turned by the pair's angle
__device__ __forceinline__ float2 turned(const float* x, int i, int rot, int adjacent, float2 cs, int& u, int& v) {
    u = adjacent ? 2 * i : i;
    v = adjacent ? 2 * i + 1 : i + rot / 2;
    return make_float2(x[u] * cs.x - x[v] * cs.y, x[v] * cs.x + x[u] * cs.y);
}
template <typename WT>
__global__ void __launch_bounds__(128) latent_write_kernel(const LatentRows a) {
    extern __shared__ __align__(16) uint8_t lw_smem[];
    float2* cs = reinterpret_cast<float2*>(lw_smem);       // [rot / 2]
    __shared__ float red[32];
    pdl_wait();
    const int t = blockIdx.x, np = a.rot / 2;
    const float* x = a.proj + (size_t)t * a.ldp;
    for (int i = threadIdx.x; i < np; i += 128) {
        float s, c;
        sincosf((float)a.pos[t] * a.inv_freq[i], &s, &c);
        cs[i] = make_float2(c * a.rot_scale, s * a.rot_scale);
    }
    const int parts = gridDim.y - 1;           // block 0: the cache row; the others: the queries (none: block 0 as well)
    if (blockIdx.y == 0) {
        float ss = 0.f;
        for (int k = threadIdx.x; k < a.R; k += 128) ss = fmaf(x[k], x[k], ss);
        const float rs = 1.f / sqrtf(block_sum(ss, red) / (float)a.R + a.eps);
        __syncthreads();
        const int sl = a.slot[t];
        if (sl >= 0) {
            WT* row = reinterpret_cast<WT*>(a.cache) + (size_t)sl * a.Rc;
            for (int k = threadIdx.x; k < a.Rc; k += 128)
                if (k < a.R || k >= a.R + a.rot) row[k] = (WT)(k < a.R ? x[k] * rs * a.w[k] : 0.f);
            for (int i = threadIdx.x; i < np; i += 128) {
                int u, v;
                const float2 y = turned(x + a.R, i, a.rot, a.adjacent, cs[i], u, v);
                row[a.R + u] = (WT)y.x;
                row[a.R + v] = (WT)y.y;
            }
        }
    }
    if (a.q != nullptr && (blockIdx.y > 0 || parts == 0)) {
        __syncthreads();
        float* q = a.q + (size_t)t * a.ldq + a.Dq - a.rot;
        const int n = a.H * np, part = parts > 0 ? blockIdx.y - 1 : 0, step = 128 * max(parts, 1);
#pragma unroll 4
        for (int j = part * 128 + threadIdx.x; j < n; j += step) {
            const int h = j / np, i = j - h * np;
            float* p = q + (size_t)h * a.Dq;
            int u, v;
            const float2 y = turned(p, i, a.rot, a.adjacent, cs[i], u, v);
            p[u] = y.x;
            p[v] = y.y;
        }
    }
    pdl_launch_dependents();
}
int latent_write(const LatentRows& a, int T, int f32, cudaStream_t s) {
    DLP_REQUIRE(a.proj && a.w && a.slot && a.cache && a.R > 0 && a.rot >= 0 && a.rot % 2 == 0 && a.Rc >= a.R + a.rot && T > 0, "latent_write: bad argument");
    DLP_REQUIRE(a.rot == 0 || (a.pos && a.inv_freq && a.rot <= 8192 && (!a.q || (a.H > 0 && a.Dq >= a.rot && a.ldq >= a.H * a.Dq))), "latent_write: rotation of %d columns", a.rot);
    const size_t smem = (size_t)(a.rot / 2) * 8;
    const int parts = a.q && a.rot > 0 && T <= 64 ? (a.H * (a.rot / 2) + 255) / 256 : 0;         // few tokens: blocks of their own for the queries
    const dim3 grid(T, 1 + (parts < 16 ? parts : 16));
    DLP_CHECK_CUDA(f32 ? launch_pdl(latent_write_kernel<float>, grid, dim3(128), smem, s, a) : launch_pdl(latent_write_kernel<__nv_bfloat16>, grid, dim3(128), smem, s, a));
    return 0;
}

// ---- HGRN2 -------------------------------------------------------------------------------------------------------
//   f = l + (1 - l) sigmoid(z),  S <- diag(f) S + (1 - f) v^T,  o = S^T silu(q)
// (gate: hgrn2_gate in layers.cuh)
__device__ __forceinline__ void scan_channel(const Hgrn2Args& a, int t, int h, int d, float& q, float& f, float& k) {
    const float* p = a.proj + (size_t)t * a.ldp + h * a.D + d;
    q = silu_exact(p[0]);
    hgrn2_gate(p[a.H * a.D] + a.fbias[h * a.D + d], a.lower[h * a.D + d], f, k);
}
__device__ __forceinline__ float scan_value(const Hgrn2Args& a, int t, int h, int c) { return a.proj[(size_t)t * a.ldp + 2 * a.H * a.D + h * a.V + c]; }
__device__ __forceinline__ float scan_out(const Hgrn2Args&, int, float o, float) { return o; }

int hgrn2_scan(const Hgrn2Args& a, cudaStream_t s) {
    DLP_REQUIRE(a.proj && a.fbias && a.lower, "hgrn2_scan: null argument");
    return recurrence_scan(a, "hgrn2_scan", s);
}

}  // namespace dlp
