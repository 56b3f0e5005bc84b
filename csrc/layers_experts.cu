// Routed experts of layer-list models.
//
//   expert_matvec_kernel  decode (1..4 rows): the chosen experts' matrices streamed once; routing and the norm in the prologue, the
//                         squared ReLU / the weighted sum over the experts in the epilogue
//   route_kernel          the same routing as one launch, in front of the grouped products (moe.cu builds the expert-sorted order)
#include "layers_rows.cuh"

namespace dlp {

// Every block routes the rows itself (a warp per row) from the router's logits.  DOWN = 0: x is one row per token, a unit is two
// rows of one chosen expert's matrix, the output row of assignment (t, j) is max(., 0)^2.  DOWN = 1: x is one row per assignment, a
// unit is a pair of output rows for one assignment, and the weighted sum over a token's experts is formed behind the units, in
// the order of the choice.
template <typename WT, bool DOWN, int U>
__global__ void __launch_bounds__(512, 1) expert_matvec_kernel(const RowStage st, const ExpertArgs a, void* out, int ldo, int T) {
    constexpr int VEC = Act<WT>::VEC, COLS = 32 * VEC * U;
    extern __shared__ __align__(16) uint8_t mv_smem[];
    __shared__ int s_id[4 * ROUTE_MAX_TOP];
    __shared__ float s_w[4 * ROUTE_MAX_TOP];
    const int K = st.Kp, A = T * a.top, xrows = DOWN ? A : T;
    WT* xs = reinterpret_cast<WT*>(mv_smem);
    float* sums = reinterpret_cast<float*>(mv_smem + (((size_t)xrows * K * sizeof(WT) + 15) & ~size_t(15)));
    const WT* w = reinterpret_cast<const WT*>(a.w);
    const int KC = (K + COLS - 1) / COLS;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int ppe = (a.rows + 1) / 2;                                   // row pairs of one expert
    const int pairs = DOWN ? ppe : A * ppe, upp = DOWN ? A * KC : KC;   // pairs of the launch, units of a pair
    const int p_lo = (int)((long long)pairs * blockIdx.x / gridDim.x), p_hi = (int)((long long)pairs * (blockIdx.x + 1) / gridDim.x);
    const int units = (p_hi - p_lo) * upp;
    pdl_wait();
    if (warp < T) route_row(a.logits + (size_t)warp * a.ldl, a.bias, a.n_expert, a.top, s_id + warp * a.top, s_w + warp * a.top);
    if (DOWN) {
        for (int i = threadIdx.x; i < A * (K / VEC); i += blockDim.x) {
            const int r = i / (K / VEC), c = i - r * (K / VEC);
            *reinterpret_cast<uint4*>(xs + (size_t)r * K + c * VEC) = *reinterpret_cast<const uint4*>(reinterpret_cast<const WT*>(st.x) + (size_t)r * st.ldx + c * VEC);
        }
        __syncthreads();
    } else {
        stage_rows_dev<WT, true>(st, 0, T, sums, false, xs, K);
    }
    float* part = sums;                  // [units][2]
    uint4 buf[2][2][U];
    auto where = [&](int u, int& as, int& row, int& c) {                // assignment, first row of the pair, column chunk
        const int pr = u / upp, rest = u - pr * upp;
        as = DOWN ? rest / KC : (p_lo + pr) / ppe;
        row = (DOWN ? p_lo + pr : (p_lo + pr) % ppe) * 2;
        c = DOWN ? rest % KC : rest;
    };
    auto issue = [&](int u, int b) {
        int as, row, c;
        where(u, as, row, c);
        const WT* e0 = w + (size_t)s_id[as] * a.rows * a.ldw + c * COLS + lane * VEC;
        const WT* r0 = e0 + (size_t)row * a.ldw;
        const WT* r1 = e0 + (size_t)min(row + 1, a.rows - 1) * a.ldw;
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const bool ok = c * COLS + i * 32 * VEC + lane * VEC < K;
            buf[b][0][i] = ok ? ldg_nc_v4(r0 + i * 32 * VEC) : make_uint4(0, 0, 0, 0);
            buf[b][1][i] = ok ? ldg_nc_v4(r1 + i * 32 * VEC) : make_uint4(0, 0, 0, 0);
        }
    };
    auto reduce = [&](int u, int b) {
        int as, row, c;
        where(u, as, row, c);
        const WT* x = xs + (size_t)(DOWN ? as : as / a.top) * K;
        float acc[2] = {0.f, 0.f};
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const int k = c * COLS + i * 32 * VEC + lane * VEC;
            if (k < K) {
                const uint4 xv = *reinterpret_cast<const uint4*>(x + k);
                const uint32_t xw[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
                for (int m = 0; m < 2; ++m) {
                    const uint32_t ww[4] = {buf[b][m][i].x, buf[b][m][i].y, buf[b][m][i].z, buf[b][m][i].w};
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        if (VEC == 8) {
                            const float2 f = bf2_to_f2(ww[j]), g = bf2_to_f2(xw[j]);
                            acc[m] = fmaf(f.x, g.x, acc[m]);
                            acc[m] = fmaf(f.y, g.y, acc[m]);
                        } else {
                            acc[m] = fmaf(__uint_as_float(ww[j]), __uint_as_float(xw[j]), acc[m]);
                        }
                    }
                }
            }
        }
        const float v0 = warp_sum(acc[0]), v1 = warp_sum(acc[1]);
        if (lane == 0) *reinterpret_cast<float2*>(part + (size_t)u * 2) = make_float2(v0, v1);
    };
    int u = warp;
    if (u < units) issue(u, 0);
    while (u < units) {
        if (u + nw < units) issue(u + nw, 1);
        reduce(u, 0);
        u += nw;
        if (u >= units) break;
        if (u + nw < units) issue(u + nw, 0);
        reduce(u, 1);
        u += nw;
    }
    pdl_launch_dependents();
    __syncthreads();
    const int np = p_hi - p_lo;
    if (DOWN) {
        for (int i = threadIdx.x; i < np * 2 * T; i += blockDim.x) {
            const int t = i / (np * 2), r = i - t * np * 2, row = p_lo * 2 + r;
            if (row >= a.rows) continue;
            float v = 0.f;
            for (int j = 0; j < a.top; ++j) {
                float s = 0.f;
                for (int c = 0; c < KC; ++c) s += part[((size_t)(r >> 1) * upp + (t * a.top + j) * KC + c) * 2 + (r & 1)];
                v = fmaf(s_w[t * a.top + j], s, v);
            }
            reinterpret_cast<float*>(out)[(size_t)t * ldo + row] = v;
        }
    } else {
        for (int i = threadIdx.x; i < np * 2; i += blockDim.x) {
            const int pr = p_lo + (i >> 1), as = pr / ppe, row = (pr - as * ppe) * 2 + (i & 1);
            if (row >= a.rows) continue;
            float v = 0.f;
            for (int c = 0; c < KC; ++c) v += part[((size_t)(i >> 1) * KC + c) * 2 + (i & 1)];
            v = fmaxf(v, 0.f);
            reinterpret_cast<WT*>(out)[(size_t)as * ldo + row] = Act<WT>::from_f(v * v);
        }
    }
}

template <typename WT, bool DOWN, int U>
static int launch_expert(const RowStage& st, const ExpertArgs& a, void* out, int ldo, int T, cudaStream_t s) {
    constexpr int COLS = 32 * Act<WT>::VEC * U;
    const int A = T * a.top, ppe = (a.rows + 1) / 2, pairs = DOWN ? ppe : A * ppe, KC = (st.Kp + COLS - 1) / COLS;
    const int grid = pairs < sm_count() ? pairs : sm_count();
    const size_t xbytes = ((size_t)(DOWN ? A : T) * st.Kp * sizeof(WT) + 15) & ~size_t(15);
    const size_t part = (size_t)((pairs + grid - 1) / grid) * (DOWN ? A * KC : KC) * 2 * 4, stg = DOWN ? 0 : stage_bytes(st, T, 16);
    const size_t smem = xbytes + (part > stg ? part : stg);
    DLP_REQUIRE(smem <= 220 * 1024, "expert_matvec: %d rows of width %d need %zu bytes of shared memory", DOWN ? A : T, st.Kp, smem);
    auto kern = expert_matvec_kernel<WT, DOWN, U>;
    if (first_use_on_device((const void*)kern)) DLP_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    DLP_CHECK_CUDA(launch_pdl(kern, dim3(grid), dim3(512), smem, s, st, a, out, ldo, T));
    return 0;
}
template <typename WT, bool DOWN>
static int launch_expert_u(const RowStage& st, const ExpertArgs& a, void* out, int ldo, int T, cudaStream_t s) {
    const int chunks = (st.Kp + 32 * Act<WT>::VEC - 1) / (32 * Act<WT>::VEC);       // the widest unit that its columns fill
    if (chunks >= 3) return launch_expert<WT, DOWN, 4>(st, a, out, ldo, T, s);
    if (chunks == 2) return launch_expert<WT, DOWN, 2>(st, a, out, ldo, T, s);
    return launch_expert<WT, DOWN, 1>(st, a, out, ldo, T, s);
}

int expert_matvec(const RowStage& st, const ExpertArgs& a, void* out, int ldo, int down, int T, int f32, cudaStream_t s) {
    int rc = check_stage(st, "expert_matvec");
    if (rc) return rc;
    DLP_REQUIRE(a.logits && a.w && out && a.rows > 0 && T >= 1 && T <= 4, "expert_matvec: bad argument (T=%d)", T);
    DLP_REQUIRE(a.n_expert >= 1 && a.n_expert <= ROUTE_MAX_EXPERTS && a.top >= 1 && a.top <= a.n_expert && a.top <= ROUTE_MAX_TOP, "expert_matvec: %d of %d experts", a.top,
                a.n_expert);
    DLP_REQUIRE(st.Kp % 8 == 0 && a.ldw % 8 == 0 && a.ldw >= st.Kp && !st.h_out, "expert_matvec: row length %d / stride %d must be multiples of 8", st.Kp, a.ldw);
    DLP_REQUIRE(!down || (st.x_f32 == (f32 != 0) && !st.y && !st.e && !st.w2 && st.ldx % 8 == 0), "expert_matvec: the down product takes activation rows as they are");
    if (f32) return down ? launch_expert_u<float, true>(st, a, out, ldo, T, s) : launch_expert_u<float, false>(st, a, out, ldo, T, s);
    return down ? launch_expert_u<__nv_bfloat16, true>(st, a, out, ldo, T, s) : launch_expert_u<__nv_bfloat16, false>(st, a, out, ldo, T, s);
}

__global__ void __launch_bounds__(128) route_kernel(const float* logits, int ld, const float* bias, int n_expert, int top, int* ids, float* w, int T) {
    pdl_wait();
    const int t = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (t < T) route_row(logits + (size_t)t * ld, bias, n_expert, top, ids + (size_t)t * top, w + (size_t)t * top);
    pdl_launch_dependents();
}
int route(const float* logits, int ld, const float* bias, int n_expert, int top, int* ids, float* w, int T, cudaStream_t s) {
    DLP_REQUIRE(logits && ids && w && T > 0 && ld >= n_expert, "route: bad argument");
    DLP_REQUIRE(n_expert >= 1 && n_expert <= ROUTE_MAX_EXPERTS && top >= 1 && top <= n_expert && top <= ROUTE_MAX_TOP, "route: %d of %d experts (at most %d of %d)", top, n_expert,
                ROUTE_MAX_TOP, ROUTE_MAX_EXPERTS);
    DLP_CHECK_CUDA(launch_pdl(route_kernel, dim3((T + 3) / 4), dim3(128), 0, s, logits, ld, bias, n_expert, top, ids, w, T));
    return 0;
}

}  // namespace dlp
