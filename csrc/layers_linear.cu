// Matrix products of the layer-list models and the row preparation around them.
//
//   matvec_kernel        decode (1..4 rows): weights streamed once; the residual sum and the norms in front of a product run in the
//                        prologue, an activation in the epilogue.  Any N, any K whose padded form is a multiple of 8.
//   stage_rows_kernel    the same row preparation as one launch, for the tcgen05 GEMM sizes (stage_reg_kernel: one norm of a wide row).
//   sgemm_kernel         fp32 storage, any number of rows (no reduced-precision product).
//   head_matmul_kernel   one small matrix per head (latent attention's key absorption and value expansion), mma.sync m16n8k16.
#include "layers_rows.cuh"
#include "mma.cuh"

namespace dlp {

__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename XT, int FORM>
__global__ void __launch_bounds__(256) stage_rows_kernel(const RowStage p, XT* xb, int ldxb) {
    extern __shared__ __align__(16) float st_sums[];
    pdl_wait();
    const int t0 = blockIdx.x;
    stage_rows_dev<XT, FORM>(p, t0, 1, st_sums, true, xb + (size_t)t0 * ldxb, ldxb);
    pdl_launch_dependents();
}

// The pre-norm form (plain residual sum, layer norm or, with CENTRED = false, RMS norm of the whole row) with the row in registers: everything is
// read once.  NV float4 per thread.
template <typename XT, int NV, bool CENTRED>
__global__ void __launch_bounds__(256) stage_reg_kernel(const RowStage p, XT* xb, int ldxb) {
    __shared__ float red[32];
    pdl_wait();
    const int t = blockIdx.x, q = p.K >> 2;
    float4 v[NV];
    float a = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int k = (i * 256 + threadIdx.x) * 4;
        v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (k < p.K) {
            v[i] = stage_x4<XT>(p, t, k);
            if (p.y) {
                const float4 y = *reinterpret_cast<const float4*>(p.y + (size_t)t * p.ldy + k);
                v[i].x += y.x; v[i].y += y.y; v[i].z += y.z; v[i].w += y.w;
            }
            if (p.e) {
                const float4 e = *reinterpret_cast<const float4*>(p.e + (size_t)t * p.lde + k);
                v[i].x += e.x; v[i].y += e.y; v[i].z += e.z; v[i].w += e.w;
            }
            if (p.h_out) *reinterpret_cast<float4*>(p.h_out + (size_t)t * p.ldh + k) = v[i];
        }
        a += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    }
    const float mean = CENTRED ? block_sum(a, red) / (float)p.K : 0.f;
    a = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
        if (i * 256 + (int)threadIdx.x < q) {
            if (CENTRED) v[i] = make_float4(v[i].x - mean, v[i].y - mean, v[i].z - mean, v[i].w - mean);
            a = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, a))));
        }
    const float r = 1.f / sqrtf(block_sum(a, red) / (float)p.K + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int k = (i * 256 + threadIdx.x) * 4;
        if (k < p.K) {
            const float4 w = *reinterpret_cast<const float4*>(p.w2 + k), b = CENTRED ? *reinterpret_cast<const float4*>(p.b2 + k) : make_float4(0.f, 0.f, 0.f, 0.f);
            put4(xb + (size_t)t * ldxb + k, make_float4(fmaf(v[i].x * r, w.x, b.x), fmaf(v[i].y * r, w.y, b.y), fmaf(v[i].z * r, w.z, b.z), fmaf(v[i].w * r, w.w, b.w)));
        }
    }
    pdl_launch_dependents();
}
template <typename XT, bool CENTRED>
static cudaError_t launch_stage_reg(const RowStage& st, XT* xb, int ldxb, int T, cudaStream_t s) {
    if (st.K <= 2048) return launch_pdl(stage_reg_kernel<XT, 2, CENTRED>, dim3(T), dim3(256), 0, s, st, xb, ldxb);
    if (st.K <= 4096) return launch_pdl(stage_reg_kernel<XT, 4, CENTRED>, dim3(T), dim3(256), 0, s, st, xb, ldxb);
    return launch_pdl(stage_reg_kernel<XT, 8, CENTRED>, dim3(T), dim3(256), 0, s, st, xb, ldxb);
}
template <typename XT>
static cudaError_t launch_stage(const RowStage& st, XT* xb, int ldxb, int T, size_t smem, cudaStream_t s) {
    const int form = stage_form(st);
    if (form != ST_MIXER && st.w2 && st.groups2 == 1 && st.w2_mod == st.K && !(st.y && st.w1) && stage_vec(st) && ldxb % 4 == 0 && st.K <= 8192)
        return st.b2 ? launch_stage_reg<XT, true>(st, xb, ldxb, T, s) : launch_stage_reg<XT, false>(st, xb, ldxb, T, s);
    auto kern = form == ST_MIXER ? stage_rows_kernel<XT, ST_MIXER> : form == ST_SUM ? stage_rows_kernel<XT, ST_SUM> : stage_rows_kernel<XT, ST_NORMED>;
    return launch_pdl(kern, dim3(T), dim3(256), smem, s, st, xb, ldxb);
}

template <typename WT>
__device__ __forceinline__ void store_tail(const OutTail& tl, void* out, int ldo, int t, int n, float v) {
    if (tl.bias != nullptr) v += tl.bias[n];
    if (n < tl.n2) reinterpret_cast<float*>(out)[(size_t)t * ldo + n] = v;
    else reinterpret_cast<WT*>(tl.out2)[(size_t)t * tl.ldo2 + n - tl.n2] = Act<WT>::from_f(xielu(v, tl.pos, tl.neg));
}
static int check_tail(const OutTail* tl, int N, int out_mode, const char* who) {
    DLP_REQUIRE(!tl || (out_mode == LO_F32 && tl->n2 >= 0 && (tl->n2 >= N || (tl->out2 && tl->ldo2 >= N - tl->n2))), "%s: what follows the sums", who);
    return 0;
}

// ---- decode mat-vec ------------------------------------------------------------------------------------------
// A unit is two weight rows x (32 * VEC * U) columns: U 16-byte loads per row and lane.  A block owns a contiguous range of row
// pairs, its warps take the units in a fixed order and always hold the next unit's loads while they reduce the current one.  The
// first unit is requested before the dependency wait: weights do not depend on the previous kernel.
template <typename WT, int NT, int FORM>
__global__ void __launch_bounds__(512, 1) matvec_kernel(const RowStage st, const WT* __restrict__ w, int ldw, int N, void* out, int ldo, int out_mode, int T, const OutTail tl) {
    constexpr int VEC = Act<WT>::VEC, U = 4, COLS = 32 * VEC * U;
    extern __shared__ __align__(16) uint8_t mv_smem[];
    WT* xs = reinterpret_cast<WT*>(mv_smem);
    const int K = st.Kp + st.K_tail;
    size_t off = ((size_t)NT * K * sizeof(WT) + 15) & ~size_t(15);
    float* sums = reinterpret_cast<float*>(mv_smem + off);
    const int KC = (K + COLS - 1) / COLS;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int pairs = (N + 1) / 2;
    const int p_lo = (int)((long long)pairs * blockIdx.x / gridDim.x), p_hi = (int)((long long)pairs * (blockIdx.x + 1) / gridDim.x);
    const int units = (p_hi - p_lo) * KC;
    uint4 buf[2][2][U];
    auto issue = [&](int u, int b) {
        const int pr = u / KC, c = u - pr * KC, row = (p_lo + pr) * 2;
        const WT* r0 = w + (size_t)row * ldw + c * COLS + lane * VEC;
        const WT* r1 = w + (size_t)min(row + 1, N - 1) * ldw + c * COLS + lane * VEC;
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const bool ok = c * COLS + i * 32 * VEC + lane * VEC < K;
            buf[b][0][i] = ok ? ldg_nc_v4(r0 + i * 32 * VEC) : make_uint4(0, 0, 0, 0);
            buf[b][1][i] = ok ? ldg_nc_v4(r1 + i * 32 * VEC) : make_uint4(0, 0, 0, 0);
        }
    };
    int u = warp;
    if (u < units) issue(u, 0);
    pdl_wait();
    if (st.K_tail > 0) stage_tails<WT>(st, T, xs, K);
    stage_rows_dev<WT, FORM>(st, 0, T, sums, blockIdx.x == 0, xs, K);
    float* part = sums;      // [units][2][NT]: the staging scratch is free again
    auto reduce = [&](int u, int b) {
        const int pr = u / KC, c = u - pr * KC;
        float acc[2][NT];
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int t = 0; t < NT; ++t) acc[m][t] = 0.f;
#pragma unroll
        for (int i = 0; i < U; ++i) {
            const int k = c * COLS + i * 32 * VEC + lane * VEC;
            if (k < K) {
                float wf[2][VEC];
#pragma unroll
                for (int m = 0; m < 2; ++m) {
                    const uint32_t ww[4] = {buf[b][m][i].x, buf[b][m][i].y, buf[b][m][i].z, buf[b][m][i].w};
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        if (VEC == 8) {
                            const float2 f = bf2_to_f2(ww[j]);
                            wf[m][(2 * j) % VEC] = f.x;
                            wf[m][(2 * j + 1) % VEC] = f.y;
                        } else {
                            wf[m][j] = __uint_as_float(ww[j]);
                        }
                    }
                }
#pragma unroll
                for (int t = 0; t < NT; ++t) {
                    if (t >= T) break;
                    const uint4 xv = *reinterpret_cast<const uint4*>(xs + (size_t)t * K + k);
                    const uint32_t xw[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        if (VEC == 8) {
                            const float2 f = bf2_to_f2(xw[j]);
#pragma unroll
                            for (int m = 0; m < 2; ++m) {
                                acc[m][t] = fmaf(wf[m][(2 * j) % VEC], f.x, acc[m][t]);
                                acc[m][t] = fmaf(wf[m][(2 * j + 1) % VEC], f.y, acc[m][t]);
                            }
                        } else {
#pragma unroll
                            for (int m = 0; m < 2; ++m) acc[m][t] = fmaf(wf[m][j], __uint_as_float(xw[j]), acc[m][t]);
                        }
                    }
                }
            }
        }
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int t = 0; t < NT; ++t) {
                const float v = warp_sum(acc[m][t]);
                if (lane == 0) part[((size_t)u * 2 + m) * NT + t] = v;
            }
    };
    // two register sets, unrolled by hand so that the set index is a constant
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
    for (int i = threadIdx.x; i < np * NT; i += blockDim.x) {
        const int pr = i / NT, t = i - pr * NT;
        if (t >= T) continue;
        float a0 = 0.f, a1 = 0.f;
        for (int c = 0; c < KC; ++c) {
            a0 += part[((size_t)(pr * KC + c) * 2) * NT + t];
            a1 += part[((size_t)(pr * KC + c) * 2 + 1) * NT + t];
        }
        const int row = (p_lo + pr) * 2;
        if (out_mode == LO_GEGLU || out_mode == LO_SWIGLU) {
            reinterpret_cast<WT*>(out)[(size_t)t * ldo + (row >> 1)] = Act<WT>::from_f((out_mode == LO_GEGLU ? gelu_tanh_f(a0) : silu_exact(a0)) * a1);
        } else if (out_mode == LO_RELU2) {
            WT* o = reinterpret_cast<WT*>(out) + (size_t)t * ldo + row;
            a0 = fmaxf(a0, 0.f);
            a1 = fmaxf(a1, 0.f);
            o[0] = Act<WT>::from_f(a0 * a0);
            if (row + 1 < N) o[1] = Act<WT>::from_f(a1 * a1);
        } else {
            store_tail<WT>(tl, out, ldo, t, row, a0);
            if (row + 1 < N) store_tail<WT>(tl, out, ldo, t, row + 1, a1);
        }
    }
}

template <typename WT, int NT>
static int launch_matvec(const RowStage& st, const void* w, int ldw, int N, void* out, int ldo, int out_mode, int T, cudaStream_t s, const OutTail& tl) {
    constexpr int COLS = 32 * Act<WT>::VEC * 4;
    const int K = st.Kp + st.K_tail, pairs = (N + 1) / 2, KC = (K + COLS - 1) / COLS;
    const int grid = pairs < sm_count() ? pairs : sm_count();
    const size_t xbytes = ((size_t)NT * K * sizeof(WT) + 15) & ~size_t(15);
    const size_t part = (size_t)((pairs + grid - 1) / grid) * KC * 2 * NT * 4, stg = stage_bytes(st, T, 16);
    const size_t smem = xbytes + (part > stg ? part : stg);
    DLP_REQUIRE(smem <= 227 * 1024, "matvec: %d rows of width %d need %zu bytes of shared memory", T, K, smem);
    const int form = stage_form(st);
    auto kern = form == ST_MIXER ? matvec_kernel<WT, NT, ST_MIXER> : form == ST_SUM ? matvec_kernel<WT, NT, ST_SUM> : matvec_kernel<WT, NT, ST_NORMED>;
    if (first_use_on_device((const void*)kern))
        DLP_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    DLP_CHECK_CUDA(launch_pdl(kern, dim3(grid), dim3(512), smem, s, st, (const WT*)w, ldw, N, out, ldo, out_mode, T, tl));
    return 0;
}

int matvec(const RowStage& st, const void* w, int ldw, int N, void* out, int ldo, int out_mode, int T, int f32, cudaStream_t s, const OutTail* tail) {
    int rc = check_stage(st, "matvec");
    if (!rc) rc = check_tail(tail, N, out_mode, "matvec");
    if (rc) return rc;
    const OutTail tl = tail ? *tail : OutTail();
    DLP_REQUIRE(w && out && N > 0 && T >= 1 && T <= 4, "matvec: bad argument (T=%d N=%d)", T, N);
    DLP_REQUIRE(st.Kp % 8 == 0 && ldw % 8 == 0 && ldw >= st.Kp + st.K_tail, "matvec: row length %d / stride %d must be multiples of 8", st.Kp, ldw);
    DLP_REQUIRE(out_mode == LO_F32 || out_mode == LO_RELU2 || ((out_mode == LO_GEGLU || out_mode == LO_SWIGLU) && N % 2 == 0), "matvec: output mode %d", out_mode);
    if (f32) {
        if (T == 1) return launch_matvec<float, 1>(st, w, ldw, N, out, ldo, out_mode, T, s, tl);
        if (T == 2) return launch_matvec<float, 2>(st, w, ldw, N, out, ldo, out_mode, T, s, tl);
        return launch_matvec<float, 4>(st, w, ldw, N, out, ldo, out_mode, T, s, tl);
    }
    if (T == 1) return launch_matvec<__nv_bfloat16, 1>(st, w, ldw, N, out, ldo, out_mode, T, s, tl);
    if (T == 2) return launch_matvec<__nv_bfloat16, 2>(st, w, ldw, N, out, ldo, out_mode, T, s, tl);
    return launch_matvec<__nv_bfloat16, 4>(st, w, ldw, N, out, ldo, out_mode, T, s, tl);
}

int stage_rows(const RowStage& st, void* xb, int ldxb, int T, int f32, cudaStream_t s) {
    int rc = check_stage(st, "stage_rows");
    if (rc) return rc;
    DLP_REQUIRE(xb && T > 0 && ldxb >= st.Kp && st.K_tail == 0, "stage_rows: bad argument");
    const size_t smem = stage_bytes(st, 1, 8);
    DLP_REQUIRE(smem <= 48 * 1024, "stage_rows: too many norm groups");
    DLP_CHECK_CUDA(f32 ? launch_stage(st, (float*)xb, ldxb, T, smem, s) : launch_stage(st, (__nv_bfloat16*)xb, ldxb, T, smem, s));
    return 0;
}

// ---- fp32 matrix product ---------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) sgemm_kernel(const float* __restrict__ x, int ldx, const float* __restrict__ w, int ldw, int N, int K, float* out, int ldo,
                                                    int out_mode, int T, const GemmGroup grp, const OutTail tl) {
    __shared__ float xs[16][68], ws[16][68];
    const int n0 = blockIdx.x * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    int t0 = blockIdx.y * 64;
    float acc[4][4] = {};
    pdl_wait();
    if (grp.tile_expert != nullptr) {        // rows sorted by expert: this tile's rows and its matrix in the stack
        if ((int)blockIdx.y >= *grp.n_tiles) return;
        t0 = grp.tile_row0[blockIdx.y];
        T = t0 + grp.tile_rows[blockIdx.y];
        w += (size_t)grp.tile_expert[blockIdx.y] * grp.rows_per_expert * ldw;
    }
    for (int k0 = 0; k0 < K; k0 += 16) {
        for (int i = threadIdx.x; i < 64 * 16; i += 256) {
            const int r = i >> 4, k = i & 15;
            xs[k][r] = (t0 + r < T && k0 + k < K) ? x[(size_t)(t0 + r) * ldx + k0 + k] : 0.f;
            ws[k][r] = (n0 + r < N && k0 + k < K) ? w[(size_t)(n0 + r) * ldw + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { a[i] = xs[k][ty * 4 + i]; b[i] = ws[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
    pdl_launch_dependents();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = t0 + ty * 4 + i;
        if (t >= T) continue;
        if (out_mode == LO_GEGLU || out_mode == LO_SWIGLU) {
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int n = n0 + tx * 4 + j;
                if (n < N) out[(size_t)t * ldo + (n >> 1)] = (out_mode == LO_GEGLU ? gelu_tanh_f(acc[i][j]) : silu_exact(acc[i][j])) * acc[i][j + 1];
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (n0 + tx * 4 + j < N) {
                    const float u = fmaxf(acc[i][j], 0.f);
                    if (out_mode == LO_RELU2) out[(size_t)t * ldo + n0 + tx * 4 + j] = u * u;
                    else store_tail<float>(tl, out, ldo, t, n0 + tx * 4 + j, acc[i][j]);
                }
        }
    }
}

int sgemm(const float* x, int ldx, const float* w, int ldw, int N, int K, void* out, int ldo, int out_mode, int T, cudaStream_t s, const GemmGroup* grp,
          const OutTail* tail) {
    DLP_REQUIRE(x && w && out && N > 0 && K > 0 && T > 0, "sgemm: bad argument");
    const int rc = check_tail(tail, N, out_mode, "sgemm");
    if (rc) return rc;
    DLP_REQUIRE(out_mode == LO_F32 || out_mode == LO_RELU2 || ((out_mode == LO_GEGLU || out_mode == LO_SWIGLU) && N % 2 == 0), "sgemm: output mode %d", out_mode);
    DLP_REQUIRE(!grp || (grp->bt == 64 && grp->max_tiles > 0 && grp->max_tiles <= 65535), "sgemm: grouped launches take 64-row tiles");
    DLP_CHECK_CUDA(launch_pdl(sgemm_kernel, dim3((N + 63) / 64, grp ? grp->max_tiles : (T + 63) / 64), dim3(256), 0, s, x, ldx, w, ldw, N, K, (float*)out, ldo, out_mode, T,
                              grp ? *grp : GemmGroup(), tail ? *tail : OutTail()));
    return 0;
}

// ---- one matrix per head: out[t, h, n] = sum_k x[t, h, k] W[h][n][k]  (* sigmoid(gate[t, h])) ---------------
// A is 16 * MT tokens of one head (shared memory), B comes straight from global memory, 16 bytes per lane: the k index inside a
// 32-wide block is permuted the same way on both operands, so that a lane's eight k values are contiguous.
template <int MT>
__global__ void __launch_bounds__(128) head_matmul_kernel(const void* x, int x_f32, int ldx, int x_head, int kx, const __nv_bfloat16* __restrict__ w, int Kp, int N,
                                                          int n_rows, __nv_bfloat16* out, int ldo, int out_head, const float* gate, int ldg, int T) {
    extern __shared__ __align__(16) uint8_t hm_smem[];
    __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(hm_smem);
    const int ldxs = Kp + 8, h = blockIdx.y, t0 = blockIdx.z * 16 * MT;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, c = lane & 3;
    pdl_wait();
    for (int i = threadIdx.x; i < 16 * MT * Kp; i += 128) {
        const int t = i / Kp, k = i - t * Kp;
        float v = 0.f;
        if (t0 + t < T && k < kx) {
            const size_t o = (size_t)(t0 + t) * ldx + (size_t)h * x_head + k;
            v = x_f32 ? reinterpret_cast<const float*>(x)[o] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(x)[o]);
        }
        xs[t * ldxs + k] = __float2bfloat16_rn(v);
    }
    __syncthreads();
    const int n0 = blockIdx.x * 64 + warp * 16;
    float acc[MT][2][4] = {};
    const __nv_bfloat16* wr[2];
    bool ok[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const int n = n0 + j * 8 + g;
        ok[j] = n < n_rows;
        wr[j] = w + ((size_t)h * n_rows + (ok[j] ? n : 0)) * Kp + c * 8;
    }
#pragma unroll 4
    for (int k = 0; k < Kp; k += 32) {
        uint4 b[2];
#pragma unroll
        for (int j = 0; j < 2; ++j) b[j] = ok[j] ? ldg_nc_v4(wr[j] + k) : make_uint4(0, 0, 0, 0);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const uint4 lo = *reinterpret_cast<const uint4*>(xs + (m * 16 + g) * ldxs + k + c * 8);
            const uint4 hi = *reinterpret_cast<const uint4*>(xs + (m * 16 + g + 8) * ldxs + k + c * 8);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                mma16816(acc[m][j], {lo.x, hi.x, lo.y, hi.y}, b[j].x, b[j].y);
                mma16816(acc[m][j], {lo.z, hi.z, lo.w, hi.w}, b[j].z, b[j].w);
            }
        }
    }
    pdl_launch_dependents();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int t = t0 + m * 16 + g + r * 8;
            if (t >= T) continue;
            const float sc = gate ? 1.f / (1.f + expf(-gate[(size_t)t * ldg + h])) : 1.f;
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int n = n0 + j * 8 + c * 2 + e;
                    if (n < N) out[(size_t)t * ldo + (size_t)h * out_head + n] = __float2bfloat16_rn(acc[m][j][r * 2 + e] * sc);
                }
        }
}

// up to 16 tokens: a block takes 16 outputs of one head, its four warps share the inner dimension, so that every weight byte of the
// block is requested at once
__global__ void __launch_bounds__(128) head_matmul_small_kernel(const void* x, int x_f32, int ldx, int x_head, int kx, const __nv_bfloat16* __restrict__ w, int Kp, int N,
                                                                int n_rows, __nv_bfloat16* out, int ldo, int out_head, const float* gate, int ldg, int T) {
    extern __shared__ __align__(16) uint8_t hm_smem[];
    __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(hm_smem);      // [T][Kp + 8]
    __shared__ float red[4][16][17];
    const int ldxs = Kp + 8, h = blockIdx.y, n0 = blockIdx.x * 16;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, c = lane & 3;
    const __nv_bfloat16* wr[2];
    bool ok[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const int n = n0 + j * 8 + g;
        ok[j] = n < n_rows;
        wr[j] = w + ((size_t)h * n_rows + (ok[j] ? n : 0)) * Kp + c * 8;
    }
    constexpr int U = 4;                       // 32-wide inner blocks in flight
    uint4 b[U][2];
    auto load = [&](int k) {
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int j = 0; j < 2; ++j) b[u][j] = (ok[j] && k + u * 128 < Kp) ? ldg_nc_v4(wr[j] + k + u * 128) : make_uint4(0, 0, 0, 0);
    };
    load(warp * 32);                           // weights do not depend on the previous kernel
    pdl_wait();
    for (int i0 = threadIdx.x; i0 < T * Kp; i0 += 8 * 128) {      // eight loads in flight per thread
        float v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int t = (i0 + i * 128) / Kp, k = (i0 + i * 128) - t * Kp;
            const size_t o = (size_t)t * ldx + (size_t)h * x_head + k;
            v[i] = (t < T && k < kx) ? (x_f32 ? reinterpret_cast<const float*>(x)[o] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(x)[o])) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int t = (i0 + i * 128) / Kp, k = (i0 + i * 128) - t * Kp;
            if (t < T) xs[t * ldxs + k] = __float2bfloat16_rn(v[i]);
        }
    }
    __syncthreads();
    float acc[2][4] = {};
    for (int k0 = warp * 32; k0 < Kp; k0 += U * 128) {
        if (k0 != warp * 32) load(k0);
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int k = k0 + u * 128;
            if (k < Kp) {
                const uint4 zero = make_uint4(0, 0, 0, 0);
                const uint4 lo = g < T ? *reinterpret_cast<const uint4*>(xs + g * ldxs + k + c * 8) : zero;
                const uint4 hi = g + 8 < T ? *reinterpret_cast<const uint4*>(xs + (g + 8) * ldxs + k + c * 8) : zero;
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    mma16816(acc[j], {lo.x, hi.x, lo.y, hi.y}, b[u][j].x, b[u][j].y);
                    mma16816(acc[j], {lo.z, hi.z, lo.w, hi.w}, b[u][j].z, b[u][j].w);
                }
            }
        }
    }
    pdl_launch_dependents();
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) red[warp][g + (e >> 1) * 8][j * 8 + c * 2 + (e & 1)] = acc[j][e];
    __syncthreads();
    for (int i = threadIdx.x; i < T * 16; i += 128) {
        const int t = i >> 4, n = n0 + (i & 15);
        if (n >= N) continue;
        float v = red[0][t][i & 15] + red[1][t][i & 15] + red[2][t][i & 15] + red[3][t][i & 15];
        if (gate) v *= 1.f / (1.f + expf(-gate[(size_t)t * ldg + h]));
        out[(size_t)t * ldo + (size_t)h * out_head + n] = __float2bfloat16_rn(v);
    }
}

__global__ void __launch_bounds__(128) head_matmul_f32_kernel(const float* x, int ldx, int x_head, int kx, const float* __restrict__ w, int Kp, int N, int n_rows,
                                                              float* out, int ldo, int out_head, const float* gate, int ldg) {
    extern __shared__ __align__(16) float hf_x[];
    const int h = blockIdx.y, t = blockIdx.z, n = blockIdx.x * 128 + threadIdx.x;
    pdl_wait();
    for (int k = threadIdx.x; k < Kp; k += 128) hf_x[k] = k < kx ? x[(size_t)t * ldx + (size_t)h * x_head + k] : 0.f;
    __syncthreads();
    pdl_launch_dependents();
    if (n >= N) return;
    const float* wr = w + ((size_t)h * n_rows + n) * Kp;
    float a = 0.f;
    for (int k = 0; k < Kp; ++k) a = fmaf(hf_x[k], wr[k], a);
    if (gate) a *= 1.f / (1.f + expf(-gate[(size_t)t * ldg + h]));
    out[(size_t)t * ldo + (size_t)h * out_head + n] = a;
}

// w is [H][n_rows][Kp] with zero padding along k; x holds kx values per head
int head_matmul(const void* x, int x_f32, int ldx, int x_head, int kx, const void* w, int Kp, int H, int N, int n_rows, void* out, int ldo, int out_head,
                const float* gate, int ldg, int T, int f32, cudaStream_t s) {
    DLP_REQUIRE(x && w && out && H > 0 && N > 0 && N <= n_rows && T > 0 && kx <= Kp && Kp % 32 == 0, "head_matmul: bad argument (Kp=%d N=%d)", Kp, N);
    if (f32) {
        for (int t = 0; t < T; t += 32768) {     // grid.z limit
            const int n = T - t < 32768 ? T - t : 32768;
            DLP_CHECK_CUDA(launch_pdl(head_matmul_f32_kernel, dim3((N + 127) / 128, H, n), dim3(128), Kp * 4, s, (const float*)x + (size_t)t * ldx, ldx, x_head, kx,
                                      (const float*)w, Kp, N, n_rows, (float*)out + (size_t)t * ldo, ldo, out_head, gate ? gate + (size_t)t * ldg : nullptr, ldg));
        }
        return 0;
    }
    if (T <= 16) {
        const size_t smem = (size_t)T * (Kp + 8) * 2;
        DLP_REQUIRE(smem <= 200 * 1024, "head_matmul: inner size %d", Kp);
        auto k1 = head_matmul_small_kernel;
        if (first_use_on_device((const void*)k1)) DLP_CHECK_CUDA(cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        DLP_CHECK_CUDA(launch_pdl(k1, dim3((N + 15) / 16, H), dim3(128), smem, s, x, x_f32, ldx, x_head, kx, (const __nv_bfloat16*)w, Kp, N, n_rows, (__nv_bfloat16*)out, ldo,
                                  out_head, gate, ldg, T));
        return 0;
    }
    constexpr int MT = 4;
    const size_t smem = (size_t)16 * MT * (Kp + 8) * 2;
    DLP_REQUIRE(smem <= 227 * 1024, "head_matmul: inner size %d", Kp);
    dim3 grid((N + 63) / 64, H, (T + 16 * MT - 1) / (16 * MT));
    auto k4 = head_matmul_kernel<MT>;
    if (first_use_on_device((const void*)k4)) DLP_CHECK_CUDA(cudaFuncSetAttribute(k4, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    DLP_CHECK_CUDA(launch_pdl(k4, grid, dim3(128), smem, s, x, x_f32, ldx, x_head, kx, (const __nv_bfloat16*)w, Kp, N, n_rows, (__nv_bfloat16*)out, ldo, out_head, gate, ldg, T));
    return 0;
}

}  // namespace dlp
