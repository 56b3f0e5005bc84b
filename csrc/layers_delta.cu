// Gated delta rule: a matrix state per head that decays, and is corrected towards the value of every new key before it is read.
//
//   S <- f_t S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t            (k, q unit vectors, q scaled)
//
//   delta_decode_kernel   one token per sequence: the state is read once, in 16-byte pieces, requested before the dependency wait; the
//                         convolution of the token (its inputs come out of the ring) is part of the launch
//   delta_scan_kernel     token by token (short portions, fp32 storage, any size)
//   delta_chunk_solve / delta_chunk_state / delta_chunk_out   64-token chunks on the tensor cores
//
// Chunks: with L the cumulative log decay inside a chunk, the writes solve a unit lower triangular system,
//   (I + A) u = beta (v - exp(L) S_start^T k),   A_ts = beta_t exp(L_t - L_s) (k_t . k_s),  s < t
// whose inverse does not depend on the state: it is formed for all chunks at once (solve), as are the weights of the outputs; the state then
// runs over the chunks (state), and
//   o_t = exp(L_t) S_start^T q_t + sum_{s <= t} exp(L_t - L_s) (q_t . k_s) u_s
// again for all chunks at once (out).  Exponents are never positive.  Rows behind the convolution are bf16 operands as they are; the factors
// that make q and k unit vectors join the fp32 token weights.  Weights, inverse, writes and states are fp32 and enter the tensor cores as two
// bf16 parts (value and remainder).
#include "layers_chunks.cuh"

namespace dlp {

constexpr float LOG2E_F = 1.4426950408889634f;
// logarithm of a token's decay, and how much of it is written
__device__ __forceinline__ float delta_log_decay(const DeltaArgs& a, int t, int h) { return a.log_decay[h] * softplus_exact(a.a[(size_t)t * a.lda + h] + a.dt_bias[h]); }
__device__ __forceinline__ float delta_beta(const DeltaArgs& a, int t, int h) { return sigmoid_exact(a.b[(size_t)t * a.ldb + h]); }

static int check_delta(const DeltaArgs& a, const char* who) {
    DLP_REQUIRE(a.q && a.k && a.v && a.a && a.b && a.log_decay && a.dt_bias && a.state && a.seg && a.seg_slot && a.pos && a.out, "%s: null argument", who);
    DLP_REQUIRE(a.H > 0 && a.H <= 65535 && a.D > 0 && a.V > 0 && a.n_seg > 0 && a.n_seg <= 65535 && a.hpg > 0 && a.H % a.hpg == 0, "%s: bad shape (%d heads of %d x %d, %d per group)", who,
                a.H, a.D, a.V, a.hpg);
    return 0;
}

// ---- token by token ------------------------------------------------------------------------------------------------------------------
// One CTA = one (segment, head, slice of 128 / RG value columns); a thread keeps RPT state rows of one column.  Both products with the state
// before the write are one pass; what the read-out owes to the write is (k . q) u.
template <int RG, int RPT>
struct DeltaScanCfg {
    static constexpr int COLS = 128 / RG, ROWS = RG * RPT, CT = 2048 / ROWS > 16 ? 16 : (2048 / ROWS < 4 ? 4 : 2048 / ROWS), GS = RPT + 4;
    static constexpr size_t SMEM = (size_t)CT * (2 * RG * GS + COLS + 5) * 4;
};
template <int RG, int RPT>
__global__ void __launch_bounds__(128) delta_scan_kernel(const DeltaArgs a) {
    using C = DeltaScanCfg<RG, RPT>;
    constexpr int COLS = C::COLS, ROWS = C::ROWS, CT = C::CT, GS = C::GS;
    extern __shared__ __align__(16) float dl_smem[];
    float* sq = dl_smem;                        // [CT][RG * GS]
    float* sk = sq + CT * RG * GS;
    float* sv = sk + CT * RG * GS;              // [CT][COLS]
    float* sf = sv + CT * COLS;                 // [CT] decay, write strength, 1 / |q| (scaled), 1 / |k|, k . q
    float *sb = sf + CT, *srq = sb + CT, *srk = srq + CT, *skq = srk + CT;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rg = tid % RG, col = tid / RG;
    const int seg = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * COLS, g = h / a.hpg;
    pdl_wait();
    const int lo = a.seg[2 * seg], hi = a.seg[2 * seg + 1];
    if (lo >= hi) return;
    float S[RPT];
    float* st = a.state + (((size_t)a.seg_slot[seg] * a.H + h) * a.D + rg * RPT) * a.V + v0 + col;
    const bool col_ok = v0 + col < a.V, fresh = a.pos[lo] == 0;
#pragma unroll
    for (int i = 0; i < RPT; ++i) S[i] = (!fresh && col_ok && rg * RPT + i < a.D) ? st[(size_t)i * a.V] : 0.f;
    for (int t0 = lo; t0 < hi; t0 += CT) {
        const int n = min(CT, hi - t0);
        __syncthreads();
        for (int i = tid; i < n * ROWS; i += 128) {
            const int t = i / ROWS, d = i - t * ROWS, o = t * RG * GS + (d / RPT) * GS + d % RPT;
            sq[o] = d < a.D ? mix_row(a.q, a.rows_f32, 0, (size_t)(t0 + t) * a.ldq + g * a.D + d) : 0.f;
            sk[o] = d < a.D ? mix_row(a.k, a.rows_f32, 0, (size_t)(t0 + t) * a.ldk + g * a.D + d) : 0.f;
        }
        for (int i = tid; i < n * COLS; i += 128) {
            const int t = i / COLS, c = i - t * COLS;
            sv[i] = v0 + c < a.V ? mix_row(a.v, a.rows_f32, 0, (size_t)(t0 + t) * a.ldv + h * a.V + v0 + c) : 0.f;
        }
        __syncthreads();
        for (int t = warp; t < n; t += 4) {
            float qq = 0.f, kk = 0.f, kq = 0.f;
            for (int d = lane; d < ROWS; d += 32) {
                const int o = t * RG * GS + (d / RPT) * GS + d % RPT;
                const float q = sq[o], k = sk[o];
                qq = fmaf(q, q, qq);
                kk = fmaf(k, k, kk);
                kq = fmaf(k, q, kq);
            }
            qq = warp_sum(qq);
            kk = warp_sum(kk);
            kq = warp_sum(kq);
            if (lane == 0) {
                const float rq = a.q_scale / sqrtf(qq + a.unit_eps), rk = 1.f / sqrtf(kk + a.unit_eps);
                sf[t] = expf(delta_log_decay(a, t0 + t, h));
                sb[t] = delta_beta(a, t0 + t, h);
                srq[t] = rq;
                srk[t] = rk;
                skq[t] = kq * rq * rk;
            }
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float4* q4 = reinterpret_cast<const float4*>(sq + t * RG * GS + rg * GS);
            const float4* k4 = reinterpret_cast<const float4*>(sk + t * RG * GS + rg * GS);
            float x0 = 0.f, x1 = 0.f, y0 = 0.f, y1 = 0.f;        // S^T k, S^T q
#pragma unroll
            for (int i = 0; i < RPT / 4; ++i) {
                const float4 q = q4[i], k = k4[i];
                x0 = fmaf(k.x, S[4 * i], x0);
                x1 = fmaf(k.y, S[4 * i + 1], x1);
                x0 = fmaf(k.z, S[4 * i + 2], x0);
                x1 = fmaf(k.w, S[4 * i + 3], x1);
                y0 = fmaf(q.x, S[4 * i], y0);
                y1 = fmaf(q.y, S[4 * i + 1], y1);
                y0 = fmaf(q.z, S[4 * i + 2], y0);
                y1 = fmaf(q.w, S[4 * i + 3], y1);
            }
            float x = x0 + x1, y = y0 + y1;
#pragma unroll
            for (int o = 1; o < RG; o <<= 1) {
                x += __shfl_xor_sync(0xffffffffu, x, o);
                y += __shfl_xor_sync(0xffffffffu, y, o);
            }
            const float f = sf[t], rk = srk[t], u = sb[t] * (sv[t * COLS + col] - f * rk * x), ku = rk * u;
#pragma unroll
            for (int i = 0; i < RPT / 4; ++i) {
                const float4 k = k4[i];
                S[4 * i] = fmaf(f, S[4 * i], k.x * ku);
                S[4 * i + 1] = fmaf(f, S[4 * i + 1], k.y * ku);
                S[4 * i + 2] = fmaf(f, S[4 * i + 2], k.z * ku);
                S[4 * i + 3] = fmaf(f, S[4 * i + 3], k.w * ku);
            }
            if (rg == 0 && col_ok) a.out[(size_t)(t0 + t) * a.ldo + h * a.V + v0 + col] = fmaf(f * srq[t], y, skq[t] * u);
        }
    }
    pdl_launch_dependents();
#pragma unroll
    for (int i = 0; i < RPT; ++i)
        if (col_ok && rg * RPT + i < a.D) st[(size_t)i * a.V] = S[i];
}
template <int RG, int RPT>
static int launch_delta_scan(const DeltaArgs& a, cudaStream_t s) {
    using C = DeltaScanCfg<RG, RPT>;
    static_assert(C::SMEM <= 48 * 1024, "scan staging");
    DLP_CHECK_CUDA(launch_pdl(delta_scan_kernel<RG, RPT>, dim3((a.V + C::COLS - 1) / C::COLS, a.H, a.n_seg), dim3(128), C::SMEM, s, a));
    return 0;
}
int delta_scan(const DeltaArgs& a, cudaStream_t s) {
    const int rc = check_delta(a, "delta_scan");
    if (rc) return rc;
    if (a.D <= 64) return launch_delta_scan<4, 16>(a, s);
    if (a.D <= 128) return launch_delta_scan<4, 32>(a, s);
    if (a.D <= 256) return launch_delta_scan<8, 32>(a, s);
    DLP_REQUIRE(a.D <= 1024, "delta_scan: %d channels per head (at most 1024)", a.D);
    return launch_delta_scan<16, 64>(a, s);
}

// ---- one token per sequence ------------------------------------------------------------------------------------------------------------
// A block takes 32 columns of one head's state: eight lanes cover the columns (four each), 32 row slots of NR rows each.
template <int NR, bool CONV>
__global__ void __launch_bounds__(256) delta_decode_kernel(const DeltaArgs a, const ConvArgs cv) {
    constexpr int COLS = 32;
    extern __shared__ __align__(16) float dl_smem[];
    float* sq = dl_smem;                    // [D]
    float* sk = sq + a.D;                   // [D]
    float* sv = sk + a.D;                   // [COLS]
    __shared__ __align__(16) float red[2][8][COLS];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, c0 = (tid & 7) * 4, rs = tid >> 3, h = blockIdx.y, v0 = blockIdx.x * COLS, g = h / a.hpg;
    // (segments, positions and states were written at least two launches back)
    const int t = a.seg[2 * blockIdx.z], slot = a.seg_slot[blockIdx.z], pos = a.pos[t];
    const bool ok = v0 + c0 < a.V;
    float* st = a.state + ((size_t)slot * a.H + h) * a.D * a.V + v0 + c0;
    float4 S[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = rs + 32 * i;
        S[i] = pos > 0 && d < a.D && ok ? *reinterpret_cast<const float4*>(st + (size_t)d * a.V) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_wait();
    const float f = expf(delta_log_decay(a, t, h)), beta = delta_beta(a, t, h);
    const bool first_block = blockIdx.x == 0 && h == g * a.hpg;       // of those that share q and k
    for (int i = tid; i < 2 * a.D + COLS; i += 256) {
        const int part = i < a.D ? 0 : i < 2 * a.D ? 1 : 2, j = i - part * a.D;
        float x = 0.f;
        if (part < 2 || v0 + j < a.V) {
            const int col = part < 2 ? g * a.D + j : h * a.V + v0 + j;
            if (CONV) {
                const float* row = reinterpret_cast<const float*>(part == 0 ? a.q : part == 1 ? a.k : a.v) + (size_t)t * cv.ldx + col;
                const int c = (int)(row - (cv.x + (size_t)t * cv.ldx));
                float* ring = cv.ring + (size_t)slot * cv.taps * cv.channels + c;
                const float now = *row;
                x = fmaf(cv.w[(size_t)(cv.taps - 1) * cv.channels + c], now, cv.b ? cv.b[c] : 0.f);
                for (int lag = 1; lag < cv.taps; ++lag)
                    if (pos >= lag) x = fmaf(cv.w[(size_t)(cv.taps - 1 - lag) * cv.channels + c], ring[(size_t)((pos - lag) % cv.taps) * cv.channels], x);
                x = silu_exact(x);
                if (part == 2 || first_block) ring[(size_t)(pos % cv.taps) * cv.channels] = now;
            } else {
                x = part == 0 ? mix_row(a.q, a.rows_f32, 0, (size_t)t * a.ldq + col) : part == 1 ? mix_row(a.k, a.rows_f32, 0, (size_t)t * a.ldk + col)
                                                                                                    : mix_row(a.v, a.rows_f32, 0, (size_t)t * a.ldv + col);
            }
        }
        dl_smem[i] = x;
    }
    __syncthreads();
    float qq = 0.f, kk = 0.f, kq = 0.f;       // every warp for itself
    for (int d = lane; d < a.D; d += 32) {
        const float q = sq[d], k = sk[d];
        qq = fmaf(q, q, qq);
        kk = fmaf(k, k, kk);
        kq = fmaf(k, q, kq);
    }
    float x[4] = {0.f, 0.f, 0.f, 0.f}, y[4] = {0.f, 0.f, 0.f, 0.f};        // S^T k, S^T q
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = rs + 32 * i;
        if (d < a.D) {
            const float k = sk[d], q = sq[d];
            x[0] = fmaf(k, S[i].x, x[0]);
            x[1] = fmaf(k, S[i].y, x[1]);
            x[2] = fmaf(k, S[i].z, x[2]);
            x[3] = fmaf(k, S[i].w, x[3]);
            y[0] = fmaf(q, S[i].x, y[0]);
            y[1] = fmaf(q, S[i].y, y[1]);
            y[2] = fmaf(q, S[i].z, y[2]);
            y[3] = fmaf(q, S[i].w, y[3]);
        }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        x[e] += __shfl_xor_sync(0xffffffffu, x[e], 8);
        y[e] += __shfl_xor_sync(0xffffffffu, y[e], 8);
        x[e] += __shfl_xor_sync(0xffffffffu, x[e], 16);
        y[e] += __shfl_xor_sync(0xffffffffu, y[e], 16);
    }
    if (lane < 8) {
        *reinterpret_cast<float4*>(&red[0][warp][c0]) = make_float4(x[0], x[1], x[2], x[3]);
        *reinterpret_cast<float4*>(&red[1][warp][c0]) = make_float4(y[0], y[1], y[2], y[3]);
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    kq = warp_sum(kq);
    const float rq = a.q_scale / sqrtf(qq + a.unit_eps), rk = 1.f / sqrtf(kk + a.unit_eps);
    __syncthreads();
    float4 xs = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < 8; ++w) {
        const float4 p = *reinterpret_cast<const float4*>(&red[0][w][c0]);
        xs.x += p.x; xs.y += p.y; xs.z += p.z; xs.w += p.w;
    }
    const float frk = f * rk;
    const float u[4] = {beta * (sv[c0] - frk * xs.x), beta * (sv[c0 + 1] - frk * xs.y), beta * (sv[c0 + 2] - frk * xs.z), beta * (sv[c0 + 3] - frk * xs.w)};
    pdl_launch_dependents();
    if (tid < 8 && ok) {
        float4 ys = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int w = 0; w < 8; ++w) {
            const float4 p = *reinterpret_cast<const float4*>(&red[1][w][c0]);
            ys.x += p.x; ys.y += p.y; ys.z += p.z; ys.w += p.w;
        }
        const float fq = f * rq, w = kq * rq * rk;
        float* o = a.out + (size_t)t * a.ldo + h * a.V + v0 + c0;
        o[0] = fmaf(fq, ys.x, w * u[0]);
        o[1] = fmaf(fq, ys.y, w * u[1]);
        o[2] = fmaf(fq, ys.z, w * u[2]);
        o[3] = fmaf(fq, ys.w, w * u[3]);
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = rs + 32 * i;
        if (d < a.D && ok) {
            const float k = sk[d] * rk;
            *reinterpret_cast<float4*>(st + (size_t)d * a.V) = make_float4(fmaf(f, S[i].x, k * u[0]), fmaf(f, S[i].y, k * u[1]), fmaf(f, S[i].z, k * u[2]), fmaf(f, S[i].w, k * u[3]));
        }
    }
}
template <int NR>
static int launch_delta_decode(const DeltaArgs& a, const ConvArgs* cv, cudaStream_t s) {
    const dim3 grid((a.V + 31) / 32, a.H, a.n_seg);
    const size_t smem = (size_t)(2 * a.D + 32) * 4;
    if (cv) DLP_CHECK_CUDA(launch_pdl(delta_decode_kernel<NR, true>, grid, dim3(256), smem, s, a, *cv));
    else DLP_CHECK_CUDA(launch_pdl(delta_decode_kernel<NR, false>, grid, dim3(256), smem, s, a, ConvArgs()));
    return 0;
}
int delta_decode(const DeltaArgs& a, const ConvArgs* cv, cudaStream_t s) {
    const int rc = check_delta(a, "delta_decode");
    if (rc) return rc;
    DLP_REQUIRE(a.D <= 256 && a.V % 4 == 0 && (reinterpret_cast<uintptr_t>(a.state) & 15) == 0, "delta_decode: state of %d x %d", a.D, a.V);
    DLP_REQUIRE(!cv || (cv->x && cv->w && cv->ring && cv->taps >= 1 && a.rows_f32 && a.ldq == cv->ldx && a.ldk == cv->ldx && a.ldv == cv->ldx), "delta_decode: convolution");
    if (a.D <= 64) return launch_delta_decode<2>(a, cv, s);
    if (a.D <= 128) return launch_delta_decode<4>(a, cv, s);
    return launch_delta_decode<8>(a, cv, s);
}

// ---- chunks --------------------------------------------------------------------------------------------------------------------------------
constexpr int DC = DELTA_CHUNK, DLT = DELTA_ROW;
typedef __nv_bfloat16 bf16;

// sums of squares of the rows of a [DC][DP + 8] tile, PT threads per row; every thread of a row gets its sum
template <int DP, int PT>
__device__ __forceinline__ float row_squares(const bf16* tile) {
    const bf16* row = tile + (threadIdx.x / PT) * (DP + 8);
    float s = 0.f;
#pragma unroll
    for (int c = (threadIdx.x % PT) * 8; c < DP; c += PT * 8) {
        const uint4 v = *reinterpret_cast<const uint4*>(row + c);
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float2 f = bf2_to_f2(w[e]);
            s = fmaf(f.x, f.x, fmaf(f.y, f.y, s));
        }
    }
#pragma unroll
    for (int o = 1; o < PT; o <<= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    return s;
}

constexpr int DGATES = DC * 4 + DC;             // floats of a chunk's gates
template <int DP> __device__ __forceinline__ bf16* chunk_keys(const DeltaArgs& a, const DeltaChunks& c, int ch, int h) {
    return reinterpret_cast<bf16*>(c.keys) + ((size_t)ch * (a.H / a.hpg) + h / a.hpg) * DC * (DP + 8);
}
__device__ __forceinline__ bf16* chunk_matrix(void* base, const DeltaArgs& a, int ch, int h) { return reinterpret_cast<bf16*>(base) + ((size_t)ch * a.H + h) * 2 * DC * DLT; }
__device__ __forceinline__ float* chunk_gates(const DeltaArgs& a, const DeltaChunks& c, int ch, int h) { return c.gates + ((size_t)ch * a.H + h) * DGATES; }
constexpr int DV = 16, DLV = DV + 8;            // value columns of a slice, and their row in shared memory
__device__ __forceinline__ size_t chunk_slice(const DeltaArgs& a, int ch, int h, int slice) { return ((size_t)ch * a.H + h) * ((a.V + DV - 1) / DV) + slice; }
// N 16-byte pieces to shared memory with cp.async, NTH threads
template <int N, int NTH>
__device__ __forceinline__ void copy_pieces(void* dst, const void* src) {
#pragma unroll
    for (int i = 0; i < (N + NTH - 1) / NTH; ++i)
        if (i * NTH + NTH - 1 < N || i * NTH + (int)threadIdx.x < N) cp_async16(reinterpret_cast<uint4*>(dst) + i * NTH + threadIdx.x, reinterpret_cast<const uint4*>(src) + i * NTH + threadIdx.x, true);
}

// Everything of a chunk that does not depend on the state: gates, the keys' tile, the weights of the outputs, and the inverse of I + A in fp32:
// its 16-row diagonal blocks by substitution (a lane per column), then what lies below them by blocks of 16 and of 32,
//   [P 0; R Q]^-1 = [P^-1 0; -Q^-1 R P^-1 Q^-1]
constexpr int DAP = DC + 4;
template <int DP>
struct DeltaSolveCfg {
    static constexpr int QT = DC * (DP + 8) * 2 > DC * DAP * 4 ? DC * (DP + 8) * 2 : DC * DAP * 4;      // the inverse takes the place of the queries
    static constexpr size_t SMEM = (size_t)DC * (DP + 8) * 2 + QT + (size_t)(DC * DAP + 4 * DC) * 4;
};
template <int DP>
__global__ void __launch_bounds__(256) delta_chunk_solve_kernel(const DeltaArgs a, const DeltaChunks cc) {
    constexpr int LDK = DP + 8;
    extern __shared__ __align__(16) uint8_t dc_smem[];
    bf16* sk = reinterpret_cast<bf16*>(dc_smem);                          // [DC][LDK]
    bf16* sq = sk + DC * LDK;                                             // [DC][LDK]
    float* Ti = reinterpret_cast<float*>(sq);                             // [DC][DAP]
    float* A = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(sq) + DeltaSolveCfg<DP>::QT);      // [DC][DAP]
    float* X = A + 32;                                                    // [32][DAP], above the blocks of A that are used
    float *sL = A + DC * DAP, *srk = sL + DC, *srq = srk + DC, *sb = srq + DC;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, ch = blockIdx.x, h = blockIdx.y;
    pdl_wait();
    const int t0 = cc.chunk[2 * ch], n = cc.chunk[2 * ch + 1];
    const size_t qk0 = (size_t)(h / a.hpg) * a.D;
    chunk_tile<bf16, DC, DP, 256>(a.k, a.ldk, qk0, t0, n, a.D, 0, sk);
    chunk_tile<bf16, DC, DP, 256>(a.q, a.ldq, qk0, t0, n, a.D, 0, sq);
    cp_commit();
    if (tid < DC) {
        float L = tid < n ? delta_log_decay(a, t0 + tid, h) * LOG2E_F : 0.f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(0xffffffffu, L, o);
            if (lane >= o) L += x;
        }
        sL[tid] = L;
        sb[tid] = tid < n ? delta_beta(a, t0 + tid, h) : 0.f;
    }
    cp_wait<0>();
    __syncthreads();
    const float carry = sL[31], kk = row_squares<DP, 4>(sk), qq = row_squares<DP, 4>(sq);
    if ((tid & 3) == 0) {
        srk[tid >> 2] = 1.f / sqrtf(kk + a.unit_eps);
        srq[tid >> 2] = a.q_scale / sqrtf(qq + a.unit_eps);
    }
    __syncthreads();
    if (tid >= 32 && tid < DC) sL[tid] += carry;
    __syncthreads();
    if (tid < DC) {
        const float L = sL[tid], end = sL[DC - 1], b = sb[tid], rk = srk[tid], from = exp2f(L);
        float* g = chunk_gates(a, cc, ch, h);
        reinterpret_cast<float4*>(g)[tid] = make_float4(b, b * from * rk, exp2f(end - L) * rk, exp2f(end));
        g[4 * DC + tid] = from * srq[tid];
    }
    if (h % a.hpg == 0) {
        bf16* out = chunk_keys<DP>(a, cc, ch, h);
        for (int i = tid; i < DC * LDK / 8; i += 256) reinterpret_cast<uint4*>(out)[i] = reinterpret_cast<const uint4*>(sk)[i];
    }
    // lower triangle in 16 x 16 blocks: A (ten blocks) and the weights (ten more)
    bf16* wout = chunk_matrix(cc.weights, a, ch, h);
    for (int idx = warp; idx < 20; idx += 8) {
        const bool is_w = idx >= 10;
        const int i = is_w ? idx - 10 : idx, mt = i < 1 ? 0 : i < 3 ? 1 : i < 6 ? 2 : 3, kb = i - mt * (mt + 1) / 2;
        const bf16* left = is_w ? sq : sk;
        float p[2][4] = {};
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) {
            uint32_t af[4], bf[4];
            ldsm_x4(af, left + (mt * 16 + (lane & 15)) * LDK + ks * 16 + (lane >> 4) * 8);
            ldsm_x4(bf, sk + (kb * 16 + (lane & 7) + (lane >> 4) * 8) * LDK + ks * 16 + ((lane >> 3) & 1) * 8);
            mma16816(p[0], af, bf[0], bf[1]);
            mma16816(p[1], af, bf[2], bf[3]);
        }
        const int ta = mt * 16 + (lane >> 2), s0 = kb * 16 + (lane & 3) * 2;
        const float* row = is_w ? srq : srk;
        float La[2] = {sL[ta], sL[ta + 8]}, fa[2] = {row[ta], row[ta + 8]};
        if (!is_w) { fa[0] *= sb[ta]; fa[1] *= sb[ta + 8]; }
#pragma unroll
        for (int b = 0; b < 2; ++b) {
            const int s = s0 + b * 8;
            const float2 Ls = *reinterpret_cast<const float2*>(sL + s), fs = *reinterpret_cast<const float2*>(srk + s);
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int t = ta + half * 8, seen = t + (is_w ? 1 : 0);
                const float x = s < seen ? p[b][half * 2] * (fa[half] * fs.x * exp2f(La[half] - Ls.x)) : 0.f;
                const float y = s + 1 < seen ? p[b][half * 2 + 1] * (fa[half] * fs.y * exp2f(La[half] - Ls.y)) : 0.f;
                if (is_w) {
                    uint32_t hi, lo;
                    split_bf16(x, y, hi, lo);
                    *reinterpret_cast<uint32_t*>(wout + t * DLT + s) = hi;
                    *reinterpret_cast<uint32_t*>(wout + (DC + t) * DLT + s) = lo;
                } else {
                    *reinterpret_cast<float2*>(A + t * DAP + s) = make_float2(x, y);
                }
            }
        }
    }
    __syncthreads();
    if (warp < 4 && lane < 16) {
        const float* Ad = A + (warp * 16) * DAP + warp * 16;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float v = i == lane ? 1.f : 0.f;
#pragma unroll
            for (int m = 0; m < i; ++m) v = fmaf(-Ad[i * DAP + m], x[m], v);
            x[i] = v;
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) Ti[(warp * 16 + i) * DAP + warp * 16 + lane] = x[i];
    }
    __syncthreads();
    // x += row (16) * mat (16 x 4 columns)
    auto mac = [](float (&x)[4], const float* row, const float* mat, int ld) {
#pragma unroll
        for (int m = 0; m < 16; m += 4) {
            const float4 w = *reinterpret_cast<const float4*>(row + m);
            const float wv[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float4 b = *reinterpret_cast<const float4*>(mat + (m + q) * ld);
                x[0] = fmaf(wv[q], b.x, x[0]);
                x[1] = fmaf(wv[q], b.y, x[1]);
                x[2] = fmaf(wv[q], b.z, x[2]);
                x[3] = fmaf(wv[q], b.w, x[3]);
            }
        }
    };
    {   // blocks (1, 0) and (3, 2): 64 threads each
        const int i = 2 * (tid >> 6) + 1, r = (tid & 63) >> 2, c4 = (tid & 3) * 4;
        float x[4] = {0.f, 0.f, 0.f, 0.f};
        if (tid < 128) {
            mac(x, A + (i * 16 + r) * DAP + (i - 1) * 16, Ti + (i - 1) * 16 * DAP + (i - 1) * 16 + c4, DAP);
            *reinterpret_cast<float4*>(X + ((tid >> 6) * 16 + r) * DAP + c4) = make_float4(x[0], x[1], x[2], x[3]);
        } else {               // what lies above the diagonal of the two 32-row blocks
            const int j = tid - 128, b = j >> 6;
            *reinterpret_cast<float4*>(Ti + (b * 32 + ((j & 63) >> 2)) * DAP + b * 32 + 16 + c4) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
        __syncthreads();
        if (tid < 128) {
            x[0] = x[1] = x[2] = x[3] = 0.f;
            mac(x, Ti + (i * 16 + r) * DAP + i * 16, X + (tid >> 6) * 16 * DAP + c4, DAP);
            *reinterpret_cast<float4*>(Ti + (i * 16 + r) * DAP + (i - 1) * 16 + c4) = make_float4(-x[0], -x[1], -x[2], -x[3]);
        }
        __syncthreads();
    }
    {   // the 32 x 32 block below
        const int r = tid >> 3, c4 = (tid & 7) * 4;
        float x[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int m = 0; m < 32; m += 16) mac(x, A + (32 + r) * DAP + m, Ti + m * DAP + c4, DAP);
        *reinterpret_cast<float4*>(X + r * DAP + c4) = make_float4(x[0], x[1], x[2], x[3]);
        __syncthreads();
        x[0] = x[1] = x[2] = x[3] = 0.f;
#pragma unroll
        for (int m = 0; m < 32; m += 16)
            if (m <= r) mac(x, Ti + (32 + r) * DAP + 32 + m, X + m * DAP + c4, DAP);
        *reinterpret_cast<float4*>(Ti + (32 + r) * DAP + c4) = make_float4(-x[0], -x[1], -x[2], -x[3]);
        __syncthreads();
    }
    bf16* out = chunk_matrix(cc.solve, a, ch, h);
#pragma unroll
    for (int i = tid; i < DC * DC / 4; i += 256) {
        const int rr = i / (DC / 4), q = i % (DC / 4) * 4;
        put_split(out + rr * DLT + q, out + (DC + rr) * DLT + q, q >> 4 > rr >> 4 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(Ti + rr * DAP + q));
    }
    pdl_launch_dependents();
}

// The state over the chunks of a segment: a block keeps DV columns of one head's state in its accumulators.  Per chunk eight warps form the products
// with the keys (S^T k of all tokens), solve the triangular system, and update the state; warp 0 brings the next chunk's operands and stores the
// state the chunk starts from meanwhile.
template <int DP>
struct DeltaStateCfg {
    static constexpr int LDK = DP + 8;
    static constexpr size_t SMEM = (size_t)(2 * DC * LDK + 4 * DC * DLT + 2 * DC * DLV + 2 * DP * DLV + 4 * DC * DLV) * 2 + 2 * DC * 16;
};
__device__ __forceinline__ void state_barrier() { asm volatile("bar.sync 1, 288;" ::: "memory"); }
template <int DP>
__global__ void __launch_bounds__(288, 2) delta_chunk_state_kernel(const DeltaArgs a, const DeltaChunks cc) {
    constexpr int LDK = DP + 8, MT = DP / 16, WN = 8 / MT, NT = DV / 8 / WN;
    extern __shared__ __align__(16) uint8_t dc_smem[];
    bf16* sk = reinterpret_cast<bf16*>(dc_smem);          // [2][DC][LDK]
    bf16* sT = sk + 2 * DC * LDK;                         // [2][part][DC][DLT]
    bf16* sv = sT + 4 * DC * DLT;                         // [2][DC][DLV]
    bf16* sS = sv + 2 * DC * DLV;                         // [part][DP][DLV]
    bf16* sr = sS + 2 * DP * DLV;                         // [part][DC][DLV]
    bf16* su = sr + 2 * DC * DLV;                         // [part][DC][DLV]
    float4* sg = reinterpret_cast<float4*>(su + 2 * DC * DLV);      // [2][DC]
    const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) - 1, g = lane >> 2, c2 = (lane & 3) * 2;
    const int v0 = blockIdx.x * DV, h = blockIdx.y, seg = blockIdx.z;
    pdl_wait();
    const int first = cc.first[seg], last = cc.first[seg + 1], lo = a.seg[2 * seg], hi = a.seg[2 * seg + 1];
    if (warp < 0) {
        const int ncol = min(DV, a.V - v0);
        for (int ch = first; ch <= last; ++ch) {          // (one step ahead of the other warps)
            const int b = (ch - first) & 1, t0 = lo + (ch - first) * DC;
            if (ch < last) {
                copy_pieces<DC * LDK / 8, 32>(sk + b * DC * LDK, chunk_keys<DP>(a, cc, ch, h));
                copy_pieces<2 * DC * DLT / 8, 32>(sT + b * 2 * DC * DLT, chunk_matrix(cc.solve, a, ch, h));
                copy_pieces<DC, 32>(sg + b * DC, chunk_gates(a, cc, ch, h));
                chunk_tile<bf16, DC, DV, 32>(a.v, a.ldv, (size_t)h * a.V + v0, t0, min(DC, hi - t0), ncol, 0, sv + b * DC * DLV);
                cp_commit();
            }
            if (ch > first) {
                uint4* out = reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(cc.states) + chunk_slice(a, ch - 1, h, blockIdx.x) * 2 * DP * DV);
#pragma unroll 8
                for (int i = lane; i < 2 * DP * DV / 8; i += 32) out[i] = *reinterpret_cast<const uint4*>(sS + (i >> 1) * DLV + (i & 1) * 8);
                state_barrier();
                state_barrier();
            }
            cp_wait<0>();
            if (ch < last) state_barrier();
        }
        pdl_launch_dependents();
        return;
    }
    const int smt = warp % MT, sn0 = (warp / MT) * NT;
    float S[NT][4];
    float* st = a.state + ((size_t)a.seg_slot[seg] * a.H + h) * a.D * a.V;
    const bool fresh = a.pos[lo] == 0;
    auto each_state = [&](auto f) {
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = smt * 16 + g + (e >> 1) * 8, v = v0 + (sn0 + j) * 8 + c2 + (e & 1);
                f(S[j][e], d < a.D && v < a.V, st + (size_t)d * a.V + v);
            }
    };
    each_state([&](float& s, bool ok, const float* p) { s = ok && !fresh ? *p : 0.f; });
    const int mt = warp & 3, nt = warp >> 2, row = mt * 16 + g, col = nt * 8 + c2;              // this warp's 16 tokens x 8 columns
    bf16* uout = reinterpret_cast<bf16*>(cc.u) + chunk_slice(a, first, h, blockIdx.x) * 2 * DC * DV + row * DV + col;
    const size_t ustep = chunk_slice(a, 1, 0, 0) * 2 * DC * DV;
    for (int ch = first; ch < last; ++ch, uout += ustep) {
        const int b = (ch - first) & 1;
        const bf16* ck = sk + b * DC * LDK;
        const bf16* cT = sT + b * 2 * DC * DLT;
        const float4* cg = sg + b * DC;
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                uint32_t x, y;
                split_bf16(S[j][e], S[j][e + 1], x, y);
                bf16* p = sS + (smt * 16 + g + (e >> 1) * 8) * DLV + (sn0 + j) * 8 + c2;
                *reinterpret_cast<uint32_t*>(p) = x;
                *reinterpret_cast<uint32_t*>(p + DP * DLV) = y;
            }
        state_barrier();
        {   // r = beta (v - decay S^T k)
            float xh[2][4] = {}, xl[2][4] = {};
#pragma unroll
            for (int ks = 0; ks < DP / 32; ++ks) {
                uint32_t bh[4], bl[4];
                ldsm_x4_t(bh, sS + (ks * 32 + lane) * DLV + nt * 8);
                ldsm_x4_t(bl, sS + (DP + ks * 32 + lane) * DLV + nt * 8);
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    uint32_t af[4];
                    ldsm_x4(af, ck + (mt * 16 + (lane & 15)) * LDK + (ks * 2 + j) * 16 + (lane >> 4) * 8);
                    mma16816(xh[j], af, bh[2 * j], bh[2 * j + 1]);
                    mma16816(xl[j], af, bl[2 * j], bl[2 * j + 1]);
                }
            }
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int o = (row + half * 8) * DLV + col;
                const float2 gt = *reinterpret_cast<const float2*>(cg + row + half * 8), v = bf2_to_f2(*reinterpret_cast<const uint32_t*>(sv + b * DC * DLV + o));
                const float x = (xh[0][2 * half] + xh[1][2 * half]) + (xl[0][2 * half] + xl[1][2 * half]);
                const float y = (xh[0][2 * half + 1] + xh[1][2 * half + 1]) + (xl[0][2 * half + 1] + xl[1][2 * half + 1]);
                uint32_t p, q;
                split_bf16(fmaf(gt.x, v.x, -gt.y * x), fmaf(gt.x, v.y, -gt.y * y), p, q);
                *reinterpret_cast<uint32_t*>(sr + o) = p;
                *reinterpret_cast<uint32_t*>(sr + DC * DLV + o) = q;
            }
        }
        state_barrier();
        {   // u = T r
            float u[2][3][4] = {};
#pragma unroll
            for (int ks = 0; ks < 2; ++ks) {
                if (ks > mt >> 1) break;
                uint32_t bh[4], bl[4];
                ldsm_x4_t(bh, sr + (ks * 32 + lane) * DLV + nt * 8);
                ldsm_x4_t(bl, sr + (DC + ks * 32 + lane) * DLV + nt * 8);
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    uint32_t ah[4], al[4];
                    const bf16* p = cT + (mt * 16 + (lane & 15)) * DLT + (ks * 2 + j) * 16 + (lane >> 4) * 8;
                    ldsm_x4(ah, p);
                    ldsm_x4(al, p + DC * DLT);
                    mma16816(u[j][0], ah, bh[2 * j], bh[2 * j + 1]);
                    mma16816(u[j][1], ah, bl[2 * j], bl[2 * j + 1]);
                    mma16816(u[j][2], al, bh[2 * j], bh[2 * j + 1]);
                }
            }
            float x[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) x[e] = (u[0][0][e] + u[1][0][e]) + ((u[0][1][e] + u[1][1][e]) + (u[0][2][e] + u[1][2][e]));
            uint32_t p, q;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int o = (row + half * 8) * DLV + col;
                const float w = cg[row + half * 8].z;
                split_bf16(x[2 * half] * w, x[2 * half + 1] * w, p, q);
                *reinterpret_cast<uint32_t*>(su + o) = p;
                *reinterpret_cast<uint32_t*>(su + DC * DLV + o) = q;
            }
            state_barrier();
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                split_bf16(x[2 * half], x[2 * half + 1], p, q);
                *reinterpret_cast<uint32_t*>(uout + half * 8 * DV) = p;
                *reinterpret_cast<uint32_t*>(uout + (DC + half * 8) * DV) = q;
            }
        }
        {   // S = decay S + sum k u^T
            const float f = cg[0].w;
            float rest[NT][2][4] = {};
#pragma unroll
            for (int j = 0; j < NT; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[j][e] *= f;
#pragma unroll
            for (int ks = 0; ks < DC / 32; ++ks) {
                uint32_t af[2][4];
#pragma unroll
                for (int i = 0; i < 2; ++i) ldsm_x4_t(af[i], ck + (ks * 32 + i * 16 + (lane & 7) + (lane >> 4) * 8) * LDK + smt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    uint32_t bh[4], bl[4];
                    ldsm_x4_t(bh, su + (ks * 32 + lane) * DLV + (sn0 + j) * 8);
                    ldsm_x4_t(bl, su + (DC + ks * 32 + lane) * DLV + (sn0 + j) * 8);
                    mma16816(S[j], af[0], bh[0], bh[1]);
                    mma16816(rest[j][0], af[1], bh[2], bh[3]);
                    mma16816(rest[j][1], af[0], bl[0], bl[1]);
                    mma16816(rest[j][1], af[1], bl[2], bl[3]);
                }
            }
#pragma unroll
            for (int j = 0; j < NT; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[j][e] += rest[j][0][e] + rest[j][1][e];
        }
    }
    pdl_launch_dependents();
    each_state([&](float& s, bool ok, float* p) { if (ok) *p = s; });
}

// Outputs of a chunk, 64 columns: what the state a chunk starts from answers to the queries, and the weighted writes.  A warp takes 16 queries and
// half of the columns.
constexpr int DO = 64, DLO = DO + 8;
template <int DP>
struct DeltaOutCfg {
    static constexpr int LDK = DP + 8;
    static constexpr size_t SMEM = (size_t)(DC * LDK + 2 * DC * DLT + 2 * DP * DLO + 2 * DC * DLO) * 2 + DC * 4;
};
template <int DP>
__global__ void __launch_bounds__(256, 2) delta_chunk_out_kernel(const DeltaArgs a, const DeltaChunks cc) {
    constexpr int LDK = DP + 8;
    extern __shared__ __align__(16) uint8_t dc_smem[];
    bf16* sq = reinterpret_cast<bf16*>(dc_smem);          // [DC][LDK]
    bf16* sw = sq + DC * LDK;                             // [part][DC][DLT]
    bf16* sS = sw + 2 * DC * DLT;                         // [part][DP][DLO]
    bf16* su = sS + 2 * DP * DLO;                         // [part][DC][DLO]
    float* se = reinterpret_cast<float*>(su + 2 * DC * DLO);        // [DC]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, mt = warp & 3, hf = warp >> 2, ch = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * DO;
    pdl_wait();
    const int t0 = cc.chunk[2 * ch], n = cc.chunk[2 * ch + 1], ncol = min(DO, a.V - v0), slices = (ncol + DV - 1) / DV;
    const size_t sl = chunk_slice(a, ch, h, v0 / DV);
    {   // 16-column slices, side by side; the two halves of a group of threads take the halves of a row
        const uint4* S = reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(cc.states) + sl * 2 * DP * DV) + tid;
        bf16* dst = sS + (tid >> 1) * DLO + (tid & 1) * 8;
#pragma unroll
        for (int s = 0; s < DO / DV; ++s)
            if (s < slices)
#pragma unroll
                for (int i = 0; i < 4 * DP / 256; ++i) cp_async16(dst + i * 128 * DLO + s * DV, S + s * 4 * DP + i * 256, true);
    }
    chunk_tile<bf16, DC, DP, 256>(a.q, a.ldq, (size_t)(h / a.hpg) * a.D, t0, n, a.D, 0, sq);
    cp_commit();
    {
        const uint4* U = reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(cc.u) + sl * 2 * DC * DV) + tid;
        bf16* dst = su + (tid >> 1) * DLO + (tid & 1) * 8;
#pragma unroll
        for (int s = 0; s < DO / DV; ++s)
            if (s < slices) cp_async16(dst + s * DV, U + s * 4 * DC, true);
    }
    copy_pieces<2 * DC * DLT / 8, 256>(sw, chunk_matrix(cc.weights, a, ch, h));
    if (tid < DC / 4) cp_async16(se + tid * 4, chunk_gates(a, cc, ch, h) + 4 * DC + tid * 4, true);
    cp_commit();
    cp_wait<1>();
    __syncthreads();
    const bool mine = mt * 16 < n && hf * 32 < ncol;
    float acc[2][2][4] = {};
    if (mine) {
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) {
            uint32_t af[4];
            ldsm_x4(af, sq + (mt * 16 + (lane & 15)) * LDK + ks * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const bf16* p = sS + (ks * 16 + (lane & 15)) * DLO + hf * 32 + j * 16 + (lane >> 4) * 8;
                uint32_t bh[4], bl[4];
                ldsm_x4_t(bh, p);
                ldsm_x4_t(bl, p + DP * DLO);
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    mma16816(acc[j][b], af, bh[2 * b], bh[2 * b + 1]);
                    mma16816(acc[j][b], af, bl[2 * b], bl[2 * b + 1]);
                }
            }
        }
    }
    cp_wait<0>();
    __syncthreads();
    pdl_launch_dependents();
    if (!mine) return;
    const int row = mt * 16 + (lane >> 2);
    const float e0 = se[row], e1 = se[row + 8];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int b = 0; b < 2; ++b) { acc[j][b][0] *= e0; acc[j][b][1] *= e0; acc[j][b][2] *= e1; acc[j][b][3] *= e1; }
#pragma unroll
    for (int kb = 0; kb < DC / 16; ++kb) {
        if (kb > mt) break;
        uint32_t ah[4], al[4];
        const bf16* p = sw + (mt * 16 + (lane & 15)) * DLT + kb * 16 + (lane >> 4) * 8;
        ldsm_x4(ah, p);
        ldsm_x4(al, p + DC * DLT);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const bf16* q = su + (kb * 16 + (lane & 15)) * DLO + hf * 32 + j * 16 + (lane >> 4) * 8;
            uint32_t bh[4], bl[4];
            ldsm_x4_t(bh, q);
            ldsm_x4_t(bl, q + DC * DLO);
#pragma unroll
            for (int b = 0; b < 2; ++b) {
                mma16816(acc[j][b], ah, bh[2 * b], bh[2 * b + 1]);
                mma16816(acc[j][b], ah, bl[2 * b], bl[2 * b + 1]);
                mma16816(acc[j][b], al, bh[2 * b], bh[2 * b + 1]);
            }
        }
    }
    const bool pair = ((a.V | a.ldo) & 1) == 0;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int t = row + half * 8;
        if (t >= n) break;
        float* o = a.out + (size_t)(t0 + t) * a.ldo + h * a.V + v0;
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int b = 0; b < 2; ++b) {
                const int c = hf * 32 + j * 16 + b * 8 + (lane & 3) * 2;
                if (c >= ncol) continue;
                const float x = acc[j][b][half * 2], y = acc[j][b][half * 2 + 1];
                if (pair) {
                    *reinterpret_cast<float2*>(o + c) = make_float2(x, y);
                } else {
                    o[c] = x;
                    if (c + 1 < ncol) o[c + 1] = y;
                }
            }
    }
}

template <int DP>
static int launch_delta_chunks(const DeltaArgs& a, const DeltaChunks& c, cudaStream_t s) {
    constexpr size_t sm1 = DeltaSolveCfg<DP>::SMEM, sm2 = DeltaStateCfg<DP>::SMEM, sm3 = DeltaOutCfg<DP>::SMEM;
    static_assert(sm1 <= 113 * 1024 && sm2 <= 113 * 1024 && sm3 <= 113 * 1024, "chunk staging, two blocks to an SM");
    auto k1 = delta_chunk_solve_kernel<DP>;
    auto k2 = delta_chunk_state_kernel<DP>;
    auto k3 = delta_chunk_out_kernel<DP>;
    if (first_use_on_device((const void*)k1)) DLP_CHECK_CUDA(cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm1));
    if (first_use_on_device((const void*)k2)) DLP_CHECK_CUDA(cudaFuncSetAttribute(k2, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm2));
    if (first_use_on_device((const void*)k3)) DLP_CHECK_CUDA(cudaFuncSetAttribute(k3, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm3));
    DLP_CHECK_CUDA(launch_pdl(k1, dim3(c.n_chunks, a.H), dim3(256), sm1, s, a, c));
    DLP_CHECK_CUDA(launch_pdl(k2, dim3((a.V + DV - 1) / DV, a.H, a.n_seg), dim3(288), sm2, s, a, c));
    DLP_CHECK_CUDA(launch_pdl(k3, dim3(c.n_chunks, a.H, (a.V + DO - 1) / DO), dim3(256), sm3, s, a, c));
    return 0;
}
int delta_chunked(const DeltaArgs& a, const DeltaChunks& c, cudaStream_t s) {
    const int rc = check_delta(a, "delta_chunked");
    if (rc) return rc;
    DLP_REQUIRE(c.chunk && c.first && c.states && c.keys && c.solve && c.weights && c.u && c.gates && c.n_chunks > 0, "delta_chunked: no chunk table");
    DLP_REQUIRE(!a.rows_f32 && a.D <= 128 && (a.V + DO - 1) / DO <= 65535, "delta_chunked: bf16 rows, state of %d x %d", a.D, a.V);
    DLP_REQUIRE(((reinterpret_cast<uintptr_t>(c.states) | reinterpret_cast<uintptr_t>(c.keys) | reinterpret_cast<uintptr_t>(c.solve) | reinterpret_cast<uintptr_t>(c.weights) |
                  reinterpret_cast<uintptr_t>(c.u) | reinterpret_cast<uintptr_t>(c.gates)) & 15) == 0, "delta_chunked: workspace alignment");
    return a.D <= 64 ? launch_delta_chunks<64>(a, c, s) : launch_delta_chunks<128>(a, c, s);
}

}  // namespace dlp
