// Linear recurrences with one decay per head and token (constant decays: lightning attention; step sizes: Mamba-2), and the short
// convolution in front of the latter.
//
//   S_t = f_t S_{t-1} + dt_t k_t v_t^T,   o_t = S_t^T q_t (+ skip v_t)
//
//   ssd_decode_kernel   one token per sequence: the state is read once, in 16-byte pieces, requested before the dependency wait; the
//                       convolution of the token (its inputs come out of the ring) is part of the launch
//   ssd_scan            token by token (short portions, fp32 storage, any size): layers_scan.cuh
//   ssd_chunk_state / chunk_scan / ssd_chunk_out   128-token chunks on the tensor cores, all chunks at once but for the scan between them
//   conv_rows_kernel    convolution and silu of whole portions
//
// Chunks: with L the cumulative log decay inside a chunk,
//   U = sum_s exp(L_end - L_s) dt_s k_s v_s^T          o_t = exp(L_t) S_start^T q_t + sum_{s <= t} exp(L_t - L_s) dt_s (q_t . k_s) v_s
// Exponents are never positive.  q, k and v (projections behind their activation) are bf16 operands; decays, step sizes, token weights and
// states are fp32 and enter the tensor cores as two bf16 parts (value and remainder).
#include "layers_chunks.cuh"
#include "layers_scan.cuh"

namespace dlp {

__device__ __forceinline__ float ssd_step(const SsdArgs& a, int t, int h) { return a.dt ? softplus_exact(a.dt[(size_t)t * a.lddt + h] + a.dt_bias[h]) : 1.f; }

// ---- token by token ------------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ void scan_channel(const SsdArgs& a, int t, int h, int d, float& q, float& f, float& k) {
    const int g = h / a.hpg;
    const float dt = ssd_step(a, t, h);
    q = mix_row(a.q, a.rows_f32, a.act, (size_t)t * a.ldq + g * a.D + d);
    k = mix_row(a.k, a.rows_f32, a.act, (size_t)t * a.ldk + g * a.D + d) * dt;
    f = a.dt ? expf(a.log_decay[h] * dt) : a.decay[h];
}
__device__ __forceinline__ float scan_value(const SsdArgs& a, int t, int h, int c) { return mix_row(a.v, a.rows_f32, a.act, (size_t)t * a.ldv + h * a.V + c); }
__device__ __forceinline__ float scan_out(const SsdArgs& a, int h, float o, float v) { return a.skip ? fmaf(a.skip[h], v, o) : o; }

static int check_ssd(const SsdArgs& a, const char* who) {
    DLP_REQUIRE(a.q && a.k && a.v && a.log_decay && (a.dt ? a.dt_bias != nullptr : a.decay != nullptr) && a.state && a.seg && a.seg_slot && a.pos && a.out, "%s: null argument", who);
    DLP_REQUIRE(a.H > 0 && a.H <= 65535 && a.D > 0 && a.V > 0 && a.n_seg > 0 && a.n_seg <= 65535 && a.hpg > 0 && a.H % a.hpg == 0, "%s: bad shape (%d heads of %d x %d, %d per group)", who,
                a.H, a.D, a.V, a.hpg);
    return 0;
}
int ssd_scan(const SsdArgs& a, cudaStream_t s) {
    const int rc = check_ssd(a, "ssd_scan");
    return rc ? rc : recurrence_scan(a, "ssd_scan", s);
}

// ---- one token per sequence ------------------------------------------------------------------------------------------------------------
// A block takes 32 columns of one head's state: eight lanes cover the columns (four each), 32 row slots of NR rows each.
template <int NR, bool CONV>
__global__ void __launch_bounds__(256) ssd_decode_kernel(const SsdArgs a, const ConvArgs cv) {
    constexpr int COLS = 32;
    extern __shared__ __align__(16) float sd_smem[];
    float* sq = sd_smem;                    // [D]
    float* sk = sq + a.D;                   // [D]
    float* sv = sk + a.D;                   // [COLS]
    __shared__ __align__(16) float red[8][COLS];
    const int tid = threadIdx.x, c0 = (tid & 7) * 4, rs = tid >> 3, h = blockIdx.y, v0 = blockIdx.x * COLS, g = h / a.hpg;
    // (segments, positions and states were written at least two launches back)
    const int t = a.seg[2 * blockIdx.z], slot = a.seg_slot[blockIdx.z], pos = a.pos[t];
    float* st = a.state + ((size_t)slot * a.H + h) * a.D * a.V + v0 + c0;
    float4 S[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = rs + 32 * i;
        S[i] = pos > 0 && d < a.D && v0 + c0 < a.V ? *reinterpret_cast<const float4*>(st + (size_t)d * a.V) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_wait();
    const float dt = ssd_step(a, t, h), f = a.dt ? expf(a.log_decay[h] * dt) : a.decay[h];
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
                x = part == 0 ? mix_row(a.q, a.rows_f32, a.act, (size_t)t * a.ldq + col) : part == 1 ? mix_row(a.k, a.rows_f32, a.act, (size_t)t * a.ldk + col)
                                                                                                      : mix_row(a.v, a.rows_f32, a.act, (size_t)t * a.ldv + col);
            }
        }
        sd_smem[i] = part == 1 ? x * dt : x;
    }
    __syncthreads();
    const float v[4] = {sv[c0], sv[c0 + 1], sv[c0 + 2], sv[c0 + 3]};
    float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = rs + 32 * i;
        if (d < a.D) {
            const float k = sk[d], q = sq[d];
            S[i] = make_float4(fmaf(f, S[i].x, k * v[0]), fmaf(f, S[i].y, k * v[1]), fmaf(f, S[i].z, k * v[2]), fmaf(f, S[i].w, k * v[3]));
            o[0] = fmaf(q, S[i].x, o[0]);
            o[1] = fmaf(q, S[i].y, o[1]);
            o[2] = fmaf(q, S[i].z, o[2]);
            o[3] = fmaf(q, S[i].w, o[3]);
        }
    }
    pdl_launch_dependents();
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        o[e] += __shfl_xor_sync(0xffffffffu, o[e], 8);
        o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
    }
    if ((tid & 31) < 8) *reinterpret_cast<float4*>(&red[tid >> 5][c0]) = make_float4(o[0], o[1], o[2], o[3]);
    __syncthreads();
    if (tid < COLS && v0 + tid < a.V) {
        float x = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) x += red[w][tid];
        a.out[(size_t)t * a.ldo + h * a.V + v0 + tid] = scan_out(a, h, x, sv[tid]);
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = rs + 32 * i;
        if (d < a.D && v0 + c0 < a.V) *reinterpret_cast<float4*>(st + (size_t)d * a.V) = S[i];
    }
}

template <int NR>
static int launch_decode(const SsdArgs& a, const ConvArgs* cv, cudaStream_t s) {
    const dim3 grid((a.V + 31) / 32, a.H, a.n_seg);
    const size_t smem = (size_t)(2 * a.D + 32) * 4;
    if (cv) DLP_CHECK_CUDA(launch_pdl(ssd_decode_kernel<NR, true>, grid, dim3(256), smem, s, a, *cv));
    else DLP_CHECK_CUDA(launch_pdl(ssd_decode_kernel<NR, false>, grid, dim3(256), smem, s, a, ConvArgs()));
    return 0;
}
int ssd_decode(const SsdArgs& a, const ConvArgs* cv, cudaStream_t s) {
    const int rc = check_ssd(a, "ssd_decode");
    if (rc) return rc;
    DLP_REQUIRE(a.D <= 256 && a.V % 4 == 0 && (reinterpret_cast<uintptr_t>(a.state) & 15) == 0, "ssd_decode: state of %d x %d", a.D, a.V);
    DLP_REQUIRE(!cv || (cv->x && cv->w && cv->ring && cv->taps >= 1 && a.rows_f32 && a.ldq == cv->ldx && a.ldk == cv->ldx && a.ldv == cv->ldx), "ssd_decode: convolution");
    if (a.D <= 64) return launch_decode<2>(a, cv, s);
    if (a.D <= 128) return launch_decode<4>(a, cv, s);
    return launch_decode<8>(a, cv, s);
}

// ---- convolution of whole portions -------------------------------------------------------------------------------------------------------
// A thread takes one channel of CONV_TILE tokens.  The thread with a segment's first tokens is the only one that touches the ring: it has read
// what it needs before it leaves the segment's last inputs there.
constexpr int CONV_TILE = 32;
template <typename OT, int TAPS>      // TAPS 0: any number up to CONV_TILE
__global__ void __launch_bounds__(128) conv_rows_kernel(const ConvArgs cv, const int* seg, const int* seg_slot, const int* pos, OT* out, int ldo) {
    pdl_wait();
    const int c = blockIdx.x * 128 + threadIdx.x, lo = seg[2 * blockIdx.z], hi = seg[2 * blockIdx.z + 1], t0 = lo + blockIdx.y * CONV_TILE;
    const int n = min(CONV_TILE, hi - t0), taps = TAPS > 0 ? TAPS : cv.taps;
    if (c < cv.channels && n > 0) {
        const float* x = cv.x + c;
        float* ring = cv.ring + (size_t)seg_slot[blockIdx.z] * taps * cv.channels + c;
        const int p0 = pos[lo];
        auto input = [&](int t) {              // t < lo: an input of an earlier portion
            if (t >= lo) return x[(size_t)t * cv.ldx];
            const int p = p0 + t - lo;
            return p >= 0 ? ring[(size_t)(p % taps) * cv.channels] : 0.f;
        };
        const float b = cv.b ? cv.b[c] : 0.f;
        if (TAPS > 0) {
            float w[TAPS > 0 ? TAPS : 1], win[TAPS > 0 ? TAPS : 1];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[j] = cv.w[(size_t)j * cv.channels + c];
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) win[j + 1] = input(t0 - (TAPS - 1) + j);
#pragma unroll 8
            for (int i = 0; i < n; ++i) {
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) win[j] = win[j + 1];
                win[TAPS - 1] = x[(size_t)(t0 + i) * cv.ldx];
                float y = b;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) y = fmaf(w[j], win[j], y);
                out[(size_t)(t0 + i) * ldo + c] = Act<OT>::from_f(sizeof(OT) == 2 ? silu_fast(y) : silu_exact(y));
            }
        } else {
            for (int i = 0; i < n; ++i) {
                float y = b;
                for (int j = 0; j < taps; ++j) y = fmaf(cv.w[(size_t)j * cv.channels + c], input(t0 + i - (taps - 1) + j), y);
                out[(size_t)(t0 + i) * ldo + c] = Act<OT>::from_f(sizeof(OT) == 2 ? silu_fast(y) : silu_exact(y));
            }
        }
        if (t0 == lo)
            for (int t = max(lo, hi - taps); t < hi; ++t) ring[(size_t)((p0 + t - lo) % taps) * cv.channels] = x[(size_t)t * cv.ldx];
    }
    pdl_launch_dependents();
}
template <typename OT>
static int launch_conv(const ConvArgs& c, const int* seg, const int* seg_slot, const int* pos, int n_seg, int longest, OT* out, int ldo, cudaStream_t s) {
    const dim3 grid((c.channels + 127) / 128, (longest + CONV_TILE - 1) / CONV_TILE, n_seg);
    auto kern = c.taps == 4 ? conv_rows_kernel<OT, 4> : c.taps == 3 ? conv_rows_kernel<OT, 3> : c.taps == 2 ? conv_rows_kernel<OT, 2> : conv_rows_kernel<OT, 0>;
    DLP_CHECK_CUDA(launch_pdl(kern, grid, dim3(128), 0, s, c, seg, seg_slot, pos, out, ldo));
    return 0;
}
int conv_rows(const ConvArgs& c, const int* seg, const int* seg_slot, const int* pos, int n_seg, int longest, void* out, int ldo, int f32, cudaStream_t s) {
    DLP_REQUIRE(c.x && c.w && c.ring && seg && seg_slot && pos && out && n_seg > 0 && n_seg <= 65535 && longest > 0 && longest <= 65535 * CONV_TILE, "conv_rows: bad argument");
    DLP_REQUIRE(c.taps >= 1 && c.taps <= CONV_TILE && c.channels > 0 && c.ldx >= c.channels && ldo >= c.channels, "conv_rows: %d taps (at most %d) of %d channels", c.taps, CONV_TILE,
                c.channels);
    return f32 ? launch_conv(c, seg, seg_slot, pos, n_seg, longest, (float*)out, ldo, s) : launch_conv(c, seg, seg_slot, pos, n_seg, longest, (__nv_bfloat16*)out, ldo, s);
}

// ---- chunks --------------------------------------------------------------------------------------------------------------------------------
constexpr int SC = SSD_CHUNK, SSD_NTH = 256, SSD_VP = 64, SSD_LDV = SSD_VP + 8;

// step sizes and cumulative log2 decays of a chunk (tokens past its end: no step, no decay); ends with a barrier
__device__ __forceinline__ void ssd_decays(const SsdArgs& a, int t0, int n, int h, float* sdt, float* sL, float* carry) {
    static_assert(SC == 128, "one warp per 32 tokens");
    const int s = threadIdx.x, lane = s & 31, warp = s >> 5;
    float dt = 0.f, L = 0.f;
    if (s < SC) {
        dt = s < n ? ssd_step(a, t0 + s, h) : 0.f;
        L = a.log_decay[h] * dt * 1.4426950408889634f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(0xffffffffu, L, o);
            if (lane >= o) L += x;
        }
        if (lane == 31) carry[warp] = L;
    }
    __syncthreads();
    if (s < SC) {
        for (int w = 0; w < warp; ++w) L += carry[w];
        sdt[s] = dt;
        sL[s] = L;
    }
    __syncthreads();
}

// U = k^T (weights * v): the weights go to the values, which are the narrower operand
template <int DP>
struct SsdStateCfg {
    static constexpr int LDK = DP + 8;
    static constexpr size_t SMEM = (size_t)(SC * LDK + 2 * SC * SSD_LDV) * 2;
};
template <int DP, typename RT>
__global__ void __launch_bounds__(SSD_NTH) ssd_chunk_state_kernel(const SsdArgs a, const ScanChunks cc) {
    constexpr int LDK = DP + 8, LDV = SSD_LDV, CG = DP == 64 ? 2 : 1, MTW = DP == 256 ? 2 : 1, NP = SSD_VP / 16 / CG;
    extern __shared__ __align__(16) uint8_t ss_smem[];
    __shared__ float sdt[SC], sL[SC], carry[SC / 32];
    __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(ss_smem);        // [SC][LDK]
    __nv_bfloat16* vhi = sk + SC * LDK;                                   // [SC][LDV]
    __nv_bfloat16* vlo = vhi + SC * LDV;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, ch = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * SSD_VP;
    pdl_wait();
    const int t0 = cc.chunk[2 * ch], n = cc.chunk[2 * ch + 1];
    chunk_tile<RT, SC, DP, SSD_NTH>(a.k, a.ldk, (size_t)(h / a.hpg) * a.D, t0, n, a.D, a.act, sk);
    cp_commit();
    ssd_decays(a, t0, n, h, sdt, sL, carry);
    const float end = sL[SC - 1];
    chunk_rows<RT, SC, SSD_VP, SSD_NTH>(reinterpret_cast<const RT*>(a.v) + (size_t)t0 * a.ldv + h * a.V + v0, a.ldv, n, min(SSD_VP, a.V - v0), a.act, [&](int s, int c, float4 x) {
        const float w = exp2f(end - sL[s]) * sdt[s];
        put_split(vhi + s * LDV + c, vlo + s * LDV + c, make_float4(x.x * w, x.y * w, x.z * w, x.w * w));
    });
    if (threadIdx.x == 0 && blockIdx.z == 0) cc.decay[(size_t)ch * a.H + h] = exp2f(end);
    cp_wait<0>();
    __syncthreads();
    const int cg = DP == 64 ? warp >> 2 : 0;
    float* u = cc.states + ((size_t)ch * a.H + h) * a.D * a.V;
#pragma unroll
    for (int m = 0; m < MTW; ++m) {
        const int mt = DP == 64 ? warp & 3 : warp + 8 * m;
        float acc[NP][2][4] = {};
#pragma unroll 4
        for (int ks = 0; ks < SC / 16; ++ks) {
            uint32_t af[4];
            ldsm_x4_t(af, sk + (ks * 16 + (lane & 7) + (lane >> 4) * 8) * LDK + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int j = 0; j < NP; ++j) {
                const int o = (ks * 16 + (lane & 15)) * LDV + (cg * NP + j) * 16 + (lane >> 4) * 8;
                uint32_t bh[4], bl[4];
                ldsm_x4_t(bh, vhi + o);
                ldsm_x4_t(bl, vlo + o);
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    mma16816(acc[j][b], af, bh[2 * b], bh[2 * b + 1]);
                    mma16816(acc[j][b], af, bl[2 * b], bl[2 * b + 1]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < NP; ++j)
#pragma unroll
            for (int b = 0; b < 2; ++b)
#pragma unroll
                for (int e = 0; e < 4; e += 2) {
                    const int d = mt * 16 + (lane >> 2) + (e >> 1) * 8, v = v0 + (cg * NP + j) * 16 + b * 8 + (lane & 3) * 2;
                    if (d >= a.D) continue;
                    if (a.V % 2 == 0) {
                        if (v < a.V) *reinterpret_cast<float2*>(u + (size_t)d * a.V + v) = make_float2(acc[j][b][e], acc[j][b][e + 1]);
                    } else {
                        if (v < a.V) u[(size_t)d * a.V + v] = acc[j][b][e];
                        if (v + 1 < a.V) u[(size_t)d * a.V + v + 1] = acc[j][b][e + 1];
                    }
                }
    }
    pdl_launch_dependents();
}

// The state takes the place of the queries, which each warp keeps in registers.
template <int DP>
struct SsdOutCfg {
    static constexpr int LDK = DP + 8;
    static constexpr int Q_ELEMS = SC * LDK, S_ELEMS = 2 * DP * SSD_LDV, QS_ELEMS = Q_ELEMS > S_ELEMS ? Q_ELEMS : S_ELEMS;
    static constexpr size_t SMEM = (size_t)(QS_ELEMS + SC * LDK + SC * SSD_LDV) * 2;
};
// Warp = 16 queries; token weights stay in registers (the accumulators of q k^T, weighted, are the operand of the product with v).
template <int DP, typename RT>
__global__ void __launch_bounds__(SSD_NTH, DP == 256 ? 1 : 2) ssd_chunk_out_kernel(const SsdArgs a, const ScanChunks cc) {
    using C = SsdOutCfg<DP>;
    constexpr int LDK = C::LDK, LDV = SSD_LDV, NP = SSD_VP / 16, SQ = DP * SSD_VP / 4 / SSD_NTH;
    extern __shared__ __align__(16) uint8_t ss_smem[];
    __shared__ float sdt[SC], sL[SC], carry[SC / 32];
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(ss_smem);        // [SC][LDK], then the state [DP][LDV] twice
    __nv_bfloat16 *shi = sq, *slo = sq + DP * LDV;
    __nv_bfloat16* sk = sq + C::QS_ELEMS;                                 // [SC][LDK]
    __nv_bfloat16* sv = sk + SC * LDK;                                    // [SC][LDV]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, cq = lane & 3, ch = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * SSD_VP;
    pdl_wait();
    const int t0 = cc.chunk[2 * ch], n = cc.chunk[2 * ch + 1], ncol = min(SSD_VP, a.V - v0);
    const size_t qk0 = (size_t)(h / a.hpg) * a.D;
    chunk_tile<RT, SC, DP, SSD_NTH>(a.q, a.ldq, qk0, t0, n, a.D, a.act, sq);
    chunk_tile<RT, SC, DP, SSD_NTH>(a.k, a.ldk, qk0, t0, n, a.D, a.act, sk);
    chunk_tile<RT, SC, SSD_VP, SSD_NTH>(a.v, a.ldv, (size_t)h * a.V + v0, t0, n, ncol, a.act, sv);
    cp_commit();
    const float* S = cc.states + ((size_t)ch * a.H + h) * a.D * a.V + v0;
    const bool s_vec = a.V % 4 == 0;
    float4 s4[SQ];
#pragma unroll
    for (int j = 0; j < SQ; ++j) {
        const int i = threadIdx.x + j * SSD_NTH, d = i / (SSD_VP / 4), c = i % (SSD_VP / 4) * 4;
        s4[j] = s_vec && d < a.D && c < ncol ? *reinterpret_cast<const float4*>(S + (size_t)d * a.V + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    ssd_decays(a, t0, n, h, sdt, sL, carry);
    cp_wait<0>();
    __syncthreads();
    const int mt = warp < 4 ? warp : 11 - warp;          // short and long rows on every scheduler
    uint32_t qf[DP / 16][4];
#pragma unroll
    for (int ks = 0; ks < DP / 16; ++ks) ldsm_x4(qf[ks], sq + (mt * 16 + (lane & 15)) * LDK + ks * 16 + (lane >> 4) * 8);
    __syncthreads();
#pragma unroll
    for (int j = 0; j < SQ; ++j) {
        const int i = threadIdx.x + j * SSD_NTH, d = i / (SSD_VP / 4), c = i % (SSD_VP / 4) * 4;
        if (!s_vec && d < a.D) {
            const float* p = S + (size_t)d * a.V + c;
            s4[j] = make_float4(c < ncol ? p[0] : 0.f, c + 1 < ncol ? p[1] : 0.f, c + 2 < ncol ? p[2] : 0.f, c + 3 < ncol ? p[3] : 0.f);
        }
        put_split(shi + d * LDV + c, slo + d * LDV + c, s4[j]);
    }
    __syncthreads();
    if (mt * 16 < n) {
        float acc[NP][2][4] = {};
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks)
#pragma unroll
            for (int j = 0; j < NP; ++j) {
                const int o = (ks * 16 + (lane & 15)) * LDV + j * 16 + (lane >> 4) * 8;
                uint32_t bh[4], bl[4];
                ldsm_x4_t(bh, shi + o);
                ldsm_x4_t(bl, slo + o);
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    mma16816(acc[j][b], qf[ks], bh[2 * b], bh[2 * b + 1]);
                    mma16816(acc[j][b], qf[ks], bl[2 * b], bl[2 * b + 1]);
                }
            }
        const float L0 = sL[mt * 16 + g], L1 = sL[mt * 16 + g + 8], e0 = exp2f(L0), e1 = exp2f(L1);
#pragma unroll
        for (int j = 0; j < NP; ++j)
#pragma unroll
            for (int b = 0; b < 2; ++b) { acc[j][b][0] *= e0; acc[j][b][1] *= e0; acc[j][b][2] *= e1; acc[j][b][3] *= e1; }
#pragma unroll 1
        for (int kb = 0; kb <= mt; ++kb) {
            float p[2][4] = {};
#pragma unroll
            for (int ks = 0; ks < DP / 16; ++ks) {
                uint32_t bf[4];
                ldsm_x4(bf, sk + (kb * 16 + (lane & 7) + (lane >> 4) * 8) * LDK + ks * 16 + ((lane >> 3) & 1) * 8);
                mma16816(p[0], qf[ks], bf[0], bf[1]);
                mma16816(p[1], qf[ks], bf[2], bf[3]);
            }
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int b = 0; b < 2; ++b) {
                float w[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int t = mt * 16 + g + (e >> 1) * 8, s = kb * 16 + b * 8 + cq * 2 + (e & 1);
                    w[e] = s <= t ? p[b][e] * (exp2f((e < 2 ? L0 : L1) - sL[s]) * sdt[s]) : 0.f;
                }
                split_bf16(w[0], w[1], hi[2 * b], lo[2 * b]);
                split_bf16(w[2], w[3], hi[2 * b + 1], lo[2 * b + 1]);
            }
#pragma unroll
            for (int j = 0; j < NP; ++j) {
                uint32_t bf[4];
                ldsm_x4_t(bf, sv + (kb * 16 + (lane & 15)) * LDV + j * 16 + (lane >> 4) * 8);
                mma16816(acc[j][0], hi, bf[0], bf[1]);
                mma16816(acc[j][1], hi, bf[2], bf[3]);
                mma16816(acc[j][0], lo, bf[0], bf[1]);
                mma16816(acc[j][1], lo, bf[2], bf[3]);
            }
        }
        const float skip = a.skip ? a.skip[h] : 0.f;
#pragma unroll
        for (int j = 0; j < NP; ++j)
#pragma unroll
            for (int b = 0; b < 2; ++b)
#pragma unroll
                for (int e = 0; e < 4; e += 2) {
                    const int t = mt * 16 + g + (e >> 1) * 8, c = j * 16 + b * 8 + cq * 2;
                    if (t >= n || v0 + c >= a.V) continue;
                    float x = acc[j][b][e], y = acc[j][b][e + 1];
                    if (a.skip) {
                        x = fmaf(skip, __bfloat162float(sv[t * LDV + c]), x);
                        y = fmaf(skip, __bfloat162float(sv[t * LDV + c + 1]), y);
                    }
                    float* o = a.out + (size_t)(t0 + t) * a.ldo + h * a.V + v0 + c;
                    if (((a.V | a.ldo) & 1) == 0) {
                        *reinterpret_cast<float2*>(o) = make_float2(x, y);
                    } else {
                        o[0] = x;
                        if (v0 + c + 1 < a.V) o[1] = y;
                    }
                }
    }
    pdl_launch_dependents();
}

template <int DP, typename RT>
static int launch_ssd_chunks(const SsdArgs& a, const ScanChunks& c, cudaStream_t s) {
    constexpr size_t sm1 = SsdStateCfg<DP>::SMEM, sm3 = SsdOutCfg<DP>::SMEM;
    static_assert(sm1 <= 227 * 1024 && sm3 <= 227 * 1024, "chunk staging");
    auto k1 = ssd_chunk_state_kernel<DP, RT>;
    auto k3 = ssd_chunk_out_kernel<DP, RT>;
    if (first_use_on_device((const void*)k1)) DLP_CHECK_CUDA(cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm1));
    if (first_use_on_device((const void*)k3)) DLP_CHECK_CUDA(cudaFuncSetAttribute(k3, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm3));
    const dim3 grid(c.n_chunks, a.H, (a.V + SSD_VP - 1) / SSD_VP);
    DLP_CHECK_CUDA(launch_pdl(k1, grid, dim3(SSD_NTH), sm1, s, a, c));
    DLP_CHECK_CUDA((launch_chunk_scan<SsdArgs, false>(a, c, s)));
    DLP_CHECK_CUDA(launch_pdl(k3, grid, dim3(SSD_NTH), sm3, s, a, c));
    return 0;
}
int ssd_chunked(const SsdArgs& a, const ScanChunks& c, cudaStream_t s) {
    const int rc = check_ssd(a, "ssd_chunked");
    if (rc) return rc;
    DLP_REQUIRE(c.chunk && c.first && c.states && c.decay && c.n_chunks > 0, "ssd_chunked: no chunk table");
    DLP_REQUIRE(a.D <= 256 && (a.V + SSD_VP - 1) / SSD_VP <= 65535, "ssd_chunked: state of %d x %d", a.D, a.V);
#define DLP_SSD_CASE(DP_) return a.rows_f32 ? launch_ssd_chunks<DP_, float>(a, c, s) : launch_ssd_chunks<DP_, __nv_bfloat16>(a, c, s)
    if (a.D <= 64) DLP_SSD_CASE(64);
    if (a.D <= 128) DLP_SSD_CASE(128);
    DLP_SSD_CASE(256);
#undef DLP_SSD_CASE
}

}  // namespace dlp
