// Row preparation in front of a matrix product (RowStage), as device code for the prologues of the mat-vec kernels and for stage_rows_kernel.
#pragma once
#include "layers.cuh"

namespace dlp {

// NT rows starting at t0, all threads of the block.  `put(t, k, v)` receives every value of the padded row.  `sums` holds
// stage_scratch(NT, groups) floats; ends with a barrier.
__host__ __device__ inline int stage_parts(int rows, int groups, int nwarps) {
    const int tg = rows * groups;
    return tg >= nwarps ? 1 : (nwarps + tg - 1) / tg;
}
__host__ __device__ inline int stage_scratch(int rows, int groups, int nwarps) { return rows * groups * (stage_parts(rows, groups, nwarps) + 1); }

template <typename XT>
__device__ __forceinline__ float stage_x0(const RowStage& p, int t, int k) {
    return p.x_f32 ? reinterpret_cast<const float*>(p.x)[(size_t)t * p.ldx + k] : Act<XT>::to_f(reinterpret_cast<const XT*>(p.x)[(size_t)t * p.ldx + k]);
}

// reciprocal root mean square of every (row, group) of f(t, k) -> sums[rows * groups * parts + t * groups + g]; returns that base
template <typename F>
__device__ __forceinline__ float* stage_rms(int rows, int groups, int K, float eps, float* sums, F f) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int parts = stage_parts(rows, groups, nw), gs = K / groups, per = ((gs + parts - 1) / parts + 31) / 32 * 32;
    for (int i = warp; i < rows * groups * parts; i += nw) {
        const int tg = i / parts, part = i - tg * parts, t = tg / groups, g = tg - t * groups;
        const int lo = part * per, hi = min(gs, lo + per);
        float a = 0.f;
#pragma unroll 4
        for (int k = lo + lane; k < hi; k += 32) {
            const float v = f(t, g * gs + k);
            a = fmaf(v, v, a);
        }
        a = warp_sum(a);
        if (lane == 0) sums[i] = a;
    }
    __syncthreads();
    float* rs = sums + rows * groups * parts;
    for (int i = threadIdx.x; i < rows * groups; i += blockDim.x) {
        float a = 0.f;
        for (int j = 0; j < parts; ++j) a += sums[i * parts + j];
        rs[i] = 1.f / sqrtf(a / (float)gs + eps);
    }
    __syncthreads();
    return rs;
}

// Mean and reciprocal standard deviation of every row of f(t, k) -> two floats per row behind the partial moments; returns their base.
// A warp takes a part of a row: its mean first, then the squared deviations from it; the parts are joined exactly
// (sum of squared deviations = those inside the parts + those of the parts' means).
__host__ __device__ inline int moment_scratch(int rows, int K, int nwarps) {
    const int a = 2 * rows * stage_parts(rows, 1, nwarps), b = 2 * rows * (K / 128);
    return (a > b ? a : b) + 2 * rows;
}
template <typename N>
__device__ __forceinline__ float* join_moments(int rows, int parts, int K, float eps, float* sums, N count) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    __syncthreads();
    float* ms = sums + 2 * rows * parts;
    for (int t = warp; t < rows; t += nw) {
        const float* p = sums + 2 * t * parts;
        float a = 0.f;
        for (int j = lane; j < parts; j += 32) a = fmaf(count(j), p[2 * j], a);
        const float mean = warp_sum(a) / (float)K;
        float q = 0.f;
        for (int j = lane; j < parts; j += 32) {
            const float d = p[2 * j] - mean;
            q += fmaf(count(j) * d, d, p[2 * j + 1]);
        }
        q = warp_sum(q);
        if (lane == 0) { ms[2 * t] = mean; ms[2 * t + 1] = 1.f / sqrtf(q / (float)K + eps); }
    }
    __syncthreads();
    return ms;
}
template <typename F>
__device__ __forceinline__ float* stage_moments(int rows, int K, float eps, float* sums, F f) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int parts = stage_parts(rows, 1, nw), per = ((K + parts - 1) / parts + 31) / 32 * 32;
    for (int i = warp; i < rows * parts; i += nw) {
        const int t = i / parts, lo = (i - t * parts) * per, hi = min(K, lo + per), n = max(0, hi - lo);
        float a = 0.f, q = 0.f;
#pragma unroll 4
        for (int k = lo + lane; k < hi; k += 32) a += f(t, k);
        const float mean = n > 0 ? warp_sum(a) / (float)n : 0.f;
#pragma unroll 4
        for (int k = lo + lane; k < hi; k += 32) {
            const float d = f(t, k) - mean;
            q = fmaf(d, d, q);
        }
        q = warp_sum(q);
        if (lane == 0) { sums[2 * i] = mean; sums[2 * i + 1] = q; }
    }
    return join_moments(rows, parts, K, eps, sums, [=](int j) { return (float)max(0, min(K, (j + 1) * per) - j * per); });
}

// Vector form: rows in slices of 128 values, one warp per slice and pass; groups are whole slices.
__host__ __device__ inline bool stage_vec(const RowStage& p) {
    return p.K % 128 == 0 && p.Kp == p.K && p.ldx % 8 == 0 && (!p.y || ((p.K / p.groups1) % 128 == 0 && p.ldy % 4 == 0)) && p.ldh % 4 == 0 && p.lde % 4 == 0 &&
           p.pair % 128 == 0 && (!p.g || (p.ldg % 4 == 0 && (reinterpret_cast<uintptr_t>(p.g) & 15) == 0)) &&
           (!p.w2 || ((p.K / p.groups2) % 128 == 0 && p.w2_mod % 128 == 0));
}
template <typename F>
__device__ __forceinline__ float* stage_rms_vec(int rows, int groups, int K, float eps, float* sums, F f) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5, spr = K >> 7, n = rows * spr;
#pragma unroll 4
    for (int i = warp; i < n; i += nw) {
        const int t = i / spr;
        const float4 v = f(t, (i - t * spr) * 128 + lane * 4);
        const float a = warp_sum(fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))));
        if (lane == 0) sums[i] = a;
    }
    __syncthreads();
    float* rs = sums + n;
    const int gs = K / groups, per = gs >> 7;
    for (int i = threadIdx.x; i < rows * groups; i += blockDim.x) {
        float a = 0.f;
        for (int j = 0; j < per; ++j) a += sums[i * per + j];
        rs[i] = 1.f / sqrtf(a / (float)gs + eps);
    }
    __syncthreads();
    return rs;
}
template <typename F>
__device__ __forceinline__ float* stage_moments_vec(int rows, int K, float eps, float* sums, F f) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5, spr = K >> 7, n = rows * spr;
#pragma unroll 4
    for (int i = warp; i < n; i += nw) {
        const int t = i / spr;
        float4 v = f(t, (i - t * spr) * 128 + lane * 4);
        const float mean = warp_sum((v.x + v.y) + (v.z + v.w)) * (1.f / 128.f);
        v = make_float4(v.x - mean, v.y - mean, v.z - mean, v.w - mean);
        const float q = warp_sum(fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))));
        if (lane == 0) { sums[2 * i] = mean; sums[2 * i + 1] = q; }
    }
    return join_moments(rows, spr, K, eps, sums, [](int) { return 128.f; });
}
template <typename XT>
__device__ __forceinline__ float4 stage_x4(const RowStage& p, int t, int k) {
    if (p.x_f32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p.x) + (size_t)t * p.ldx + k);
    if (sizeof(XT) == 4) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p.x) + (size_t)t * p.ldx + k);
    const uint2 u = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p.x) + (size_t)t * p.ldx + k);
    const float2 a = bf2_to_f2(u.x), b = bf2_to_f2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
// What a launch is compiled for (fewer registers in the prologue than one form for everything): norms behind the sublayers; plain sums
// and layer norms as well (y without w1, e, b2); outputs of a mixer with its gate.
enum StageForm : int { ST_NORMED = 0, ST_SUM = 1, ST_MIXER = 2 };
inline int stage_form(const RowStage& p) { return p.g || p.pair ? ST_MIXER : p.e || p.b2 || (p.y && !p.w1) ? ST_SUM : ST_NORMED; }
// gates: a row that is staged in bf16 takes the hardware exponential
template <typename XT> __device__ __forceinline__ float row_silu(float z) { return sizeof(XT) == 2 ? silu_fast(z) : silu_exact(z); }
template <typename XT> __device__ __forceinline__ float row_sigmoid(float z) { return sizeof(XT) == 2 ? __fdividef(1.f, 1.f + __expf(-z)) : sigmoid_exact(z); }
__device__ __forceinline__ bool gate_after(const RowStage& p) { return p.gate == GATE_SIGMOID_AFTER || p.gate == GATE_SILU_AFTER; }
// place in an x row of value k of the first map (the second one lies `pair` values on)
__device__ __forceinline__ int stage_pair(const RowStage& p, int k) { return k + k / p.pair * p.pair; }
template <typename XT>
__device__ __forceinline__ float4 stage_mixer4(const RowStage& p, int t, int k) {
    float4 v;
    if (p.pair) {
        const int o = stage_pair(p, k);
        const float4 b = stage_x4<XT>(p, t, o + p.pair);
        v = stage_x4<XT>(p, t, o);
        v = make_float4(fmaf(-p.lam, b.x, v.x), fmaf(-p.lam, b.y, v.y), fmaf(-p.lam, b.z, v.z), fmaf(-p.lam, b.w, v.w));
    } else {
        v = stage_x4<XT>(p, t, k);
    }
    if (p.gate == GATE_SILU_BEFORE) {
        const float4 g = *reinterpret_cast<const float4*>(p.g + (size_t)t * p.ldg + k);
        v = make_float4(v.x * row_silu<XT>(g.x), v.y * row_silu<XT>(g.y), v.z * row_silu<XT>(g.z), v.w * row_silu<XT>(g.w));
    }
    return v;
}
template <typename XT>
__device__ __forceinline__ float4 stage_gate4(const RowStage& p, int t, int k, float4 v) {
    const float4 g = *reinterpret_cast<const float4*>(p.g + (size_t)t * p.ldg + k);
    if (p.gate == GATE_SILU_AFTER) return make_float4(v.x * row_silu<XT>(g.x), v.y * row_silu<XT>(g.y), v.z * row_silu<XT>(g.z), v.w * row_silu<XT>(g.w));
    return make_float4(v.x * row_sigmoid<XT>(g.x), v.y * row_sigmoid<XT>(g.y), v.z * row_sigmoid<XT>(g.z), v.w * row_sigmoid<XT>(g.w));
}
template <typename XT>
__device__ __forceinline__ float stage_mixer(const RowStage& p, int t, int k) {
    float v;
    if (p.pair) {
        const int o = stage_pair(p, k);
        v = fmaf(-p.lam, stage_x0<XT>(p, t, o + p.pair), stage_x0<XT>(p, t, o));
    } else {
        v = stage_x0<XT>(p, t, k);
    }
    return p.gate == GATE_SILU_BEFORE ? v * row_silu<XT>(p.g[(size_t)t * p.ldg + k]) : v;
}
// Mixer outputs with every value in registers between the sums and the norm: up to HELD slices per warp.
constexpr int STAGE_HELD = 8;
template <typename XT, typename Put4>
__device__ __forceinline__ void stage_mixer_held(const RowStage& p, int t0, int rows, float* sums, Put4 put) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5, spr = p.K >> 7, n = rows * spr;
    float4 v[STAGE_HELD];
#pragma unroll
    for (int j = 0; j < STAGE_HELD; ++j) {
        const int i = warp + j * nw, t = i / spr;
        v[j] = i < n ? stage_mixer4<XT>(p, t0 + t, (i - t * spr) * 128 + lane * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float* rs = nullptr;
    const int per = p.w2 ? spr / p.groups2 : 1;
    if (p.w2) {
#pragma unroll
        for (int j = 0; j < STAGE_HELD; ++j) {
            const int i = warp + j * nw;
            if (i < n) {
                const float a = warp_sum(fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, fmaf(v[j].z, v[j].z, v[j].w * v[j].w))));
                if (lane == 0) sums[i] = a;
            }
        }
        __syncthreads();
        float* r = sums + n;
        for (int i = threadIdx.x; i < rows * p.groups2; i += blockDim.x) {
            float a = 0.f;
            for (int j = 0; j < per; ++j) a += sums[i * per + j];
            r[i] = 1.f / sqrtf(a / (float)(per << 7) + p.eps);
        }
        __syncthreads();
        rs = r;
    }
#pragma unroll
    for (int j = 0; j < STAGE_HELD; ++j) {
        const int i = warp + j * nw, t = i / spr, k = (i - t * spr) * 128 + lane * 4;
        if (i < n) {
            if (p.w2) {
                const float r = rs[i / per];
                const float4 w = *reinterpret_cast<const float4*>(p.w2 + k % p.w2_mod);
                v[j] = make_float4(v[j].x * r * w.x, v[j].y * r * w.y, v[j].z * r * w.z, v[j].w * r * w.w);
            }
            if (gate_after(p)) v[j] = stage_gate4<XT>(p, t0 + t, k, v[j]);
            put(t, k, v[j]);
        }
    }
    __syncthreads();
}
template <typename XT, int FORM, typename Put4>
__device__ __forceinline__ void stage_rows_vec(const RowStage& p, int t0, int rows, float* sums, bool store_h, Put4 put) {
    if (FORM == ST_MIXER && rows * (p.K >> 7) <= STAGE_HELD * (int)(blockDim.x >> 5)) {
        stage_mixer_held<XT>(p, t0, rows, sums, put);
        return;
    }
    constexpr bool FULL = FORM == ST_SUM;
    const float* rs1 = nullptr;
    const float* rs2 = nullptr;
    const int gs1 = p.y ? p.K / p.groups1 : 1, gs2 = p.w2 ? p.K / p.groups2 : 1;
    auto y4 = [&](int t, int k) { return *reinterpret_cast<const float4*>(p.y + (size_t)(t0 + t) * p.ldy + k); };
    if (FORM != ST_MIXER && p.y && (!FULL || p.w1)) {
        rs1 = stage_rms_vec(rows, p.groups1, p.K, p.eps, sums, y4);
        sums += rows * (p.K / 128 + p.groups1);
    }
    auto add4 = [](float4& v, float4 a) { v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w; };
    auto base = [&](int t, int k) {
        if (FORM == ST_MIXER) return stage_mixer4<XT>(p, t0 + t, k);
        float4 v = stage_x4<XT>(p, t0 + t, k);
        if (FULL && p.y && !p.w1) {
            add4(v, y4(t, k));
        } else if (p.y) {
            const float4 y = y4(t, k), w = *reinterpret_cast<const float4*>(p.w1 + k);
            const float r = rs1[t * p.groups1 + k / gs1];
            v.x = fmaf(y.x * r, w.x, v.x);
            v.y = fmaf(y.y * r, w.y, v.y);
            v.z = fmaf(y.z * r, w.z, v.z);
            v.w = fmaf(y.w * r, w.w, v.w);
        }
        if (FULL && p.e) add4(v, *reinterpret_cast<const float4*>(p.e + (size_t)(t0 + t) * p.lde + k));
        return v;
    };
    if (p.w2) rs2 = FULL && p.b2 ? stage_moments_vec(rows, p.K, p.eps, sums, base) : stage_rms_vec(rows, p.groups2, p.K, p.eps, sums, base);
    const int q = p.K >> 2;
#pragma unroll 2
    for (int i = threadIdx.x; i < rows * q; i += blockDim.x) {
        const int t = i / q, k = (i - t * q) * 4;
        float4 v = base(t, k);
        if (store_h && p.h_out) *reinterpret_cast<float4*>(p.h_out + (size_t)(t0 + t) * p.ldh + k) = v;
        if (FULL && p.w2 && p.b2) {
            const float m = rs2[2 * t], r = rs2[2 * t + 1];
            const float4 w = *reinterpret_cast<const float4*>(p.w2 + k), b = *reinterpret_cast<const float4*>(p.b2 + k);
            v = make_float4(fmaf((v.x - m) * r, w.x, b.x), fmaf((v.y - m) * r, w.y, b.y), fmaf((v.z - m) * r, w.z, b.z), fmaf((v.w - m) * r, w.w, b.w));
        } else if (p.w2) {
            const float r = rs2[t * p.groups2 + k / gs2];
            const float4 w = *reinterpret_cast<const float4*>(p.w2 + k % p.w2_mod);
            v = make_float4(v.x * r * w.x, v.y * r * w.y, v.z * r * w.z, v.w * r * w.w);
        }
        if (FORM == ST_MIXER && gate_after(p)) v = stage_gate4<XT>(p, t0 + t, k, v);
        put(t, k, v);
    }
    __syncthreads();
}
__device__ __forceinline__ void put4(__nv_bfloat16* d, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(d) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}
__device__ __forceinline__ void put4(float* d, float4 v) { *reinterpret_cast<float4*>(d) = v; }

template <typename XT, int FORM>
__device__ __forceinline__ void stage_rows_dev(const RowStage& p, int t0, int rows, float* sums, bool store_h, XT* dst, int ldd) {
    if (stage_vec(p)) {
        stage_rows_vec<XT, FORM>(p, t0, rows, sums, store_h, [&](int t, int k, float4 v) { put4(dst + (size_t)t * ldd + k, v); });
        return;
    }
    constexpr bool FULL = FORM == ST_SUM;
    const float* rs1 = nullptr;
    const float* rs2 = nullptr;
    const int gs1 = p.y ? p.K / p.groups1 : 1, gs2 = p.w2 ? p.K / p.groups2 : 1;
    if (FORM != ST_MIXER && p.y && (!FULL || p.w1)) rs1 = stage_rms(rows, p.groups1, p.K, p.eps, sums, [&](int t, int k) { return p.y[(size_t)(t0 + t) * p.ldy + k]; });
    auto base = [&](int t, int k) {
        if (FORM == ST_MIXER) return stage_mixer<XT>(p, t0 + t, k);
        float v = stage_x0<XT>(p, t0 + t, k);
        if (p.y) v += !FULL || p.w1 ? p.y[(size_t)(t0 + t) * p.ldy + k] * rs1[t * p.groups1 + k / gs1] * p.w1[k] : p.y[(size_t)(t0 + t) * p.ldy + k];
        if (FULL && p.e) v += p.e[(size_t)(t0 + t) * p.lde + k];
        return v;
    };
    if (FORM != ST_MIXER && p.y && (!FULL || p.w1)) sums += stage_scratch(rows, p.groups1, blockDim.x >> 5);
    if (p.w2) rs2 = FULL && p.b2 ? stage_moments(rows, p.K, p.eps, sums, base) : stage_rms(rows, p.groups2, p.K, p.eps, sums, base);
    for (int t = 0; t < rows; ++t) {
#pragma unroll 4
        for (int k = threadIdx.x; k < p.Kp; k += blockDim.x) {
            float v = 0.f;
            if (k < p.K) {
                v = base(t, k);
                if (store_h && p.h_out) p.h_out[(size_t)(t0 + t) * p.ldh + k] = v;
                if (p.w2) v = FULL && p.b2 ? fmaf((v - rs2[2 * t]) * rs2[2 * t + 1], p.w2[k], p.b2[k]) : v * (rs2[t * p.groups2 + k / gs2] * p.w2[k % p.w2_mod]);
                if (FORM == ST_MIXER && gate_after(p)) {
                    const float g = p.g[(size_t)(t0 + t) * p.ldg + k];
                    v *= p.gate == GATE_SILU_AFTER ? row_silu<XT>(g) : row_sigmoid<XT>(g);
                }
            }
            dst[(size_t)t * ldd + k] = Act<XT>::from_f(v);
        }
    }
    __syncthreads();
}
// the rows' tails behind their Kp values (no barrier: the rows themselves are staged next)
template <typename XT>
__device__ __forceinline__ void stage_tails(const RowStage& p, int rows, XT* dst, int ldd) {
    constexpr int VEC = Act<XT>::VEC;
    const int n = p.K_tail / VEC;
    for (int i = threadIdx.x; i < rows * n; i += blockDim.x) {
        const int t = i / n, k = (i - t * n) * VEC;
        *reinterpret_cast<uint4*>(dst + (size_t)t * ldd + p.Kp + k) = *reinterpret_cast<const uint4*>(reinterpret_cast<const XT*>(p.tail) + (size_t)t * p.ld_tail + k);
    }
}
inline size_t stage_bytes(const RowStage& p, int rows, int nwarps) {
    auto need = [&](int groups) {
        const int a = stage_scratch(rows, groups, nwarps), b = rows * (p.K / 128 + groups);
        return (size_t)(a > b ? a : b);
    };
    return ((p.y && p.w1 ? need(p.groups1) : 0) + (p.w2 ? (p.b2 ? (size_t)moment_scratch(rows, p.K, nwarps) : need(p.groups2)) : 0)) * 4 + 16;
}

inline int check_stage(const RowStage& st, const char* who) {
    DLP_REQUIRE(st.x && st.K > 0 && st.Kp >= st.K, "%s: bad input row", who);
    DLP_REQUIRE(!(st.pair || st.g) || (!st.y && !st.e && !st.b2 && !st.h_out && st.pair >= 0 && (!st.pair || st.K % st.pair == 0) && (st.gate == GATE_NONE || st.g)), "%s: pairs of %d, gate %d",
                who, st.pair, st.gate);
    DLP_REQUIRE(st.K_tail == 0 || (st.K_tail > 0 && st.K_tail % 8 == 0 && st.Kp % 8 == 0 && st.tail && st.ld_tail % 8 == 0 && (reinterpret_cast<uintptr_t>(st.tail) & 15) == 0),
                "%s: tail of %d values", who, st.K_tail);
    DLP_REQUIRE(!st.y || (st.groups1 > 0 && st.K % st.groups1 == 0), "%s: %d norm groups do not divide the width %d", who, st.groups1, st.K);
    DLP_REQUIRE(!st.b2 || (st.w2 && st.groups2 == 1 && st.w2_mod == st.K), "%s: a layer norm spans the whole row", who);
    DLP_REQUIRE(!st.w2 || (st.w2_mod > 0 && st.groups2 > 0 && st.K % st.groups2 == 0), "%s: %d norm groups do not divide the width %d", who, st.groups2, st.K);
    return 0;
}

}  // namespace dlp
