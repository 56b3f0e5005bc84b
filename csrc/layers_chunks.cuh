// Loading of token rows and operand helpers shared by the recurrences that run in chunks on the tensor cores (layers_ssd.cu, layers_delta.cu).
#pragma once
#include "layers.cuh"
#include "mma.cuh"

namespace dlp {

__device__ __forceinline__ float softplus_exact(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// one value of a row, behind silu when `act`
__device__ __forceinline__ float mix_row(const void* rows, int f32, int act, size_t i) {
    const float x = f32 ? reinterpret_cast<const float*>(rows)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(rows)[i]);
    return act ? silu_exact(x) : x;
}
// NTH threads: R rows of W columns (columns past ncols and rows past n are zero), four values a time: put(row, column, values)
template <typename RT, int R, int W, int NTH, typename Put>
__device__ __forceinline__ void chunk_rows(const RT* base, int ld, int n, int ncols, int act, Put put) {
    constexpr int QN = R * W / 4 / NTH, QB = QN < 8 ? QN : 8;
    const bool vec = ld % 4 == 0 && ncols % 4 == 0 && (reinterpret_cast<uintptr_t>(base) & (4 * sizeof(RT) - 1)) == 0;
#pragma unroll 1
    for (int b = 0; b < QN; b += QB) {
        float4 x[QB];
#pragma unroll
        for (int j = 0; j < QB; ++j) {
            const int i = threadIdx.x + (b + j) * NTH, s = i / (W / 4), c = i % (W / 4) * 4;
            const RT* p = base + (size_t)s * ld + c;
            x[j] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (s < n && c < ncols) {
                if (vec) {
                    if (sizeof(RT) == 4) {
                        x[j] = *reinterpret_cast<const float4*>(p);
                    } else {
                        const uint2 u = *reinterpret_cast<const uint2*>(p);
                        const float2 lo = bf2_to_f2(u.x), hi = bf2_to_f2(u.y);
                        x[j] = make_float4(lo.x, lo.y, hi.x, hi.y);
                    }
                } else {
                    x[j].x = Act<RT>::to_f(p[0]);
                    if (c + 1 < ncols) x[j].y = Act<RT>::to_f(p[1]);
                    if (c + 2 < ncols) x[j].z = Act<RT>::to_f(p[2]);
                    if (c + 3 < ncols) x[j].w = Act<RT>::to_f(p[3]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < QB; ++j) {
            const int i = threadIdx.x + (b + j) * NTH;
            if (act) x[j] = make_float4(silu_fast(x[j].x), silu_fast(x[j].y), silu_fast(x[j].z), silu_fast(x[j].w));
            put(i / (W / 4), i % (W / 4) * 4, x[j]);
        }
    }
}
__device__ __forceinline__ void put_bf16(__nv_bfloat16* d, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(d) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ void put_split(__nv_bfloat16* hi, __nv_bfloat16* lo, float4 v) {
    uint2 h, l;
    split_bf16(v.x, v.y, h.x, l.x);
    split_bf16(v.z, v.w, h.y, l.y);
    *reinterpret_cast<uint2*>(hi) = h;
    *reinterpret_cast<uint2*>(lo) = l;
}
// the chunk's rows as bf16 in shared memory [R][W + 8]; bf16 rows arrive with cp.async (the caller waits)
template <typename RT, int R, int W, int NTH>
__device__ __forceinline__ void chunk_tile(const void* rows, int ld, size_t col0, int t0, int n, int ncols, int act, __nv_bfloat16* dst) {
    const RT* base = reinterpret_cast<const RT*>(rows) + (size_t)t0 * ld + col0;
    if (sizeof(RT) == 2 && !act && ld % 8 == 0 && ncols % 8 == 0 && (reinterpret_cast<uintptr_t>(base) & 15) == 0) {
#pragma unroll 4
        for (int i = threadIdx.x; i < R * W / 8; i += NTH) {
            const int s = i / (W / 8), c = i % (W / 8) * 8;
            const bool ok = s < n && c < ncols;
            cp_async16(dst + s * (W + 8) + c, ok ? base + (size_t)s * ld + c : base, ok);
        }
        return;
    }
    chunk_rows<RT, R, W, NTH>(base, ld, n, ncols, act, [&](int s, int c, float4 x) { put_bf16(dst + s * (W + 8) + c, x); });
}

}  // namespace dlp
