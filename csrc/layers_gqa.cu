// Grouped-query softmax attention of layer-list models over paged keys and values: sliding window, kept first tokens, chunks, one or two
// maps per head over the same values.
//
//   gqa_prepare_kernel    projection rows -> normalised, rotated queries, and keys / values into their pages (prompts, mixed batches)
//   gqa_attn_mma_kernel   bf16, heads up to 256 wide: a tile is the query heads of one key / value head for one or more tokens of a
//                         request, mma.sync m16n8k16 over key tiles that arrive with cp.async; the key range is split over a thread-block
//                         cluster and joined through distributed shared memory.  The fused form takes single tokens straight from the
//                         projection (norm, rotation, cache write and attention in one launch)
//   gqa_attn_kernel       any width, bf16 or fp32 storage
//
// Keys are counted through the window: index v < nk is the kept key v, the others are the keys from the first one the window still
// shows (to the first token of the tile).  Scores and softmax weights stay in fp32: for the tensor cores a weight is split into two
// bf16 parts (the rounded value and the rest), whose products with the values are summed.
//
// Two maps: a key tile holds both keys of a token side by side, and a query row is zero under the other map's key, so that both maps'
// rows share one tile of keys and values.
#include <cooperative_groups.h>
#include <type_traits>

#include "layers.cuh"
#include "mma.cuh"

namespace dlp {

// dimension d of a head after norm and rotation: x, w point at the head's first value, cs holds (cos, sin) of every pair
__device__ __forceinline__ float gqa_value(const float* x, const float* w, float r, const float2* cs, int rot, int adjacent, int d) {
    const float a = x[d] * (w ? r * w[d] : 1.f);
    if (d >= rot) return a;
    if (adjacent) {
        const float b = x[d ^ 1] * (w ? r * w[d ^ 1] : 1.f);
        const float2 c = cs[d >> 1];
        return d & 1 ? a * c.x + b * c.y : a * c.x - b * c.y;
    }
    const int half = rot >> 1, o = d < half ? d + half : d - half;
    const float b = x[o] * (w ? r * w[o] : 1.f);
    const float2 c = cs[d < half ? d : o];
    return d < half ? a * c.x - b * c.y : a * c.x + b * c.y;
}
__device__ __forceinline__ void gqa_angles(const GqaArgs& a, int pos, float2* cs) {
    for (int i = threadIdx.x; i < a.rot / 2; i += blockDim.x) {
        float s, c;
        sincosf((float)pos * a.inv_freq[i], &s, &c);
        cs[i] = make_float2(c * a.rot_scale, s * a.rot_scale);
    }
}
// value i of the projection, mixed with the first mixing layer's; `keep`: this is that layer, and the caller stores its values
__device__ __forceinline__ float gqa_mixed(const GqaArgs& a, int t, const float* v, int i, bool keep) {
    if (a.v_mix == 0) return v[i];
    float* first = a.v_first + (size_t)t * a.G * a.V + i;
    if (a.v_mix == 2) return fmaf(a.v_lam, *first, (1.f - a.v_lam) * v[i]);
    if (keep) *first = v[i];
    return v[i];
}
__device__ __forceinline__ float gqa_sumsq(const float* x, int n) {      // this thread's share
    float s = 0.f;
    if (((reinterpret_cast<uintptr_t>(x) | (uintptr_t)(4 * n)) & 15) == 0) {
#pragma unroll 4
        for (int i = threadIdx.x; i < n / 4; i += blockDim.x) {
            const float4 v = reinterpret_cast<const float4*>(x)[i];
            s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
        }
    } else {
#pragma unroll 4
        for (int i = threadIdx.x; i < n; i += blockDim.x) s = fmaf(x[i], x[i], s);
    }
    return s;
}

__device__ __forceinline__ void put2(__nv_bfloat16* d, float x, float y) { *reinterpret_cast<__nv_bfloat162*>(d) = __floats2bfloat162_rn(x, y); }
__device__ __forceinline__ void put2(float* d, float x, float y) { *reinterpret_cast<float2*>(d) = make_float2(x, y); }

template <typename WT>
__global__ void __launch_bounds__(256) gqa_prepare_kernel(const GqaArgs a) {
    extern __shared__ __align__(16) uint8_t gq_smem[];
    float2* cs = reinterpret_cast<float2*>(gq_smem);
    __shared__ float red[32];
    pdl_wait();
    const int t = blockIdx.x, slot = a.slot[t];
    const float* q = a.proj + (size_t)t * a.ldp;
    const float* k = q + a.H * a.D;
    const float* v = k + a.G * a.maps * a.D;
    gqa_angles(a, a.pos[t], cs);
    const float rq = a.q_norm ? 1.f / sqrtf(block_sum(gqa_sumsq(q, a.H * a.D), red) / (float)(a.H * a.D) + a.eps) : 1.f;
    const float rk = a.k_norm ? 1.f / sqrtf(block_sum(gqa_sumsq(k, a.G * a.maps * a.D), red) / (float)(a.G * a.maps * a.D) + a.eps) : 1.f;
    __syncthreads();
    // a warp per head: query heads, then key heads, then value heads
    const int lane = threadIdx.x & 31;
    const size_t page = max(slot, 0) / a.page_size, off = max(slot, 0) % a.page_size;
    const int kh = a.G * a.maps;
    for (int i = threadIdx.x >> 5; i < a.H + (slot >= 0 ? kh + a.G : 0); i += 8) {
        if (i < a.H + kh) {
            const bool is_q = i < a.H;
            const int h = is_q ? i : i - a.H;
            const float* x = (is_q ? q : k) + h * a.D;
            const float* w = is_q ? a.q_norm : a.k_norm;
            if (w) w += h * a.D;
            WT* o = is_q ? reinterpret_cast<WT*>(a.q) + ((size_t)t * a.H + h) * a.Dc : reinterpret_cast<WT*>(a.kc) + ((page * kh + h) * a.page_size + off) * a.Dc;
            const float r = is_q ? rq : rk;
            for (int d = lane * 2; d < a.Dc; d += 64) put2(o + d, d < a.D ? gqa_value(x, w, r, cs, a.rot, a.adjacent, d) : 0.f, d + 1 < a.D ? gqa_value(x, w, r, cs, a.rot, a.adjacent, d + 1) : 0.f);
        } else {
            const int g = i - a.H - kh;
            WT* o = reinterpret_cast<WT*>(a.vc) + ((page * a.G + g) * a.page_size + off) * a.Vc;
            for (int d = lane * 2; d < a.Vc; d += 64) put2(o + d, d < a.V ? gqa_mixed(a, t, v, g * a.V + d, true) : 0.f, d + 1 < a.V ? gqa_mixed(a, t, v, g * a.V + d + 1, true) : 0.f);
        }
    }
    pdl_launch_dependents();
}

// first key that the window and the chunk of a position show
__device__ __forceinline__ int first_key(const GqaArgs& a, int pos) { return max(max(0, pos - a.window + 1), a.chunk > 0 ? pos / a.chunk * a.chunk : 0); }
// keys that some row of a tile sees (positions q_lo .. q_hi), and the part of them this split reads
struct WindowKeys {
    int win_lo, nk, n, lo, hi;
    __device__ __forceinline__ int key(int v) const { return v < nk ? v : win_lo + v - nk; }
};
__device__ __forceinline__ WindowKeys window_keys(const GqaArgs& a, int q_lo, int q_hi, int split, int step) {
    WindowKeys w;
    const int len = min(q_hi + 1, a.max_pages * a.page_size);
    w.win_lo = first_key(a, q_lo);
    w.nk = min(a.keep, w.win_lo);
    w.n = w.nk + max(0, len - w.win_lo);
    const int per = ((w.n + a.n_splits - 1) / a.n_splits + step - 1) / step * step;
    w.lo = min(w.n, split * per);
    w.hi = min(w.n, w.lo + per);
    return w;
}

constexpr int GQA_BN = 64;
__host__ __device__ inline int gqa_heads(int R, int bm) { return R < bm ? R : bm; }       // query heads of a tile
static size_t gqa_smem(const GqaArgs& a, int bm, int fused) {
    const int LDK = a.maps * a.Dc + 8, LDV = a.Vc + 8;
    size_t n = (size_t)bm * LDK * 2 + (size_t)2 * GQA_BN * (LDK + LDV) * 2 + (size_t)bm * (GQA_BN + 4) * 4 + bm * 3 * 4 + (size_t)bm * 16 * 4 + a.maps * 2 * GQA_BN * 4;
    if (fused) n += (size_t)(a.maps * a.Dc + a.Vc) * 2 + (a.rot / 2) * 8 + 16;
    return n;
}

// MW: 16-row blocks of a tile; NWARP warps share a tile as MW x (NWARP / MW).
template <int MW, int NWARP, int VMAX, bool FUSED, int MAPS>
__global__ void __launch_bounds__(32 * NWARP) gqa_attn_mma_kernel(const GqaArgs a) {
    namespace cg = cooperative_groups;
    constexpr int BN = GQA_BN, NTH = 32 * NWARP, BM = 16 * MW, NW = NWARP / MW, KPW = BN / NW, LS = BN + 4, TPR = NTH / BM;
    constexpr int NPAIR = (VMAX / 16 + NW - 1) / NW;      // 16-column output blocks of a warp
    extern __shared__ __align__(16) uint8_t gq_smem[];
    __shared__ float red[32];
    const int KD = MAPS * a.Dc, LDK = KD + 8, LDV = a.Vc + 8;
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(gq_smem);
    __nv_bfloat16* ks = qs + BM * LDK;                    // [2][BN][LDK]
    __nv_bfloat16* vs = ks + 2 * BN * LDK;                // [2][BN][LDV]
    float* S = reinterpret_cast<float*>(vs + 2 * BN * LDV);
    float* s_alpha = S + BM * LS;
    float* s_m = s_alpha + BM;
    float* s_l = s_m + BM;
    float* s_w = s_l + BM;                                // [BM][16] weight of every split
    int* offs = reinterpret_cast<int*>(s_w + BM * 16);    // [2][BN] value row of every key of a tile (-1: none, -2: the new key)
    int* koffs = offs + (MAPS > 1 ? 2 * BN : 0);          // [2][BN] key row of the first map
    float2* cs = reinterpret_cast<float2*>(offs + MAPS * 2 * BN);
    __nv_bfloat16* k_new = reinterpret_cast<__nv_bfloat16*>(cs + (FUSED ? a.rot / 2 : 0));
    __nv_bfloat16* v_new = k_new + KD;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, mw = warp / NW, nw = warp % NW, gr = lane >> 2, c = lane & 3;
    const int split = blockIdx.x, tile = blockIdx.z, R = a.H / a.G, hb = gqa_heads(R, BM), hgroups = (R + hb - 1) / hb;
    const int g = blockIdx.y / hgroups, hg = blockIdx.y - g * hgroups, h0 = g * R + hg * hb, hn = min(hb, R - hg * hb);
    if (!FUSED) pdl_wait();
    // (fused: tile table, positions and pages were written at least two launches back, cached rows in earlier steps)
    const int t0 = a.tile_row0[tile], nt = FUSED ? 1 : a.tile_rows[tile], rows = nt * hn;
    if (nt <= 0) return;
    const int q_lo = a.pos[t0], q_hi = q_lo + nt - 1;
    const WindowKeys wk = window_keys(a, q_lo, q_hi, split, 16);
    const int* bt = a.block_table + (size_t)a.tok_slot[t0] * a.max_pages;
    const __nv_bfloat16* kc = reinterpret_cast<const __nv_bfloat16*>(a.kc);
    const __nv_bfloat16* vc = reinterpret_cast<const __nv_bfloat16*>(a.vc);
    auto cache_row = [&](int key) { return (bt[key / a.page_size] * a.G + g) * a.page_size + key % a.page_size; };
    auto find_rows = [&](int v0, int b) {
        if (tid < BN) {
            const int v = v0 + tid;
            int row = -1;
            if (v < wk.hi) {
                const int key = wk.key(v);
                row = FUSED && key == q_hi ? -2 : cache_row(key);
            }
            offs[b * BN + tid] = row;
            if (MAPS > 1) koffs[b * BN + tid] = MAPS * row - (MAPS - 1) * (max(row, 0) % a.page_size);
        }
    };
    const int kch = KD / 8, vch = a.Vc / 8, mch = a.Dc / 8;
    auto load_tile = [&](int b) {           // eight threads per key
#pragma unroll
        for (int part = 0; part < BN / (NTH / 8); ++part) {
            const int kk = part * (NTH / 8) + (tid >> 3), row = offs[b * BN + kk];
            if (!FUSED || row != -2) {
                const __nv_bfloat16* sk = kc + (size_t)max(koffs[b * BN + kk], 0) * a.Dc;
                const __nv_bfloat16* sv = vc + (size_t)max(row, 0) * a.Vc;
                __nv_bfloat16* dk = ks + ((size_t)b * BN + kk) * LDK;
                __nv_bfloat16* dv = vs + ((size_t)b * BN + kk) * LDV;
                for (int ch = tid & 7; ch < kch; ch += 8) cp_async16(dk + ch * 8, MAPS > 1 && ch >= mch ? sk + (size_t)a.page_size * a.Dc + (ch - mch) * 8 : sk + ch * 8, row >= 0);
                for (int ch = tid & 7; ch < vch; ch += 8) cp_async16(dv + ch * 8, sv + ch * 8, row >= 0);
            }
        }
        cp_commit();
    };
    const int n_tiles = (wk.hi - wk.lo + BN - 1) / BN;
    find_rows(wk.lo, 0);
    find_rows(wk.lo + BN, 1);
    __syncthreads();
    if (n_tiles > 0) load_tile(0);
    const bool owns_new = FUSED && wk.hi == wk.n && wk.hi > wk.lo;
    if (FUSED) {
        gqa_angles(a, q_hi, cs);
        pdl_wait();
        const float* qp = a.proj + (size_t)t0 * a.ldp;
        const float* kp = qp + a.H * a.D;
        const float rq = a.q_norm ? 1.f / sqrtf(block_sum(gqa_sumsq(qp, a.H * a.D), red) / (float)(a.H * a.D) + a.eps) : 1.f;
        __syncthreads();
        for (int i = tid; i < BM * KD; i += NTH) {
            const int r = i / KD, c = i - r * KD, m = MAPS > 1 ? c / a.Dc : 0, d = c - m * a.Dc, o = (h0 + r) * a.D;
            const bool mine = r < hn && d < a.D && (MAPS == 1 || (h0 + r) % MAPS == m);
            qs[r * LDK + c] = __float2bfloat16_rn(mine ? gqa_value(qp + o, a.q_norm ? a.q_norm + o : nullptr, rq, cs, a.rot, a.adjacent, d) : 0.f);
        }
        if (owns_new) {                     // the new token's key and value: into the pages and, below, into this block's last tile
            const int kd = a.G * MAPS * a.D;
            const float* vp = kp + kd;
            const float rk = a.k_norm ? 1.f / sqrtf(block_sum(gqa_sumsq(kp, kd), red) / (float)kd + a.eps) : 1.f;
            const size_t row = cache_row(q_hi);
            const size_t krow = MAPS * row - (MAPS - 1) * (row % a.page_size);
            for (int c = tid; c < KD; c += NTH) {
                const int m = MAPS > 1 ? c / a.Dc : 0, d = c - m * a.Dc, o = (g * MAPS + m) * a.D;
                const __nv_bfloat16 x = __float2bfloat16_rn(d < a.D ? gqa_value(kp + o, a.k_norm ? a.k_norm + o : nullptr, rk, cs, a.rot, a.adjacent, d) : 0.f);
                k_new[c] = x;
                if (hg == 0) reinterpret_cast<__nv_bfloat16*>(a.kc)[(krow + (size_t)m * a.page_size) * a.Dc + d] = x;
            }
            for (int d = tid; d < a.Vc; d += NTH) {
                const __nv_bfloat16 x = __float2bfloat16_rn(d < a.V ? gqa_mixed(a, t0, vp, g * a.V + d, hg == 0) : 0.f);
                v_new[d] = x;
                if (hg == 0) reinterpret_cast<__nv_bfloat16*>(a.vc)[row * a.Vc + d] = x;
            }
            __syncthreads();
        }
    } else {
        const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(a.q);
        for (int i = tid; i < BM * kch; i += NTH) {
            const int r = i / kch, ch = i - r * kch, t = t0 + r / hn, h = h0 + r % hn, m = MAPS > 1 ? ch / mch : 0;
            *reinterpret_cast<uint4*>(qs + r * LDK + ch * 8) =
                r < rows && (MAPS == 1 || h % MAPS == m) ? *reinterpret_cast<const uint4*>(q + ((size_t)t * a.H + h) * a.Dc + (ch - m * mch) * 8) : make_uint4(0, 0, 0, 0);
        }
    }
    const int sr = tid / TPR, sub = tid % TPR;             // softmax: TPR threads per row
    const int my_pos = sr < rows ? q_lo + sr / hn : -1, my_first = first_key(a, max(my_pos, 0));
    float m_run = -INFINITY, l_run = 0.f;
    float acc[NPAIR][2][4] = {};
    for (int it = 0; it < n_tiles; ++it) {
        const int v0 = wk.lo + it * BN, b = it & 1;
        if (it + 1 < n_tiles) { load_tile(b ^ 1); cp_wait<1>(); } else { cp_wait<0>(); }
        if (owns_new && it == n_tiles - 1) {
            const int kk = wk.hi - 1 - v0;
            for (int d = tid; d < KD; d += NTH) ks[((size_t)b * BN + kk) * LDK + d] = k_new[d];
            for (int d = tid; d < a.Vc; d += NTH) vs[((size_t)b * BN + kk) * LDV + d] = v_new[d];
        }
        __syncthreads();
        if (it + 2 < n_tiles) find_rows(v0 + 2 * BN, b);      // read behind the barriers of this iteration
        const __nv_bfloat16* kt = ks + (size_t)b * BN * LDK;
        const __nv_bfloat16* vt = vs + (size_t)b * BN * LDV;
        {   // scores: 16 rows x KPW keys per warp
            constexpr int NJ = KPW / 8;
            float sacc[NJ][4] = {};
#pragma unroll 4
            for (int k = 0; k < KD; k += 16) {
                uint32_t af[4];
                ldsm_x4(af, qs + (mw * 16 + (lane & 15)) * LDK + k + (lane >> 4) * 8);
#pragma unroll
                for (int j = 0; j < NJ; j += 2) {
                    uint32_t bf[4];
                    ldsm_x4(bf, kt + (nw * KPW + j * 8 + (lane & 7) + (lane >> 4) * 8) * LDK + k + ((lane >> 3) & 1) * 8);
                    mma16816(sacc[j], af, bf[0], bf[1]);
                    mma16816(sacc[j + 1], af, bf[2], bf[3]);
                }
            }
#pragma unroll
            for (int j = 0; j < NJ; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[(mw * 16 + gr + (e >> 1) * 8) * LS + nw * KPW + j * 8 + c * 2 + (e & 1)] = sacc[j][e] * a.scale;
        }
        __syncthreads();
        {   // running softmax
            float* row = S + sr * LS;
            float v[BN / TPR], mx = m_run;
#pragma unroll
            for (int i = 0; i < BN / TPR; ++i) {
                const int kk = i * TPR + sub;
                const int key = wk.key(v0 + kk);
                v[i] = (v0 + kk < wk.hi && key <= my_pos && (key >= my_first || key < a.keep)) ? row[kk] : -INFINITY;
                mx = fmaxf(mx, v[i]);
            }
#pragma unroll
            for (int x = 1; x < TPR; x <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
            const float ms = mx == -INFINITY ? 0.f : mx;
            const float alpha = m_run == -INFINITY ? 0.f : expf(m_run - ms);
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < BN / TPR; ++i) {
                const float p = expf(v[i] - ms);
                sum += p;
                row[i * TPR + sub] = p;
            }
#pragma unroll
            for (int x = 1; x < TPR; x <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, x);
            l_run = l_run * alpha + sum;
            m_run = mx;
            if (sub == 0) s_alpha[sr] = alpha;
        }
        __syncthreads();
        {   // values: 16 rows x this warp's 16-column blocks
            const float a0 = s_alpha[mw * 16 + gr], a1 = s_alpha[mw * 16 + gr + 8];
#pragma unroll
            for (int j = 0; j < NPAIR; ++j)
#pragma unroll
                for (int n = 0; n < 2; ++n) { acc[j][n][0] *= a0; acc[j][n][1] *= a0; acc[j][n][2] *= a1; acc[j][n][3] *= a1; }
#pragma unroll
            for (int kk = 0; kk < BN / 16; ++kk) {
                uint32_t hi[4], lo[4];
                const float* r0 = S + (mw * 16 + gr) * LS + kk * 16 + c * 2;
                const float* r1 = r0 + 8 * LS;
                split_bf16(r0[0], r0[1], hi[0], lo[0]);
                split_bf16(r1[0], r1[1], hi[1], lo[1]);
                split_bf16(r0[8], r0[9], hi[2], lo[2]);
                split_bf16(r1[8], r1[9], hi[3], lo[3]);
#pragma unroll
                for (int j = 0; j < NPAIR; ++j) {
                    const int col = (j * NW + nw) * 16;
                    if (col < a.Vc) {
                        uint32_t bf[4];
                        ldsm_x4_t(bf, vt + (kk * 16 + (lane & 15)) * LDV + col + (lane >> 4) * 8);
                        mma16816(acc[j][0], hi, bf[0], bf[1]);
                        mma16816(acc[j][1], hi, bf[2], bf[3]);
                        mma16816(acc[j][0], lo, bf[0], bf[1]);
                        mma16816(acc[j][1], lo, bf[2], bf[3]);
                    }
                }
            }
        }
        __syncthreads();      // the next load overwrites this tile's buffer two iterations on, S in the next one
    }
    pdl_launch_dependents();
    if (sub == 0) { s_m[sr] = m_run; s_l[sr] = l_run; }
    __syncthreads();
    using OT = std::conditional_t<MAPS == 1, __nv_bfloat16, float>;
    OT* out = reinterpret_cast<OT*>(a.out);
    float* po = reinterpret_cast<float*>(vs);              // [rows][Vc]: the tiles have been read
    const bool one = a.n_splits == 1;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = mw * 16 + gr + half * 8;
        if (r >= rows) continue;
        const float inv = s_l[r] > 0.f ? 1.f / s_l[r] : 0.f;
        OT* o = out + (size_t)(t0 + r / hn) * a.ldo + (size_t)(h0 + r % hn) * a.V;
#pragma unroll
        for (int j = 0; j < NPAIR; ++j)
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int col = (j * NW + nw) * 16 + n * 8 + c * 2 + e;
                    if (one) {
                        if (col < a.V) o[col] = Act<OT>::from_f(acc[j][n][half * 2 + e] * inv);
                    } else if (col < a.Vc) {
                        po[r * a.Vc + col] = acc[j][n][half * 2 + e];
                    }
                }
    }
    if (one) return;
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    for (int i = tid; i < rows; i += NTH) {
        float ms[16], m = -INFINITY, l = 0.f;
#pragma unroll
        for (int s = 0; s < 16; ++s) {
            ms[s] = s < a.n_splits ? cluster.map_shared_rank(s_m, s)[i] : -INFINITY;
            m = fmaxf(m, ms[s]);
        }
#pragma unroll
        for (int s = 0; s < 16; ++s) {
            ms[s] = ms[s] == -INFINITY ? 0.f : expf(ms[s] - m);
            if (ms[s] > 0.f) l = fmaf(ms[s], cluster.map_shared_rank(s_l, s)[i], l);
        }
#pragma unroll
        for (int s = 0; s < 16; ++s) s_w[i * 16 + s] = l > 0.f ? ms[s] / l : 0.f;
    }
    __syncthreads();
    for (int i = split * NTH + tid; i < rows * a.V; i += a.n_splits * NTH) {       // every block of the cluster writes its share
        const int r = i / a.V, col = i - r * a.V;
        float x[16], v = 0.f;
#pragma unroll
        for (int s = 0; s < 16; ++s) x[s] = s < a.n_splits ? cluster.map_shared_rank(po, s)[r * a.Vc + col] : 0.f;
#pragma unroll
        for (int s = 0; s < 16; ++s) v = fmaf(x[s], s_w[r * 16 + s], v);
        out[(size_t)(t0 + r / hn) * a.ldo + (size_t)(h0 + r % hn) * a.V + col] = Act<OT>::from_f(v);
    }
    cluster.sync();           // nobody leaves while its shared memory is read
}

// ---- any width, any storage: one CTA per tile and head ----------------------------------------------------------
template <typename WT>
__global__ void __launch_bounds__(128) gqa_attn_kernel(const GqaArgs a) {
    extern __shared__ __align__(16) uint8_t gq_smem[];
    float* q = reinterpret_cast<float*>(gq_smem);         // [D]
    float* acc = q + a.D;                                 // [V]
    float* s = acc + a.V;                                 // [64]
    int* row = reinterpret_cast<int*>(s + 64);            // [64] value rows
    int* krow = row + 64;                                 // [64] key rows
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, tile = blockIdx.x, h = blockIdx.y, g = h / (a.H / a.G);
    pdl_wait();
    const int t0 = a.tile_row0[tile], nt = a.tile_rows[tile];
    const int* bt = a.block_table + (size_t)a.tok_slot[t0] * a.max_pages;
    for (int t = t0; t < t0 + nt; ++t) {
        const int pos = a.pos[t];
        const WindowKeys wk = window_keys(a, pos, pos, 0, 1);          // n_splits is 1 here
        for (int d = tid; d < a.D; d += 128) q[d] = (float)reinterpret_cast<const WT*>(a.q)[((size_t)t * a.H + h) * a.Dc + d];
        for (int d = tid; d < a.V; d += 128) acc[d] = 0.f;
        float m = -INFINITY, l = 0.f;
        for (int v0 = 0; v0 < wk.n; v0 += 64) {
            const int n = min(64, wk.n - v0);
            if (tid < n) {
                const int key = wk.key(v0 + tid);
                row[tid] = (bt[key / a.page_size] * a.G + g) * a.page_size + key % a.page_size;
                krow[tid] = ((bt[key / a.page_size] * a.G + g) * a.maps + h % a.maps) * a.page_size + key % a.page_size;
            }
            __syncthreads();
            for (int kk = warp; kk < 64; kk += 4) {
                float d = 0.f;
                if (kk < n) {
                    const WT* kr = reinterpret_cast<const WT*>(a.kc) + (size_t)krow[kk] * a.Dc;
                    for (int r = lane; r < a.D; r += 32) d = fmaf(q[r], (float)kr[r], d);
                }
                d = warp_sum(d);
                if (lane == 0) s[kk] = kk < n ? d * a.scale : -INFINITY;
            }
            __syncthreads();
            const float s0 = s[lane], s1 = s[lane + 32];
            const float mn = fmaxf(m, warp_max(fmaxf(s0, s1)));
            const float p0 = expf(s0 - mn), p1 = expf(s1 - mn), alpha = m == -INFINITY ? 0.f : expf(m - mn);
            l = l * alpha + warp_sum(p0 + p1);
            m = mn;
            __syncthreads();
            if (warp == 0) { s[lane] = p0; s[lane + 32] = p1; }
            __syncthreads();
            for (int r = tid; r < a.V; r += 128) {
                float v = acc[r] * alpha;
#pragma unroll 4
                for (int kk = 0; kk < n; ++kk) v = fmaf(s[kk], (float)reinterpret_cast<const WT*>(a.vc)[(size_t)row[kk] * a.Vc + r], v);
                acc[r] = v;
            }
            __syncthreads();
        }
        const float inv = l > 0.f ? 1.f / l : 0.f;
        for (int r = tid; r < a.V; r += 128) {
            const size_t o = (size_t)t * a.ldo + (size_t)h * a.V + r;
            if (a.maps > 1) reinterpret_cast<float*>(a.out)[o] = acc[r] * inv;
            else reinterpret_cast<WT*>(a.out)[o] = Act<WT>::from_f(acc[r] * inv);
        }
    }
    pdl_launch_dependents();
}

static int check_gqa(const GqaArgs& a, const char* who) {
    DLP_REQUIRE(a.kc && a.vc && a.block_table && a.tok_slot && a.pos, "%s: null argument", who);
    DLP_REQUIRE(a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.D > 0 && a.V > 0 && a.Dc >= a.D && a.Vc >= a.V && a.Dc % 16 == 0 && a.Vc % 16 == 0, "%s: heads %d / %d of %d and %d", who,
                a.H, a.G, a.D, a.V);
    DLP_REQUIRE(a.rot >= 0 && a.rot % 2 == 0 && a.rot <= a.D && (a.rot == 0 || a.inv_freq), "%s: rotation of %d dimensions", who, a.rot);
    DLP_REQUIRE(a.T > 0 && a.page_size > 0 && a.max_pages > 0 && a.window >= 1 && a.keep >= 0 && a.chunk >= 0, "%s: bad shape", who);
    DLP_REQUIRE(a.v_mix >= 0 && a.v_mix <= 2 && (a.v_mix == 0 || a.v_first), "%s: value mixing %d", who, a.v_mix);
    DLP_REQUIRE((a.maps == 1 || a.maps == 2) && (a.H / a.G) % a.maps == 0, "%s: %d maps", who, a.maps);
    return 0;
}

int gqa_prepare(const GqaArgs& a, int f32, cudaStream_t s) {
    int rc = check_gqa(a, "gqa_prepare");
    if (rc) return rc;
    DLP_REQUIRE(a.proj && a.q && a.slot && a.rot <= 8192, "gqa_prepare: bad argument");
    const size_t smem = (size_t)(a.rot / 2) * 8;
    DLP_CHECK_CUDA(f32 ? launch_pdl(gqa_prepare_kernel<float>, dim3(a.T), dim3(256), smem, s, a) : launch_pdl(gqa_prepare_kernel<__nv_bfloat16>, dim3(a.T), dim3(256), smem, s, a));
    return 0;
}

template <int MW, int NWARP, int VMAX, bool FUSED, int MAPS>
static int launch_gqa_maps(const GqaArgs& a, cudaStream_t s) {
    constexpr int BM = 16 * MW;
    const size_t smem = gqa_smem(a, BM, FUSED);
    DLP_REQUIRE(smem <= 226 * 1024, "gqa_attention: %zu bytes of shared memory", smem);
    auto kern = gqa_attn_mma_kernel<MW, NWARP, VMAX, FUSED, MAPS>;
    if (first_use_on_device((const void*)kern)) {
        DLP_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024));
        DLP_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
    }
    const int R = a.H / a.G, hb = gqa_heads(R, BM);
    DLP_CHECK_CUDA(launch_pdl_cluster(kern, dim3(a.n_splits, a.G * ((R + hb - 1) / hb), a.n_tiles), dim3(32 * NWARP), smem, s, a.n_splits, a));
    return 0;
}

template <int MW, int NWARP, int VMAX, bool FUSED>
static int launch_gqa(const GqaArgs& a, cudaStream_t s) {
    return a.maps == 1 ? launch_gqa_maps<MW, NWARP, VMAX, FUSED, 1>(a, s) : launch_gqa_maps<MW, NWARP, VMAX, FUSED, 2>(a, s);
}

// tiles: bm / min(H / G, bm) tokens at most
int gqa_attention(const GqaArgs& a, int fused, int f32, cudaStream_t s) {
    int rc = check_gqa(a, "gqa_attention");
    if (rc) return rc;
    DLP_REQUIRE(a.out && a.tile_row0 && a.tile_rows && a.n_tiles > 0 && a.n_tiles <= 65535 && (fused ? a.proj != nullptr : a.q != nullptr), "gqa_attention: bad argument");
    if (!f32 && a.maps * a.Dc <= 256 && a.Vc <= 256) {
        DLP_REQUIRE(a.n_splits >= 1 && a.n_splits <= 16 && (a.bm == 16 || (a.bm == 64 && !fused)), "gqa_attention: %d key ranges, tile of %d rows", a.n_splits, a.bm);
        if (fused) return a.Vc <= 128 ? launch_gqa<1, 4, 128, true>(a, s) : launch_gqa<1, 4, 256, true>(a, s);
        if (a.bm == 16) return a.Vc <= 128 ? launch_gqa<1, 4, 128, false>(a, s) : launch_gqa<1, 4, 256, false>(a, s);
        return a.Vc <= 128 ? launch_gqa<4, 8, 128, false>(a, s) : launch_gqa<4, 8, 256, false>(a, s);
    }
    DLP_REQUIRE(!fused && a.n_splits == 1 && a.H <= 65535, "gqa_attention: this width takes prepared queries and one key range");
    const size_t smem = (size_t)(a.D + a.V + 192) * 4;
    DLP_REQUIRE(smem <= 48 * 1024, "gqa_attention: heads of %d and %d", a.D, a.V);
    DLP_CHECK_CUDA(f32 ? launch_pdl(gqa_attn_kernel<float>, dim3(a.n_tiles, a.H), dim3(128), smem, s, a)
                       : launch_pdl(gqa_attn_kernel<__nv_bfloat16>, dim3(a.n_tiles, a.H), dim3(128), smem, s, a));
    return 0;
}

}  // namespace dlp
