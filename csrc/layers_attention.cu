// Attention in the latent space of latent attention: the cached latent row is key and value of every head at once, the queries
// arrive multiplied into that space.  A tile is up to BM consecutive (token, head) rows of one request; rows of a tile share every
// latent row they read.  Scores and softmax weights stay in fp32: for the tensor cores a weight is split into two bf16 parts (the
// rounded value and the rest), whose products with the latent rows are summed.
//
// The values may be the leading columns only (behind them: a key part with positions that the heads share); a sliding window may hide early keys.
//
//   latent_attn_mma_kernel   bf16 latents up to 512 wide: mma.sync m16n8k16, latent tiles double-buffered with cp.async
//   latent_attn_kernel       any width, bf16 or fp32 storage
//   latent_combine_kernel    joins the key ranges of a split launch
#include "layers.cuh"
#include "mma.cuh"

namespace dlp {

struct KeyRange { int lo, hi; };           // the part that this split reads of the keys some row of the tile sees
__device__ __forceinline__ KeyRange tile_keys(const LatentArgs& a, int row_first, int row_last, int split, int step) {
    const int len = min(a.pos[row_last / a.H] + 1, a.max_pages * a.page_size), first = min(len, max(0, a.pos[row_first / a.H] - a.window + 1));
    const int per = ((len - first + a.n_splits - 1) / a.n_splits + step - 1) / step * step;
    KeyRange k;
    k.lo = min(len, first + split * per);
    k.hi = min(len, k.lo + per);
    return k;
}

// MW: 16-row blocks of a tile; NWARP warps share a tile as MW x (NWARP / MW); BN keys per step.  (Four warps and 32-key steps, two blocks
// to an SM, measured no faster for the 16- and 32-row decode tiles.)
template <int MW, int NWARP, int BN, int RMAX>
__global__ void __launch_bounds__(32 * NWARP, 1) latent_attn_mma_kernel(const LatentArgs a) {
    constexpr int NTH = 32 * NWARP, BM = 16 * MW, NW = NWARP / MW, KPW = BN / NW, LS = BN + 4;
    constexpr int NPAIR = (RMAX / 16 + NW - 1) / NW;      // 16-column output blocks of a warp
    extern __shared__ __align__(16) uint8_t la_smem[];
    const int Rc = a.Rc, Vc = a.Vc, LD = Rc + 8;
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(la_smem);
    __nv_bfloat16* cs = qs + BM * LD;                     // [2][BN][LD]
    float* S = reinterpret_cast<float*>(cs + 2 * BN * LD);
    float* s_alpha = S + BM * LS;
    float* s_l = s_alpha + BM;
    int* offs = reinterpret_cast<int*>(s_l + BM);         // [2][BN] cache row of every key of a tile (-1: outside the range)
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, mw = warp / NW, nw = warp % NW, g = lane >> 2, c = lane & 3;
    const int tile = blockIdx.x, split = blockIdx.y;
    pdl_wait();
    const int row0 = a.tile_row0[tile], rows = a.tile_rows[tile];
    if (rows <= 0) return;
    const KeyRange kr = tile_keys(a, row0, row0 + rows - 1, split, BN);
    const int* bt = a.block_table + (size_t)a.tok_slot[row0 / a.H] * a.max_pages;
    const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(a.cache);
    const int chunks = Rc / 8;
    auto find_rows = [&](int k0, int b) {
        if (tid < BN) {
            const int key = k0 + tid;
            offs[b * BN + tid] = key < kr.hi ? bt[key / a.page_size] * a.page_size + key % a.page_size : -1;
        }
    };
    auto load_tile = [&](int b) {           // eight threads per latent row
#pragma unroll
        for (int part = 0; part < BN / (NTH / 8); ++part) {
            const int kk = part * (NTH / 8) + (tid >> 3), row = offs[b * BN + kk];
            const __nv_bfloat16* src = cache + (size_t)max(row, 0) * Rc;
            __nv_bfloat16* dst = cs + ((size_t)b * BN + kk) * LD;
            for (int ch = tid & 7; ch < chunks; ch += 8) cp_async16(dst + ch * 8, src + ch * 8, row >= 0);
        }
        cp_commit();
    };
    const int n_tiles = (kr.hi - kr.lo + BN - 1) / BN;
    find_rows(kr.lo, 0);
    find_rows(kr.lo + BN, 1);
    __syncthreads();
    if (n_tiles > 0) load_tile(0);
    {
        const uint4* q = reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(a.q) + (size_t)row0 * Rc);
        for (int i = tid; i < BM * chunks; i += NTH) {
            const int r = i / chunks, ch = i - r * chunks;
            *reinterpret_cast<uint4*>(qs + r * LD + ch * 8) = r < rows ? q[(size_t)r * chunks + ch] : make_uint4(0, 0, 0, 0);
        }
    }
    constexpr int TPR = NTH / BM;                          // softmax threads per row
    const int sr = tid / TPR, sub = tid % TPR;
    const int my_pos = sr < rows ? a.pos[(row0 + sr) / a.H] : -1;
    float m_run = -INFINITY, l_run = 0.f;
    float acc[NPAIR][2][4] = {};
    for (int it = 0; it < n_tiles; ++it) {
        const int k0 = kr.lo + it * BN, b = it & 1;
        if (it + 1 < n_tiles) { load_tile(b ^ 1); cp_wait<1>(); } else { cp_wait<0>(); }
        __syncthreads();
        if (it + 2 < n_tiles) find_rows(k0 + 2 * BN, b);      // read behind the barriers of this iteration
        const __nv_bfloat16* ct = cs + (size_t)b * BN * LD;
        {   // scores: 16 rows x KPW keys per warp
            constexpr int NJ = KPW / 8, CH = NJ >= 4 ? 1 : NJ == 2 ? 2 : 4;      // independent accumulation chains
            float sacc[CH][NJ][4] = {};
#pragma unroll 2
            for (int k = 0; k < Rc; k += 16 * CH) {
#pragma unroll
                for (int x = 0; x < CH; ++x) {
                    if (CH > 2 && k + x * 16 >= Rc) break;           // Rc is a multiple of 32
                    uint32_t af[4];
                    ldsm_x4(af, qs + (mw * 16 + (lane & 15)) * LD + k + x * 16 + (lane >> 4) * 8);
#pragma unroll
                    for (int j = 0; j < NJ; ++j) {
                        uint32_t bf[2];
                        ldsm_x2(bf, ct + (nw * KPW + j * 8 + (lane & 7)) * LD + k + x * 16 + ((lane >> 3) & 1) * 8);
                        mma16816(sacc[x][j], af, bf[0], bf[1]);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < NJ; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    float v = sacc[0][j][e];
#pragma unroll
                    for (int x = 1; x < CH; ++x) v += sacc[x][j][e];
                    S[(mw * 16 + g + (e >> 1) * 8) * LS + nw * KPW + j * 8 + c * 2 + (e & 1)] = v * a.scale;
                }
        }
        __syncthreads();
        {   // running softmax
            float* row = S + sr * LS;
            float v[BN / TPR], mx = m_run;
#pragma unroll
            for (int i = 0; i < BN / TPR; ++i) {
                const int kk = i * TPR + sub, key = k0 + kk;
                v[i] = (key <= my_pos && key > my_pos - a.window && key < kr.hi) ? row[kk] : -INFINITY;
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
        {   // context: 16 rows x this warp's 16-column blocks
            const float a0 = s_alpha[mw * 16 + g], a1 = s_alpha[mw * 16 + g + 8];
#pragma unroll
            for (int j = 0; j < NPAIR; ++j)
#pragma unroll
                for (int n = 0; n < 2; ++n) { acc[j][n][0] *= a0; acc[j][n][1] *= a0; acc[j][n][2] *= a1; acc[j][n][3] *= a1; }
#pragma unroll
            for (int kk = 0; kk < BN / 16; ++kk) {
                uint32_t hi[4], lo[4];
                const float* r0 = S + (mw * 16 + g) * LS + kk * 16 + c * 2;
                const float* r1 = r0 + 8 * LS;
                split_bf16(r0[0], r0[1], hi[0], lo[0]);
                split_bf16(r1[0], r1[1], hi[1], lo[1]);
                split_bf16(r0[8], r0[9], hi[2], lo[2]);
                split_bf16(r1[8], r1[9], hi[3], lo[3]);
#pragma unroll
                for (int j = 0; j < NPAIR; ++j) {
                    const int col = (j * NW + nw) * 16;
                    if (col < Vc) {
                        uint32_t bf[4];
                        ldsm_x4_t(bf, ct + (kk * 16 + (lane & 15)) * LD + col + (lane >> 4) * 8);
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
    if (sub == 0) {
        s_l[sr] = l_run;
        if (a.n_splits > 1 && sr < rows) {
            float* ml = a.part_ml + ((size_t)split * a.T * a.H + row0 + sr) * 2;
            ml[0] = m_run;
            ml[1] = l_run;
        }
    }
    __syncthreads();
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = mw * 16 + g + half * 8;
        if (r >= rows) continue;
        const float inv = s_l[r] > 0.f ? 1.f / s_l[r] : 0.f;
        const size_t row = (size_t)row0 + r;
#pragma unroll
        for (int j = 0; j < NPAIR; ++j)
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const int col = (j * NW + nw) * 16 + n * 8 + c * 2;
                if (col >= Vc) continue;
                const float x = acc[j][n][half * 2], y = acc[j][n][half * 2 + 1];
                if (a.n_splits > 1)
                    *reinterpret_cast<float2*>(a.part_o + ((size_t)split * a.T * a.H + row) * Vc + col) = make_float2(x, y);
                else
                    *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<__nv_bfloat16*>(a.out) + row * Vc + col) = __floats2bfloat162_rn(x * inv, y * inv);
            }
    }
}

// ---- any width, any storage: one CTA per (token, head) row and key range --------------------------------------------
template <typename WT>
__global__ void __launch_bounds__(128) latent_attn_kernel(const LatentArgs a) {
    extern __shared__ __align__(16) uint8_t la_smem[];
    float* q = reinterpret_cast<float*>(la_smem);         // [Rc]
    float* acc = q + a.Rc;                                // [Vc]
    float* s = acc + a.Vc;                                // [64]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int row = blockIdx.x, t = row / a.H, split = blockIdx.y, Rc = a.Rc, Vc = a.Vc;
    pdl_wait();
    const KeyRange kr = tile_keys(a, row, row, split, 64);
    const int* bt = a.block_table + (size_t)a.tok_slot[t] * a.max_pages;
    const WT* cache = reinterpret_cast<const WT*>(a.cache);
    for (int r = tid; r < Rc; r += 128) {
        q[r] = (float)reinterpret_cast<const WT*>(a.q)[(size_t)row * Rc + r];
        if (r < Vc) acc[r] = 0.f;
    }
    float m = -INFINITY, l = 0.f;
    for (int k0 = kr.lo; k0 < kr.hi; k0 += 64) {
        __syncthreads();
        const int n = min(64, kr.hi - k0);
        for (int kk = warp; kk < 64; kk += 4) {
            float d = 0.f;
            if (kk < n) {
                const int key = k0 + kk;
                const WT* cr = cache + ((size_t)bt[key / a.page_size] * a.page_size + key % a.page_size) * Rc;
                for (int r = lane; r < Rc; r += 32) d = fmaf(q[r], (float)cr[r], d);
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
        for (int r = tid; r < Vc; r += 128) {
            float v = acc[r] * alpha;
            for (int kk = 0; kk < n; ++kk) {
                const int key = k0 + kk;
                v = fmaf(s[kk], (float)cache[((size_t)bt[key / a.page_size] * a.page_size + key % a.page_size) * Rc + r], v);
            }
            acc[r] = v;
        }
    }
    pdl_launch_dependents();
    if (a.n_splits > 1) {
        const size_t o = (size_t)split * a.T * a.H + row;
        for (int r = tid; r < Vc; r += 128) a.part_o[o * Vc + r] = acc[r];
        if (tid == 0) { a.part_ml[o * 2] = m; a.part_ml[o * 2 + 1] = l; }
    } else {
        const float inv = l > 0.f ? 1.f / l : 0.f;
        for (int r = tid; r < Vc; r += 128) reinterpret_cast<WT*>(a.out)[(size_t)row * Vc + r] = (WT)(acc[r] * inv);
    }
}

template <typename WT>
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentArgs a) {
    __shared__ float w[32];                       // weight of every key range
    pdl_wait();
    const int row = blockIdx.x, lane = threadIdx.x & 31;
    const size_t stride = (size_t)a.T * a.H;
    if (threadIdx.x < 32) {
        const bool ok = lane < a.n_splits;
        const float ms = ok ? a.part_ml[(lane * stride + row) * 2] : -INFINITY, ls = ok ? a.part_ml[(lane * stride + row) * 2 + 1] : 0.f;
        const float m = warp_max(ms), e = ms == -INFINITY ? 0.f : expf(ms - m);
        const float l = warp_sum(e * ls);
        w[lane] = l > 0.f ? e / l : 0.f;
    }
    __syncthreads();
    const int r = blockIdx.y * 128 + threadIdx.x;
    if (r < a.Vc) {
        float x[32], v = 0.f;
#pragma unroll
        for (int s = 0; s < 32; ++s) x[s] = (s < a.n_splits && w[s] != 0.f) ? a.part_o[(s * stride + row) * a.Vc + r] : 0.f;
#pragma unroll
        for (int s = 0; s < 32; ++s) v = fmaf(x[s], w[s], v);
        reinterpret_cast<WT*>(a.out)[(size_t)row * a.Vc + r] = (WT)v;
    }
    pdl_launch_dependents();
}

template <int MW, int NWARP, int BN, int RMAX>
static int launch_latent_mma(const LatentArgs& a, cudaStream_t s) {
    constexpr int BM = 16 * MW;
    const size_t smem = (size_t)(BM + 2 * BN) * (a.Rc + 8) * 2 + (size_t)BM * (BN + 4) * 4 + BM * 8 + 2 * BN * 4;
    DLP_REQUIRE(smem <= 227 * 1024, "latent_attention: %zu bytes of shared memory", smem);
    auto kern = latent_attn_mma_kernel<MW, NWARP, BN, RMAX>;
    if (first_use_on_device((const void*)kern)) DLP_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    DLP_CHECK_CUDA(launch_pdl(kern, dim3(a.n_tiles, a.n_splits), dim3(32 * NWARP), smem, s, a));
    return 0;
}
template <int RMAX>
static int launch_latent_tile(const LatentArgs& a, cudaStream_t s) {
    if (a.bm == 16) return launch_latent_mma<1, 8, 64, RMAX>(a, s);
    if (a.bm == 32) return launch_latent_mma<2, 8, 64, RMAX>(a, s);
    return launch_latent_mma<4, 8, 64, RMAX>(a, s);
}

int latent_attention(const LatentArgs& a, int f32, cudaStream_t s) {
    DLP_REQUIRE(a.q && a.cache && a.block_table && a.tok_slot && a.pos && a.out && a.tile_row0 && a.tile_rows, "latent_attention: null argument");
    DLP_REQUIRE(a.H > 0 && a.Rc > 0 && a.Rc % 32 == 0 && a.T > 0 && a.n_tiles > 0 && a.page_size > 0 && a.max_pages > 0, "latent_attention: bad shape");
    DLP_REQUIRE(a.Vc > 0 && a.Vc % 32 == 0 && a.Vc <= a.Rc && a.window >= 1, "latent_attention: values of %d of %d columns, window of %d", a.Vc, a.Rc, a.window);
    DLP_REQUIRE(a.n_splits >= 1 && a.n_splits <= 32 && (a.n_splits == 1 || (a.part_o && a.part_ml)), "latent_attention: %d key ranges", a.n_splits);
    int rc = 0;
    if (!f32 && a.Vc <= 512 && a.Rc <= 640) {
        DLP_REQUIRE(a.bm == 16 || a.bm == 32 || a.bm == 64, "latent_attention: tile of %d rows", a.bm);
        rc = a.Vc <= 128 ? launch_latent_tile<128>(a, s) : launch_latent_tile<512>(a, s);
    } else {
        const size_t smem = (size_t)(a.Rc + a.Vc + 64) * 4;
        DLP_REQUIRE(smem <= 48 * 1024, "latent_attention: latent of %d", a.Rc);
        DLP_CHECK_CUDA(f32 ? launch_pdl(latent_attn_kernel<float>, dim3(a.T * a.H, a.n_splits), dim3(128), smem, s, a)
                           : launch_pdl(latent_attn_kernel<__nv_bfloat16>, dim3(a.T * a.H, a.n_splits), dim3(128), smem, s, a));
    }
    if (rc) return rc;
    if (a.n_splits > 1) {
        if (f32) DLP_CHECK_CUDA(launch_pdl(latent_combine_kernel<float>, dim3(a.T * a.H, (a.Vc + 127) / 128), dim3(128), 0, s, a));
        else DLP_CHECK_CUDA(launch_pdl(latent_combine_kernel<__nv_bfloat16>, dim3(a.T * a.H, (a.Vc + 127) / 128), dim3(128), 0, s, a));
    }
    return 0;
}

}  // namespace dlp
