// Launcher interface of the layer-list kernels (layers_*.cu): models whose layers are described one by one (recurrent mixers, latent
// attention, windowed grouped-query attention, routed experts, norms in front of or behind the sublayers).  Every kernel exists in two
// storage forms: bf16 operands with fp32 accumulation, and fp32 throughout (`f32` != 0).
#pragma once
#include "kernels.cuh"

namespace dlp {

// How a row of x is formed before a matrix product (fused into the mat-vec prologue, or run by stage_rows_kernel for GEMM sizes):
//   v = x                                       (fp32 residual stream or activation-typed rows)
//   v = x1 - lam * x2                           when pair: x rows hold two vectors of `pair` values for every head, x1 and x2 of them
//   v = v * silu(g)                             when gate == 2
//   v = v + gnorm(y; groups1) * w1              when y and w1: norm of the sublayer's output, then the residual sum (-> h_out)
//   v = v + y                                   when y without w1: the output joins as it is (-> h_out)
//   v = v + e                                   when e: a second addend (the embedding output at the start of a loop pass; -> h_out)
//   v = gnorm(v; groups2) * w2[k % w2_mod]      when w2 without b2: final norm, or the per-head norm of a recurrent mixer
//   v = (v - mean) / sqrt(var + eps) * w2 + b2  when w2 and b2: layer norm over the row (groups2 = 1)
//   v = v * sigmoid(g)                          when gate == 1;  v * silu(g) when gate == 3
// and behind the row's Kp values, `tail` values in the activation type as they are (the other half of a stacked product's input; mat-vec only).
// (pair and gate come with mixer outputs, y and e with the residual stream: never both)
// gnorm splits the row into equal consecutive groups and divides each by its own sqrt(mean square + eps).
struct RowStage {
    const void* x;
    int x_f32;            // x is fp32 (else: activation type)
    int ldx;
    const float* y;
    int ldy;
    const float* w1;
    int groups1;
    float* h_out;         // where the updated residual stream goes (written once; nullptr: not kept)
    int ldh;
    const float* w2;
    int groups2, w2_mod;
    float eps;
    int K;                // row width; K .. Kp-1 are staged as zeros
    int Kp;
    const float* b2;
    const float* e;
    int lde;
    int pair;             // values of one map and head (0: x is used as it is)
    const float* g;       // [T, ldg] logits of the gate
    int ldg;
    int gate;             // GATE_*
    float lam;
    const void* tail;     // [T, ld_tail]
    int ld_tail, K_tail;
};
enum RowGate : int { GATE_NONE = 0, GATE_SIGMOID_AFTER = 1, GATE_SILU_BEFORE = 2, GATE_SILU_AFTER = 3 };

// GEGLU, SWIGLU: weight rows 2i / 2i+1 are gate_i / up_i, the output is gelu_tanh(gate) * up or silu(gate) * up.  RELU2: max(., 0)^2.
// All three in the activation type.
enum LinOut : int { LO_F32 = 0, LO_GEGLU = 1, LO_BF16 = 2, LO_RELU2 = 3, LO_SWIGLU = 4 };

// Routed experts.  softmax: logits + bias -> the `top` largest, weights = softmax over those.  sigmoid: s = sigmoid(logits), choice by s + bias -
// first the `keep` best of `groups` groups of neighbours (by their two largest), then the `top` largest of those; weights = the chosen s
// divided by their sum, times scale.  Expert matrices are stacked, `rows` rows each.
constexpr int ROUTE_MAX_EXPERTS = 256, ROUTE_MAX_TOP = 32;
struct RouteRule {
    const float* bias;    // [n_expert] (nullptr: none)
    int n_expert, top, sigmoid, groups, keep;
    float scale;
};
struct ExpertArgs {
    const float* logits;  // [T, ldl] without the bias; with a shared expert column n_expert is the logit of its gate
    RouteRule rule;
    const void* w;        // [n_expert * rows, ldw]
    int ldl, rows, ldw;
    int act;              // up products: LO_RELU2, or LO_SWIGLU over interleaved rows
    // an expert that every token uses, weighted by the sigmoid of its own logit (w_s nullptr: none)
    const void* w_s;      // [rows_s, ldw_s]
    const void* x_s;      // down: its rows [T, ldx_s]
    void* act_s;          // up: its output [T, ld_act_s]
    int rows_s, K_s;      // up: rows of w_s;  down: its inner size (padded)
    int ldw_s, ldx_s, ld_act_s;
};

int matvec(const RowStage& st, const void* w, int ldw, int N, void* out, int ldo, int out_mode, int T, int f32, cudaStream_t s, const OutTail* tail = nullptr);
int stage_rows(const RowStage& st, void* xb, int ldxb, int T, int f32, cudaStream_t s);
int sgemm(const float* x, int ldx, const float* w, int ldw, int N, int K, void* out, int ldo, int out_mode, int T, cudaStream_t s, const GemmGroup* grp = nullptr,
          const OutTail* tail = nullptr);
// 1..4 rows: down = 0: act(W_e h) of every chosen expert -> act [T * top, ldo]; down = 1: sum of the weighted W_e act rows -> fp32 [T, ldo]
int expert_matvec(const RowStage& st, const ExpertArgs& a, void* out, int ldo, int down, int T, int f32, cudaStream_t s);
int route(const float* logits, int ld, const RouteRule& rule, int* ids, float* w, int T, cudaStream_t s);
int head_matmul(const void* x, int x_f32, int ldx, int x_head, int kx, const void* w, int Kp, int H, int N, int n_rows, void* out, int ldo, int out_head,
                const float* gate, int ldg, int T, int f32, cudaStream_t s);
int embed_rows(const void* table, int ld, const int* ids, float* h, int E, int T, int vocab, float scale, int f32, cudaStream_t s);
// Cache rows of latent attention: the first R columns behind their RMS norm, then `rot` columns turned by their position; with q also the last
// `rot` of every head's Dq query columns, in place.  Pairs are neighbours when `adjacent`, else half-split.
struct LatentRows {
    const float* proj;        // [T, ldp]
    const float* w;           // [R]
    const int* slot;          // [T] (below zero: not cached)
    void* cache;              // rows of Rc
    const int* pos;           // [T]
    const float* inv_freq;    // [rot / 2]
    float* q;                 // [T, ldq] (nullptr: none)
    int ldp, R, Rc, rot, adjacent, ldq, H, Dq;
    float eps, rot_scale;     // rot_scale: factor on cosine and sine
};
int latent_write(const LatentRows& a, int T, int f32, cudaStream_t s);

struct Hgrn2Args {
    const float* proj;    // [T, ldp]: q_raw [H*D] | f_raw [H*D] | v [H*V]
    int ldp;
    const float* fbias;   // [H*D]
    const float* lower;   // [H*D]
    float* state;         // [slots, H, D, V]
    const int* seg;       // [n_seg][2] token range of every segment
    const int* seg_slot;  // [n_seg] state slot
    const int* pos;       // [T] (a segment that starts at position 0 starts from the zero state)
    float* out;           // [T, ldo]
    int ldo, H, D, V, n_seg;
};
// Long segments in chunks of HGRN2_CHUNK tokens (layers_hgrn2.cu); `a.seg` / `a.seg_slot` list those segments only.
constexpr int HGRN2_CHUNK = 64;
struct ScanChunks {
    const int* chunk;     // [n_chunks][2] first token, number of tokens (chunks of a segment follow each other)
    const int* first;     // [n_seg + 1] first chunk of every segment
    float* states;        // [n_chunks, H, D, V] workspace: what a chunk adds to the state, then the state a chunk starts from
    float* decay;         // [n_chunks, H, D] workspace
    int n_chunks, pad;
};
int hgrn2_scan(const Hgrn2Args& a, cudaStream_t s);
int hgrn2_chunked(const Hgrn2Args& a, const ScanChunks& c, cudaStream_t s);

// Recurrences with one decay per head and token (layers_ssd.cu): S <- f S + dt k v^T, o = S^T q (+ skip v).  `hpg` consecutive heads share q and k.
//   constant decay (dt nullptr):  f = decay[h], log_decay[h] its logarithm, dt = 1
//   step sizes:                   dt = softplus(raw dt + dt_bias[h]), f = exp(log_decay[h] * dt)
struct SsdArgs {
    const void* q;        // rows of T tokens: first column of the first head; fp32 or (rows_f32 = 0) bf16
    const void* k;
    const void* v;
    const float* decay;     // [H]
    const float* log_decay; // [H]
    const float* dt;        // [T, lddt]
    const float* dt_bias;   // [H]
    const float* skip;      // [H] (nullptr: none)
    float* state;           // [slots, H, D, V]
    const int* seg;         // [n_seg][2]
    const int* seg_slot;
    const int* pos;         // [T]
    float* out;             // [T, ldo]
    int ldq, ldk, ldv, rows_f32, act, hpg, lddt, ldo, H, D, V, n_seg;      // act: silu on q, k and v
};
// Causal convolution per channel with silu behind it.  The last inputs of a sequence are kept in a ring of `taps` rows: position p in row p % taps
// (one row more than the next token needs, so that a single token's row overwrites nothing another block still reads).
struct ConvArgs {
    const float* x;       // [T, ldx]
    const float* w;       // [taps, channels], the last row is the current token's
    const float* b;       // [channels] (nullptr: none)
    float* ring;          // [slots, taps, channels]
    int ldx, taps, channels;
};
int ssd_scan(const SsdArgs& a, cudaStream_t s);
constexpr int SSD_CHUNK = 128;
int ssd_chunked(const SsdArgs& a, const ScanChunks& c, cudaStream_t s);                 // chunks of SSD_CHUNK tokens; c.decay: [n_chunks, H]
int ssd_decode(const SsdArgs& a, const ConvArgs* conv, cudaStream_t s);                 // one token per segment; conv: q, k, v point into conv->x
int conv_rows(const ConvArgs& c, const int* seg, const int* seg_slot, const int* pos, int n_seg, int longest, void* out, int ldo, int f32, cudaStream_t s);

// Gated delta rule (layers_delta.cu): S <- f S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.  q and k are made unit vectors per head
// (x / sqrt(sum x^2 + unit_eps)), q is scaled by q_scale;  f = exp(log_decay[h] softplus(a + dt_bias[h])), beta = sigmoid(b).
struct DeltaArgs {
    const void* q;            // rows of T tokens behind convolution and activation: first column of the first head; fp32 or (rows_f32 = 0) bf16
    const void* k;
    const void* v;
    const float* a;           // [T, lda]
    const float* b;           // [T, ldb]
    const float* log_decay;   // [H]
    const float* dt_bias;     // [H]
    float* state;             // [slots, H, D, V]
    const int* seg;           // [n_seg][2]
    const int* seg_slot;
    const int* pos;           // [T]
    float* out;               // [T, ldo]
    int ldq, ldk, ldv, rows_f32, hpg, lda, ldb, ldo, H, D, V, n_seg;      // hpg consecutive heads share q and k
    float unit_eps, q_scale;
};
constexpr int DELTA_CHUNK = 64;
// Workspaces of the chunked form, in the layouts in which they are read into shared memory.  Dp: D rounded up to 64 or 128; S: slices of 16 value
// columns; pairs of bf16 parts are value and remainder.
constexpr int DELTA_ROW = DELTA_CHUNK + 8;      // row of a 64 x 64 matrix
struct DeltaChunks {
    const int* chunk;         // [n_chunks][2], as in ScanChunks
    const int* first;         // [n_seg + 1]
    void* states;             // [n_chunks, H, S][2][Dp][16] bf16: the state a chunk starts from
    void* keys;               // [n_chunks, H / hpg][64][Dp + 8] bf16
    void* solve;              // [n_chunks, H][2][64][DELTA_ROW] bf16: the chunk's triangular inverse
    void* weights;            // [n_chunks, H][2][64][DELTA_ROW] bf16: what a token's output takes of every write up to its own
    void* u;                  // [n_chunks, H, S][2][64][16] bf16: what every token writes
    float* gates;             // [n_chunks, H][64 x 4 | 64]: write strength, the same times decay from the chunk's start / |k|, decay to its end / |k|,
                              //                             decay of the whole chunk | decay from the start times scale / |q|
    int n_chunks, pad;
};
int delta_scan(const DeltaArgs& a, cudaStream_t s);
int delta_decode(const DeltaArgs& a, const ConvArgs* conv, cudaStream_t s);        // one token per segment; conv: q, k, v point into conv->x
int delta_chunked(const DeltaArgs& a, const DeltaChunks& c, cudaStream_t s);

#ifdef __CUDACC__
template <typename T> struct Act;
template <> struct Act<__nv_bfloat16> {
    static constexpr int VEC = 8;
    static __device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
    static __device__ __forceinline__ __nv_bfloat16 from_f(float v) { return __float2bfloat16_rn(v); }
};
template <> struct Act<float> {
    static constexpr int VEC = 4;
    static __device__ __forceinline__ float to_f(float v) { return v; }
    static __device__ __forceinline__ float from_f(float v) { return v; }
};

// where the result is rounded to bf16
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }
__device__ __forceinline__ float sigmoid_exact(float z) {
    const float e = expf(-fabsf(z)), hi = 1.f / (1.f + e);
    return z >= 0.f ? hi : e * hi;
}

// One warp: close the experts outside the `keep` best of `groups` groups of neighbours.  v holds the choice scores of experts lane + 32 i; a
// group's score is the sum of its two largest (of its only one).  scores, ranks: ROUTE_MAX_EXPERTS floats of shared memory each.  A power of two
// of lanes shares a group.
__device__ __forceinline__ void route_groups(const RouteRule& r, float* scores, float* ranks, float (&v)[ROUTE_MAX_EXPERTS / 32]) {
    const int lane = threadIdx.x & 31, size = r.n_expert / r.groups;
#pragma unroll
    for (int i = 0; i < ROUTE_MAX_EXPERTS / 32; ++i)
        if (lane + 32 * i < r.n_expert) scores[lane + 32 * i] = v[i];
    __syncwarp();
    int lg = 0;                          // log2 of the lanes that share a group
    while ((r.groups << (lg + 1)) <= 32) ++lg;
    const int share = 1 << lg;
#pragma unroll 1
    for (int g0 = 0; g0 < r.groups; g0 += 32 >> lg) {
        const int g = g0 + (lane >> lg);
        float a = -INFINITY, b = -INFINITY;
        if (g < r.groups)
#pragma unroll 1
            for (int e = g * size + (lane & (share - 1)); e < (g + 1) * size; e += share) {
                const float c = scores[e];
                b = fmaxf(b, fminf(a, c));
                a = fmaxf(a, c);
            }
#pragma unroll 1
        for (int o = 1; o < share; o <<= 1) {
            const float a2 = __shfl_xor_sync(0xffffffffu, a, o), b2 = __shfl_xor_sync(0xffffffffu, b, o);
            b = fmaxf(fminf(a, a2), fmaxf(b, b2));
            a = fmaxf(a, a2);
        }
        if (g < r.groups && (lane & (share - 1)) == 0) ranks[g] = size > 1 ? a + b : a;
    }
    __syncwarp();
#pragma unroll 1
    for (int g = lane; g < r.groups; g += 32) {
        const float mine = ranks[g];
        int better = 0;                  // groups ahead of this one (equal scores: the lower group first)
#pragma unroll 4
        for (int j = 0; j < r.groups; ++j) better += ranks[j] > mine || (ranks[j] == mine && j < g);
        scores[g] = better < r.keep ? 1.f : 0.f;          // the choice scores have been read
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < ROUTE_MAX_EXPERTS / 32; ++i) {
        if (32 * i >= r.n_expert) break;
        const int e = lane + 32 * i;
        if (e < r.n_expert && scores[e / size] == 0.f) v[i] = -INFINITY;
    }
}

// floats as unsigned numbers of the same order
__device__ __forceinline__ unsigned order_key(float x) {
    const unsigned u = __float_as_uint(x);
    return u ^ (u >> 31 ? 0xffffffffu : 0x80000000u);
}
__device__ __forceinline__ float order_value(unsigned k) { return __uint_as_float(k ^ (k >> 31 ? 0x80000000u : 0xffffffffu)); }

// One warp: chosen experts (ties: the lower index first) and their weights, into ids[top] and w[top]; scratch: ROUTE_SCRATCH floats of shared
// memory.
constexpr int ROUTE_SCRATCH = 3 * ROUTE_MAX_EXPERTS;
__device__ __forceinline__ void route_row(const float* logits, const RouteRule& r, float* scratch, int* ids, float* w) {
    constexpr int NG = ROUTE_MAX_EXPERTS / 32;
    const int lane = threadIdx.x & 31, n_expert = r.n_expert, top = r.top;
    float v[NG];
#pragma unroll
    for (int i = 0; i < NG; ++i) v[i] = -INFINITY;
#pragma unroll
    for (int i = 0; i < NG; ++i) {
        if (32 * i >= n_expert) break;
        const int e = lane + 32 * i;
        if (e < n_expert) {
            const float z = logits[e], b = r.bias ? r.bias[e] : 0.f;
            if (r.sigmoid) {
                const float s = sigmoid_exact(z);
                scratch[ROUTE_MAX_EXPERTS + e] = s;
                v[i] = s + b;
            } else {
                v[i] = z + b;
            }
        }
    }
    if (r.sigmoid && r.keep < r.groups) route_groups(r, scratch, scratch + 2 * ROUTE_MAX_EXPERTS, v);
    unsigned key[NG];                    // 0: not to be chosen (again)
#pragma unroll
    for (int i = 0; i < NG; ++i) key[i] = lane + 32 * i < n_expert ? order_key(v[i]) : 0u;
    unsigned mine = 0u;                  // lane j keeps the j-th choice
    int mine_id = 0;
    for (int j = 0; j < top; ++j) {
        unsigned best = 0u;
        int bi = 0x7fffffff;
#pragma unroll
        for (int i = 0; i < NG; ++i)
            if (key[i] > best) { best = key[i]; bi = lane + 32 * i; }
        const unsigned m = __reduce_max_sync(0xffffffffu, best);
        const int id = min(__reduce_min_sync(0xffffffffu, best == m ? bi : 0x7fffffff), n_expert - 1);
        if (lane == j) { mine = m; mine_id = id; }
#pragma unroll
        for (int i = 0; i < NG; ++i)
            if (id == lane + 32 * i) key[i] = 0u;
    }
    if (r.sigmoid) {
        __syncwarp();
        const float p = lane < top ? scratch[ROUTE_MAX_EXPERTS + mine_id] : 0.f;
        const float sum = warp_sum(p);
        if (lane < top) { ids[lane] = mine_id; w[lane] = p / (sum + 1e-20f) * r.scale; }
        return;
    }
    const float x = order_value(mine), m = __shfl_sync(0xffffffffu, x, 0);
    const float p = lane < top ? expf(x - m) : 0.f;
    const float sum = warp_sum(p);
    if (lane < top) { ids[lane] = mine_id; w[lane] = p / sum; }
}

// 1 - f = (1 - l) sigmoid(-z) is formed on its own: the difference would lose its digits where f is close to one.
__device__ __forceinline__ void hgrn2_gate(float z, float l, float& f, float& k) {
    const float e = expf(-fabsf(z)), hi = 1.f / (1.f + e), lo = e * hi;     // sigmoid(|z|), sigmoid(-|z|)
    const float sp = z >= 0.f ? hi : lo, sn = z >= 0.f ? lo : hi;
    f = l + (1.f - l) * sp;
    k = (1.f - l) * sn;
}
__device__ __forceinline__ float silu_exact(float z) {
    const float e = expf(-fabsf(z)), hi = 1.f / (1.f + e);
    return z * (z >= 0.f ? hi : e * hi);
}
#endif

struct LatentArgs {
    const void* q;            // [T, H, Rc] absorbed queries
    const void* cache;        // [pages, page, Rc]
    const int* block_table;   // [slots, max_pages]
    const int* tok_slot;      // [T] block-table row of every token
    const int* pos;           // [T]
    const int* tile_row0;     // [n_tiles] first (token * H + head) row of a tile; a tile never spans two requests
    const int* tile_rows;     // [n_tiles]
    void* out;                // [T, H, Vc]
    float* part_o;            // [n_splits][T * H][Vc]  (n_splits > 1)
    float* part_ml;           // [n_splits][T * H][2]
    int max_pages, page_size, H, Rc, Vc, T, n_tiles, bm, n_splits, window;      // Vc: leading columns of a cached row that are values; position i sees i - window + 1 .. i
    float scale;
};
int latent_attention(const LatentArgs& a, int f32, cudaStream_t s);
int latent_gather(const void* cache, const int* bt, int page, int Rc, void* out, int S, cudaStream_t s);
int head_rows(const float* x, int ldx, int D, int Dp, int H, void* out, int T, cudaStream_t s);
int rows_attention(const void* q, const void* kv, int ldkv, int S, int T, int pos0, int H, int Dp, int Vp, int V, int window, float scale, const float* gate, int ldg, void* out,
                   int ldo, cudaStream_t s);
int rows_attention_error(int* flag);
int* flash_error_flag();      // device flag a bounded wait raises (nullptr: error set)


// Grouped-query softmax attention over paged keys [pages, G * maps, page, Dc] and values [pages, G, page, Vc]: position i sees key j <= i
// when i - j < window and (chunk > 0) both lie in the same chunk, or when j < keep.  Queries and keys are RMS-normalised over their whole projection (when q_norm / k_norm are given) and
// rotated (the first `rot` dimensions: half-split pairs, or neighbours when `adjacent`) before they are used or cached.
// maps = 2: a head is two attentions over the same values; H counts (head, map) query rows, row h reads key head g * 2 + h % 2 of its
// key / value head g, and every row's result is kept, in fp32 (RowStage joins them).
struct GqaArgs {
    const float* proj;        // [T, ldp]: q [H * D] | k [G * maps * D] | v [G * V]
    const float* q_norm;
    const float* k_norm;
    const float* inv_freq;    // [rot / 2]
    void* q;                  // [T, H * Dc] prepared queries (not used by the fused decode form)
    void* kc;
    void* vc;
    const int* block_table;   // [slots, max_pages]
    const int* tok_slot;      // [T]
    const int* pos;           // [T]
    const int* slot;          // [T] cache row
    const int* tile_row0;     // [n_tiles] first token of a tile; tokens of a tile follow each other in one request
    const int* tile_rows;     // [n_tiles] tokens
    void* out;                // [T, ldo] (maps > 1: fp32)
    int ldp, ldo, T, H, G, D, V, Dc, Vc, rot, max_pages, page_size, n_pages, n_tiles, bm, n_splits, window, keep, chunk, maps, adjacent;
    float eps, scale;
    float rot_scale;          // factor on cosine and sine
    float* v_first;           // [T, G * V] values that several layers share a part of: written (v_mix 1), or mixed in (v_mix 2): (1 - v_lam) v + v_lam v_first
    int v_mix;
    float v_lam;
};
int gqa_prepare(const GqaArgs& a, int f32, cudaStream_t s);                   // proj -> q rows and cache rows
int gqa_attention(const GqaArgs& a, int fused, int f32, cudaStream_t s);      // tiles of (token, head) rows; fused: single tokens straight from proj
int gqa_flash(const GqaArgs& a, cudaStream_t s);                              // bf16, 128-token tiles, tcgen05

}  // namespace dlp
