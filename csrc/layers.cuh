// Launcher interface of the layer-list kernels (layers_*.cu): models whose layers are described one by one (recurrent mixers, latent
// attention, windowed grouped-query attention, routed experts, norms in front of or behind the sublayers).  Every kernel exists in two
// storage forms: bf16 operands with fp32 accumulation, and fp32 throughout (`f32` != 0).
#pragma once
#include "kernels.cuh"

namespace dlp {

// How a row of x is formed before a matrix product (fused into the mat-vec prologue, or run by stage_rows_kernel for GEMM sizes):
//   v = x                                       (fp32 residual stream or activation-typed rows)
//   v = v + gnorm(y; groups1) * w1              when y and w1: norm of the sublayer's output, then the residual sum (-> h_out)
//   v = v + y                                   when y without w1: the output joins as it is (-> h_out)
//   v = v + e                                   when e: a second addend (the embedding output at the start of a loop pass; -> h_out)
//   v = gnorm(v; groups2) * w2[k % w2_mod]      when w2 without b2: final norm, or the per-head norm of a recurrent mixer
//   v = (v - mean) / sqrt(var + eps) * w2 + b2  when w2 and b2: layer norm over the row (groups2 = 1)
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
};

// GEGLU: weight rows 2i / 2i+1 are gate_i / up_i, the output is gelu_tanh(gate) * up.  RELU2: max(., 0)^2 in the activation type.
enum LinOut : int { LO_F32 = 0, LO_GEGLU = 1, LO_BF16 = 2, LO_RELU2 = 3 };

// Routed experts: logits + bias -> the `top` largest, weights = softmax over those.  Expert matrices are stacked, `rows` rows each.
constexpr int ROUTE_MAX_EXPERTS = 256, ROUTE_MAX_TOP = 32;
struct ExpertArgs {
    const float* logits;  // [T, ldl] without the bias
    const float* bias;    // [n_expert] (nullptr: none)
    const void* w;        // [n_expert * rows, ldw]
    int ldl, n_expert, top, rows, ldw;
};

int matvec(const RowStage& st, const void* w, int ldw, int N, void* out, int ldo, int out_mode, int T, int f32, cudaStream_t s);
int stage_rows(const RowStage& st, void* xb, int ldxb, int T, int f32, cudaStream_t s);
int sgemm(const float* x, int ldx, const float* w, int ldw, int N, int K, void* out, int ldo, int out_mode, int T, cudaStream_t s, const GemmGroup* grp = nullptr);
// 1..4 rows: down = 0: relu(W_e h)^2 of every chosen expert -> act [T * top, ldo]; down = 1: sum of the weighted W_e act rows -> fp32 [T, ldo]
int expert_matvec(const RowStage& st, const ExpertArgs& a, void* out, int ldo, int down, int T, int f32, cudaStream_t s);
int route(const float* logits, int ld, const float* bias, int n_expert, int top, int* ids, float* w, int T, cudaStream_t s);
int head_matmul(const void* x, int x_f32, int ldx, int x_head, int kx, const void* w, int Kp, int H, int N, int n_rows, void* out, int ldo, int out_head,
                const float* gate, int ldg, int T, int f32, cudaStream_t s);
int embed_rows(const void* table, int ld, const int* ids, float* h, int E, int T, int vocab, int f32, cudaStream_t s);
int latent_write(const float* proj, int ldp, const float* w, float eps, int R, int Rc, const int* slot, void* cache, int T, int f32, cudaStream_t s);

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
struct Hgrn2Chunks {
    const int* chunk;     // [n_chunks][2] first token, number of tokens (chunks of a segment follow each other)
    const int* first;     // [n_seg + 1] first chunk of every segment
    float* states;        // [n_chunks, H, D, V] workspace: what a chunk adds to the state, then the state a chunk starts from
    float* decay;         // [n_chunks, H, D] workspace
    int n_chunks, pad;
};
int hgrn2_scan(const Hgrn2Args& a, cudaStream_t s);
int hgrn2_chunked(const Hgrn2Args& a, const Hgrn2Chunks& c, cudaStream_t s);

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

// One warp: the `top` largest of logits + bias (ties: the lower index first) and the softmax over them, into ids[top] and w[top].
__device__ __forceinline__ void route_row(const float* logits, const float* bias, int n_expert, int top, int* ids, float* w) {
    const int lane = threadIdx.x & 31;
    float v[ROUTE_MAX_EXPERTS / 32];
#pragma unroll
    for (int i = 0; i < ROUTE_MAX_EXPERTS / 32; ++i) {
        const int e = lane + 32 * i;
        v[i] = e < n_expert ? logits[e] + (bias ? bias[e] : 0.f) : -INFINITY;
    }
    float mine = -INFINITY;              // lane j keeps the j-th choice
    int mine_id = 0;
    for (int j = 0; j < top; ++j) {
        float best = -INFINITY;
        int bi = 0x7fffffff;
#pragma unroll
        for (int i = 0; i < ROUTE_MAX_EXPERTS / 32; ++i)
            if (v[i] > best || (v[i] == best && bi == 0x7fffffff && lane + 32 * i < n_expert)) { best = v[i]; bi = lane + 32 * i; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
        }
        bi = min(bi, n_expert - 1);      // logits that are no numbers choose some expert, not a place outside the stack
        if (lane == j) { mine = best; mine_id = bi; }
#pragma unroll
        for (int i = 0; i < ROUTE_MAX_EXPERTS / 32; ++i)
            if (bi == lane + 32 * i) v[i] = -INFINITY;
    }
    const float m = __shfl_sync(0xffffffffu, mine, 0);
    const float p = lane < top ? expf(mine - m) : 0.f;
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
    void* out;                // [T, H, Rc]
    float* part_o;            // [n_splits][T * H][Rc]  (n_splits > 1)
    float* part_ml;           // [n_splits][T * H][2]
    int max_pages, page_size, H, Rc, T, n_tiles, bm, n_splits;
    float scale;
};
int latent_attention(const LatentArgs& a, int f32, cudaStream_t s);
int latent_gather(const void* cache, const int* bt, int page, int Rc, void* out, int S, cudaStream_t s);
int head_rows(const float* x, int ldx, int D, int Dp, int H, void* out, int T, cudaStream_t s);
int rows_attention(const void* q, const void* kv, int ldkv, int S, int T, int pos0, int H, int Dp, int Vp, int V, float scale, const float* gate, int ldg, void* out, int ldo,
                   cudaStream_t s);
int rows_attention_error(int* flag);
int* flash_error_flag();      // device flag a bounded wait raises (nullptr: error set)


// Grouped-query softmax attention over paged keys and values [pages, G, page, Dc | Vc]: position i sees key j <= i when i - j < window
// or j < keep.  Queries and keys are RMS-normalised over their whole projection (when q_norm / k_norm are given) and rotated (half-split
// pairs of the first `rot` dimensions) before they are used or cached.
struct GqaArgs {
    const float* proj;        // [T, ldp]: q [H * D] | k [G * D] | v [G * V]
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
    void* out;                // [T, ldo]
    int ldp, ldo, T, H, G, D, V, Dc, Vc, rot, max_pages, page_size, n_pages, n_tiles, bm, n_splits, window, keep;
    float eps, scale;
};
int gqa_prepare(const GqaArgs& a, int f32, cudaStream_t s);                   // proj -> q rows and cache rows
int gqa_attention(const GqaArgs& a, int fused, int f32, cudaStream_t s);      // tiles of (token, head) rows; fused: single tokens straight from proj
int gqa_flash(const GqaArgs& a, cudaStream_t s);                              // bf16, 128-token tiles, tcgen05

}  // namespace dlp
