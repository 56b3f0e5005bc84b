// Launcher interface of the layer-list kernels (layers_linear.cu, layers_mixers.cu, layers_attention.cu): models whose layers are
// described one by one (recurrent mixers, latent attention, norms behind the sublayers).  Every kernel exists in two storage forms:
// bf16 operands with fp32 accumulation, and fp32 throughout (`f32` != 0).
#pragma once
#include "common.cuh"

namespace dlp {

// How a row of x is formed before a matrix product (fused into the mat-vec prologue, or run by stage_rows_kernel for GEMM sizes):
//   v = x                                       (fp32 residual stream or activation-typed rows)
//   v = v + gnorm(y; groups1) * w1              when y != nullptr: norm of the sublayer's output, then the residual sum (-> h_out)
//   v = gnorm(v; groups2) * w2[k % w2_mod]      when w2 != nullptr: final norm, or the per-head norm of a recurrent mixer
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
};

enum LinOut : int { LO_F32 = 0, LO_GEGLU = 1, LO_BF16 = 2 };   // GEGLU: weight rows 2i / 2i+1 are gate_i / up_i, the output is gelu_tanh(gate) * up

int matvec(const RowStage& st, const void* w, int ldw, int N, void* out, int ldo, int out_mode, int T, int f32, cudaStream_t s);
int stage_rows(const RowStage& st, void* xb, int ldxb, int T, int f32, cudaStream_t s);
int sgemm(const float* x, int ldx, const float* w, int ldw, int N, int K, void* out, int ldo, int out_mode, int T, cudaStream_t s);
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

}  // namespace dlp
