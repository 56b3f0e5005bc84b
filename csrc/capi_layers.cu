// C surface of the layer-list kernels (declarations: include/dlp_b200.h).
#include <string.h>

#include "../include/dlp_b200.h"
#include "kernels.cuh"
#include "layers.cuh"

using namespace dlp;

static_assert(sizeof(dlp_row_stage) == sizeof(RowStage) && sizeof(dlp_hgrn2_args) == sizeof(Hgrn2Args) && sizeof(dlp_hgrn2_chunks) == sizeof(Hgrn2Chunks) && sizeof(dlp_latent_args) == sizeof(LatentArgs), "argument layout");

extern "C" {

int dlp_layers_matvec(const dlp_row_stage* st, const void* w, int ldw, int N, void* out, int ldo, int out_mode, int T, int f32, void* stream) {
    DLP_REQUIRE(st, "dlp_layers_matvec: null argument");
    return matvec(*reinterpret_cast<const RowStage*>(st), w, ldw, N, out, ldo, out_mode, T, f32, (cudaStream_t)stream);
}
int dlp_layers_stage_rows(const dlp_row_stage* st, void* xb, int ldxb, int T, int f32, void* stream) {
    DLP_REQUIRE(st, "dlp_layers_stage_rows: null argument");
    return stage_rows(*reinterpret_cast<const RowStage*>(st), xb, ldxb, T, f32, (cudaStream_t)stream);
}
int dlp_layers_linear(const void* x, int ldx, const void* w, int ldw, int N, int K, void* out, int ldo, int out_mode, int T, int f32, void* ws, size_t ws_bytes, void* stream) {
    DLP_REQUIRE(x && w && out && N > 0 && T > 0, "dlp_layers_linear: bad argument");
    if (f32) return sgemm((const float*)x, ldx, (const float*)w, ldw, N, K, out, ldo, out_mode, T, (cudaStream_t)stream);
    if (out_mode == LO_GEGLU)       // rows 2i / 2i+1 of the interleaved matrix: two operands with twice the row stride
        return gemm_f16(w, (const uint8_t*)w + (size_t)ldw * 2, 2 * ldw, x, ldx, out, ldo, T, N / 2, K, 6, 1, 0, (cudaStream_t)stream, nullptr, nullptr, ws, ws_bytes);
    DLP_REQUIRE(out_mode == LO_F32 || out_mode == LO_BF16, "dlp_layers_linear: output mode %d", out_mode);
    return gemm_f16(w, nullptr, ldw, x, ldx, out, ldo, T, N, K, out_mode == LO_BF16 ? 4 : 1, 1, 0, (cudaStream_t)stream, nullptr, nullptr, ws, ws_bytes);
}
int dlp_layers_head_matmul(const void* x, int x_f32, int ldx, int x_head, int kx, const void* w, int Kp, int H, int N, int n_rows, void* out, int ldo, int out_head,
                           const float* gate, int ldg, int T, int f32, void* stream) {
    return head_matmul(x, x_f32, ldx, x_head, kx, w, Kp, H, N, n_rows, out, ldo, out_head, gate, ldg, T, f32, (cudaStream_t)stream);
}
int dlp_layers_embed(const void* table, int ld, const int32_t* ids, float* h, int E, int T, int vocab, int f32, void* stream) {
    return embed_rows(table, ld, ids, h, E, T, vocab, f32, (cudaStream_t)stream);
}
int dlp_layers_latent_write(const float* proj, int ldp, const float* w, float eps, int R, int Rc, const int32_t* slot, void* cache, int T, int f32, void* stream) {
    return latent_write(proj, ldp, w, eps, R, Rc, slot, cache, T, f32, (cudaStream_t)stream);
}
int dlp_layers_hgrn2(const dlp_hgrn2_args* a, const dlp_hgrn2_chunks* chunks, void* stream) {
    DLP_REQUIRE(a, "dlp_layers_hgrn2: null argument");
    if (chunks) return hgrn2_chunked(*reinterpret_cast<const Hgrn2Args*>(a), *reinterpret_cast<const Hgrn2Chunks*>(chunks), (cudaStream_t)stream);
    return hgrn2_scan(*reinterpret_cast<const Hgrn2Args*>(a), (cudaStream_t)stream);
}
int dlp_layers_latent_attention(const dlp_latent_args* a, int f32, void* stream) {
    DLP_REQUIRE(a, "dlp_layers_latent_attention: null argument");
    return latent_attention(*reinterpret_cast<const LatentArgs*>(a), f32, (cudaStream_t)stream);
}

int dlp_layers_latent_gather(const void* cache, const int32_t* bt_row, int page, int Rc, void* out, int S, void* stream) {
    return latent_gather(cache, bt_row, page, Rc, out, S, (cudaStream_t)stream);
}
int dlp_layers_head_rows(const float* x, int ldx, int D, int Dp, int H, void* out, int T, void* stream) {
    return head_rows(x, ldx, D, Dp, H, out, T, (cudaStream_t)stream);
}
int dlp_layers_rows_attention(const void* q, const void* kv, int ldkv, int S, int T, int pos0, int H, int Dp, int Vp, int V, float scale, const float* gate, int ldg,
                              void* out, int ldo, void* stream) {
    return rows_attention(q, kv, ldkv, S, T, pos0, H, Dp, Vp, V, scale, gate, ldg, out, ldo, (cudaStream_t)stream);
}
int dlp_layers_rows_attention_error(int* flag) { return rows_attention_error(flag); }

}  // extern "C"
