// C surface of the layer-list kernels (declarations: include/dlp_b200.h).
#include <string.h>

#include "../include/dlp_b200.h"
#include "kernels.cuh"
#include "layers.cuh"

using namespace dlp;

static_assert(sizeof(dlp_row_stage) == sizeof(RowStage) && sizeof(dlp_hgrn2_args) == sizeof(Hgrn2Args) && sizeof(dlp_scan_chunks) == sizeof(ScanChunks) && sizeof(dlp_latent_args) == sizeof(LatentArgs) &&
              sizeof(dlp_expert_args) == sizeof(ExpertArgs) && sizeof(dlp_route_rule) == sizeof(RouteRule) && sizeof(dlp_ssd_args) == sizeof(SsdArgs) &&
              sizeof(dlp_conv_args) == sizeof(ConvArgs) && sizeof(dlp_gqa_args) == sizeof(GqaArgs) && sizeof(dlp_out_tail) == sizeof(OutTail) &&
              sizeof(dlp_latent_rows) == sizeof(LatentRows) && sizeof(dlp_delta_args) == sizeof(DeltaArgs) && sizeof(dlp_delta_chunks) == sizeof(DeltaChunks), "argument layout");

extern "C" {

int dlp_layers_matvec(const dlp_row_stage* st, const void* w, int ldw, int N, void* out, int ldo, int out_mode, const dlp_out_tail* tail, int T, int f32, void* stream) {
    DLP_REQUIRE(st, "dlp_layers_matvec: null argument");
    return matvec(*reinterpret_cast<const RowStage*>(st), w, ldw, N, out, ldo, out_mode, T, f32, (cudaStream_t)stream, reinterpret_cast<const OutTail*>(tail));
}
int dlp_layers_stage_rows(const dlp_row_stage* st, void* xb, int ldxb, int T, int f32, void* stream) {
    DLP_REQUIRE(st, "dlp_layers_stage_rows: null argument");
    return stage_rows(*reinterpret_cast<const RowStage*>(st), xb, ldxb, T, f32, (cudaStream_t)stream);
}
int dlp_layers_linear(const void* x, int ldx, const void* w, int ldw, int N, int K, void* out, int ldo, int out_mode, const dlp_out_tail* tail, int T, int f32, void* ws, size_t ws_bytes,
                      void* stream) {
    const OutTail* tl = reinterpret_cast<const OutTail*>(tail);
    DLP_REQUIRE(x && w && out && N > 0 && T > 0, "dlp_layers_linear: bad argument");
    if (f32) return sgemm((const float*)x, ldx, (const float*)w, ldw, N, K, out, ldo, out_mode, T, (cudaStream_t)stream, nullptr, tl);
    DLP_REQUIRE(!tl || (out_mode == LO_F32 && tl->n2 >= 0 && (tl->n2 >= N || (tl->out2 && tl->ldo2 >= N - tl->n2))), "dlp_layers_linear: what follows the sums");
    if (out_mode == LO_GEGLU || out_mode == LO_SWIGLU)       // rows 2i / 2i+1 of the interleaved matrix: two operands with twice the row stride
        return gemm_f16(w, (const uint8_t*)w + (size_t)ldw * 2, 2 * ldw, x, ldx, out, ldo, T, N / 2, K, out_mode == LO_GEGLU ? 6 : 8, 1, 0, (cudaStream_t)stream, nullptr, nullptr, ws, ws_bytes);
    DLP_REQUIRE(out_mode == LO_F32 || out_mode == LO_BF16 || out_mode == LO_RELU2, "dlp_layers_linear: output mode %d", out_mode);
    return gemm_f16(w, nullptr, ldw, x, ldx, out, ldo, T, N, K, tl ? 9 : out_mode == LO_BF16 ? 4 : out_mode == LO_RELU2 ? 7 : 1, 1, 0, (cudaStream_t)stream, nullptr, nullptr, ws, ws_bytes,
                    tl);
}
int dlp_layers_head_matmul(const void* x, int x_f32, int ldx, int x_head, int kx, const void* w, int Kp, int H, int N, int n_rows, void* out, int ldo, int out_head,
                           const float* gate, int ldg, int T, int f32, void* stream) {
    return head_matmul(x, x_f32, ldx, x_head, kx, w, Kp, H, N, n_rows, out, ldo, out_head, gate, ldg, T, f32, (cudaStream_t)stream);
}
int dlp_layers_embed(const void* table, int ld, const int32_t* ids, float* h, int E, int T, int vocab, float scale, int f32, void* stream) {
    return embed_rows(table, ld, ids, h, E, T, vocab, scale, f32, (cudaStream_t)stream);
}
int dlp_layers_latent_write(const dlp_latent_rows* a, int T, int f32, void* stream) {
    DLP_REQUIRE(a, "dlp_layers_latent_write: null argument");
    return latent_write(*reinterpret_cast<const LatentRows*>(a), T, f32, (cudaStream_t)stream);
}
int dlp_layers_delta(const dlp_delta_args* a, const dlp_delta_chunks* chunks, const dlp_conv_args* conv, int mode, void* stream) {
    DLP_REQUIRE(a && mode >= 0 && mode <= 2 && (mode != 1 || chunks), "dlp_layers_delta: bad argument");
    const DeltaArgs& d = *reinterpret_cast<const DeltaArgs*>(a);
    if (mode == 1) return delta_chunked(d, *reinterpret_cast<const DeltaChunks*>(chunks), (cudaStream_t)stream);
    return mode == 2 ? delta_decode(d, reinterpret_cast<const ConvArgs*>(conv), (cudaStream_t)stream) : delta_scan(d, (cudaStream_t)stream);
}
int dlp_layers_hgrn2(const dlp_hgrn2_args* a, const dlp_scan_chunks* chunks, void* stream) {
    DLP_REQUIRE(a, "dlp_layers_hgrn2: null argument");
    if (chunks) return hgrn2_chunked(*reinterpret_cast<const Hgrn2Args*>(a), *reinterpret_cast<const ScanChunks*>(chunks), (cudaStream_t)stream);
    return hgrn2_scan(*reinterpret_cast<const Hgrn2Args*>(a), (cudaStream_t)stream);
}
int dlp_layers_ssd(const dlp_ssd_args* a, const dlp_scan_chunks* chunks, const dlp_conv_args* conv, int mode, void* stream) {
    DLP_REQUIRE(a && mode >= 0 && mode <= 2 && (mode != 1 || chunks), "dlp_layers_ssd: bad argument");
    const SsdArgs& s = *reinterpret_cast<const SsdArgs*>(a);
    if (mode == 1) return ssd_chunked(s, *reinterpret_cast<const ScanChunks*>(chunks), (cudaStream_t)stream);
    return mode == 2 ? ssd_decode(s, reinterpret_cast<const ConvArgs*>(conv), (cudaStream_t)stream) : ssd_scan(s, (cudaStream_t)stream);
}
int dlp_layers_conv_rows(const dlp_conv_args* c, const int32_t* seg, const int32_t* seg_slot, const int32_t* pos, int n_seg, int longest, void* out, int ldo, int f32, void* stream) {
    DLP_REQUIRE(c, "dlp_layers_conv_rows: null argument");
    return conv_rows(*reinterpret_cast<const ConvArgs*>(c), seg, seg_slot, pos, n_seg, longest, out, ldo, f32, (cudaStream_t)stream);
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
int dlp_layers_rows_attention(const void* q, const void* kv, int ldkv, int S, int T, int pos0, int H, int Dp, int Vp, int V, int window, float scale, const float* gate,
                              int ldg, void* out, int ldo, void* stream) {
    return rows_attention(q, kv, ldkv, S, T, pos0, H, Dp, Vp, V, window, scale, gate, ldg, out, ldo, (cudaStream_t)stream);
}
int dlp_layers_route(const float* logits, int ld, const dlp_route_rule* rule, int32_t* ids, float* weights, int T, void* stream) {
    DLP_REQUIRE(rule, "dlp_layers_route: null argument");
    return route(logits, ld, *reinterpret_cast<const RouteRule*>(rule), ids, weights, T, (cudaStream_t)stream);
}
int dlp_layers_expert_matvec(const dlp_row_stage* st, const dlp_expert_args* a, void* out, int ldo, int down, int T, int f32, void* stream) {
    DLP_REQUIRE(st && a, "dlp_layers_expert_matvec: null argument");
    return expert_matvec(*reinterpret_cast<const RowStage*>(st), *reinterpret_cast<const ExpertArgs*>(a), out, ldo, down, T, f32, (cudaStream_t)stream);
}
int dlp_layers_linear_grouped(const void* xs, int ldx, const void* w, int ldw, int rows_per_expert, int K, void* out, int ldo, int out_mode, int n_assign, int n_expert,
                              int token_tile, const dlp_moe_plan_bufs* b, int f32, void* ws, size_t ws_bytes, void* stream) {
    DLP_REQUIRE(xs && w && out && b && b->tile_expert && n_assign > 0 && n_expert > 0 && rows_per_expert > 0 && token_tile > 0, "dlp_layers_linear_grouped: bad argument");
    DLP_REQUIRE(out_mode == LO_F32 || out_mode == LO_RELU2 || (out_mode == LO_SWIGLU && rows_per_expert % 2 == 0), "dlp_layers_linear_grouped: output mode %d", out_mode);
    GemmGroup g;
    g.tile_expert = b->tile_expert; g.tile_row0 = b->tile_row0; g.tile_rows = b->tile_rows; g.n_tiles = b->n_tiles;
    g.rows_per_expert = rows_per_expert; g.n_expert = n_expert; g.bt = token_tile;
    const int most = (n_assign + token_tile - 1) / token_tile + n_expert;      // every expert may end with one partial tile,
    g.max_tiles = most < n_assign ? most : n_assign;                           // and a tile holds at least one row
    if (f32) return sgemm((const float*)xs, ldx, (const float*)w, ldw, rows_per_expert, K, out, ldo, out_mode, n_assign, (cudaStream_t)stream, &g);
    if (out_mode == LO_SWIGLU) {       // two operands with twice the row stride, as in dlp_layers_linear
        g.rows_per_expert = rows_per_expert / 2;
        return gemm_f16(w, (const uint8_t*)w + (size_t)ldw * 2, 2 * ldw, xs, ldx, out, ldo, n_assign, rows_per_expert / 2, K, 8, 1, ws ? 0 : 1, (cudaStream_t)stream, nullptr, &g, ws,
                        ws_bytes);
    }
    return gemm_f16(w, nullptr, ldw, xs, ldx, out, ldo, n_assign, rows_per_expert, K, out_mode == LO_RELU2 ? 7 : 1, 1, ws ? 0 : 1, (cudaStream_t)stream, nullptr, &g, ws,
                    ws_bytes);
}
int dlp_layers_combine(const float* y, int ldy, const int32_t* pos, const float* weights, int T, int top, int E, float* out, const float* ys, const float* gs, int ldgs,
                       void* stream) {
    DLP_REQUIRE(y && pos && weights && out && top > 0 && (!ys || gs), "dlp_layers_combine: bad argument");
    return moe_combine(y, pos, weights, T, top, E, out, (cudaStream_t)stream, ldy, 0, ys, gs, ldgs);
}
int dlp_layers_gqa_prepare(const dlp_gqa_args* a, int f32, void* stream) {
    DLP_REQUIRE(a, "dlp_layers_gqa_prepare: null argument");
    return gqa_prepare(*reinterpret_cast<const GqaArgs*>(a), f32, (cudaStream_t)stream);
}
int dlp_layers_gqa_attention(const dlp_gqa_args* a, int fused, int f32, void* stream) {
    DLP_REQUIRE(a, "dlp_layers_gqa_attention: null argument");
    return gqa_attention(*reinterpret_cast<const GqaArgs*>(a), fused, f32, (cudaStream_t)stream);
}
int dlp_layers_gqa_flash(const dlp_gqa_args* a, void* stream) {
    DLP_REQUIRE(a, "dlp_layers_gqa_flash: null argument");
    return gqa_flash(*reinterpret_cast<const GqaArgs*>(a), (cudaStream_t)stream);
}
int dlp_layers_rows_attention_error(int* flag) { return rows_attention_error(flag); }

}  // extern "C"
