// The part of the C surface every build of the library has: error plumbing, device facts, step bookkeeping, sampling, the dense
// tcgen05 GEMM, the routing plan of expert layers (declarations: include/dlp_b200.h).
#include <stdarg.h>
#include <stdlib.h>
#include <string.h>

#include "../include/dlp_b200.h"
#include "kernels.cuh"
#include <mutex>
#include <set>
#include <utility>

namespace dlp {

static thread_local char g_err[512] = "";

void set_error(const char* fmt, ...) {
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_err, sizeof(g_err), fmt, ap);
    va_end(ap);
}
const char* get_error() { return g_err; }

static int g_pdl = -1;
bool pdl_enabled() {
    if (g_pdl < 0) {
        const char* e = getenv("DLP_PDL");
        g_pdl = (e && e[0] == '0') ? 0 : 1;
    }
    return g_pdl != 0;
}
void set_pdl(bool on) { g_pdl = on ? 1 : 0; }
bool first_use_on_device(const void* kernel) {
    static std::mutex mu;
    static std::set<std::pair<int, const void*>> seen;
    int dev = 0;
    cudaGetDevice(&dev);
    std::lock_guard<std::mutex> lock(mu);
    return seen.insert({dev, kernel}).second;
}
static unsigned long long* g_trace = nullptr;
unsigned long long* trace_buffer() { return g_trace; }
void set_trace_buffer(unsigned long long* buf) { g_trace = buf; }

int sm_count() {
    static int cached[64] = {0};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 148;
    if (cached[dev] == 0) {
        int n = 0;
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) n = 148;
        cached[dev] = n;
    }
    return cached[dev];
}

}  // namespace dlp

using namespace dlp;

extern "C" {

const char* dlp_last_error(void) { return get_error(); }
int dlp_version(void) { return 100; }
int dlp_sm_count(void) { return sm_count(); }
int dlp_set_pdl(int on) { set_pdl(on != 0); return 0; }
int dlp_set_trace(void* buf) { set_trace_buffer((unsigned long long*)buf); return 0; }

int dlp_gemm_f16(const void* w0, const void* w1, int ldw, const void* x, int ldx, void* y, int ldy, int T, int N,
                 int K, int epilogue, int is_bf16, int split_k, void* stream) {
    DLP_REQUIRE(w0 && x && y, "dlp_gemm_f16: null argument");
    return gemm_f16(w0, w1, ldw, x, ldx, y, ldy, T, N, K, epilogue, is_bf16, split_k, (cudaStream_t)stream);
}

int dlp_advance(int32_t* seq_len, const int32_t* active, int32_t* pos, int32_t* slot, int32_t* kv_len,
                const int32_t* block_table, int max_pages, int page_size, int n, void* stream) {
    DLP_REQUIRE(seq_len && pos && slot && block_table && n > 0, "dlp_advance: bad argument");
    return advance(seq_len, active, pos, slot, kv_len, block_table, max_pages, page_size, n, (cudaStream_t)stream);
}

int dlp_argmax(const float* logits, int R, int V, int ld, int32_t* out, void* stream) {
    DLP_REQUIRE(logits && out, "dlp_argmax: null argument");
    return argmax(logits, R, V, ld, out, (cudaStream_t)stream);
}
int dlp_sample(const float* logits, int R, int V, int ld, int top_k, float top_p, float min_p, float temp,
               uint32_t seed, const int32_t* step_ctr, int32_t* out, void* stream) {
    DLP_REQUIRE(logits && out, "dlp_sample: null argument");
    return sample(logits, R, V, ld, top_k, top_p, min_p, temp, seed, step_ctr, out, (cudaStream_t)stream);
}
int dlp_sample_dev(const float* logits, int R, int V, int ld, dlp_sample_params* params, const int32_t* row_slot, int32_t* out,
                   void* stream) {
    DLP_REQUIRE(logits && out && params, "dlp_sample_dev: null argument");
    static_assert(sizeof(dlp_sample_params) == sizeof(SampleParams), "sampler record layout");
    return sample_dev(logits, R, V, ld, reinterpret_cast<SampleParams*>(params), row_slot, out, (cudaStream_t)stream);
}
int dlp_moe_plan(const int32_t* ids, int n_assign, int n_expert, int token_tile, dlp_moe_plan_bufs* b, void* stream) {
    DLP_REQUIRE(ids && b && b->pos && b->src && b->bounds && b->tile_expert && b->tile_row0 && b->tile_rows && b->n_tiles, "dlp_moe_plan: null argument");
    return moe_plan(ids, n_assign, n_expert, token_tile, b->pos, b->src, b->bounds, b->tile_expert, b->tile_row0, b->tile_rows, b->n_tiles,
                    (cudaStream_t)stream);
}
int dlp_moe_gather(const void* x, int ldx, const int32_t* src, int top_k, int n_assign, int K, void* xs, void* stream) {
    DLP_REQUIRE(x && src && xs && n_assign > 0, "dlp_moe_gather: bad argument");
    return moe_gather((const __half*)x, ldx, src, top_k, n_assign, K, (__half*)xs, (cudaStream_t)stream);
}
}  // extern "C"
