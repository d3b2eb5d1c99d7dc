// core.cu — library state shared by every part: the error channel, the per-device context, the launch counter, the
// programmatic-dependent-launch switch and the registry of mapped weight ranges, with the C functions that expose them.
#include "../../include/jllm_b200.h"
#include "common.cuh"
#include <atomic>
#include <cstdarg>
#include <cstring>
#include <mutex>

namespace jb {

// ── error channel ─────────────────────────────────────────────────────────
static thread_local char g_err[512] = "";
static thread_local int  g_err_code = 0;
int set_error(int code, const char* fmt, ...) {
    va_list ap; va_start(ap, fmt);
    vsnprintf(g_err, sizeof g_err, fmt, ap);
    va_end(ap);
    g_err_code = code;
    return code;
}
int cuda_error(cudaError_t e, const char* what) {
    cudaGetLastError();
    return set_error(JB_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
}

// ── contexts ──────────────────────────────────────────────────────────────
static DeviceCtx g_ctx[16];
static std::mutex g_ctx_mu;
DeviceCtx* ctx() {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess) { cuda_error(cudaGetLastError(), "cudaGetDevice"); return nullptr; }
    if (dev < 0 || dev >= 16) { set_error(JB_ERR_LIMIT, "device ordinal %d out of range", dev); return nullptr; }
    DeviceCtx* c = &g_ctx[dev];
    if (c->device == dev) return c;
    std::lock_guard<std::mutex> lk(g_ctx_mu);
    if (c->device == dev) return c;
    cudaDeviceProp pr;
    if (cudaGetDeviceProperties(&pr, dev) != cudaSuccess) { cuda_error(cudaGetLastError(), "cudaGetDeviceProperties"); return nullptr; }
    if (pr.major != 10) { set_error(JB_ERR_STATE, "device %d is sm_%d%d; this library is built for sm_100a only", dev, pr.major, pr.minor); return nullptr; }
    c->sm_count = pr.multiProcessorCount;
    c->max_smem_optin = (int)pr.sharedMemPerBlockOptin;
    // two CTAs per SM: half the SM's shared memory each, minus the per-CTA system reservation and 2 KB of static arrays
    c->gemv_smem_budget = (int)(pr.sharedMemPerMultiprocessor / 2 - pr.reservedSharedMemPerBlock) - 2048;
    c->gemv_smem_budget &= ~127;
    if (cudaMalloc(&c->d_status, 256) != cudaSuccess) { cuda_error(cudaGetLastError(), "cudaMalloc(status)"); return nullptr; }
    cudaMemset(c->d_status, 0, 256);
    if (cudaMalloc(&c->attn_tickets, ATTN_TICKET_WORDS * sizeof(unsigned int)) != cudaSuccess) { cuda_error(cudaGetLastError(), "cudaMalloc(tickets)"); return nullptr; }
    cudaMemset(c->attn_tickets, 0, ATTN_TICKET_WORDS * sizeof(unsigned int));
    c->device = dev;
    return c;
}

static std::atomic<long long> g_launches{0};
static std::atomic<int> g_pdl{1};
void count_launch(int n) { g_launches += n; }
bool pdl_enabled() { return g_pdl.load() != 0; }

// ── weight pointer resolution (gemv_q4.cu:105-128, model.cpp:39-66) ─────────
struct MappedRegion { const char* host; const char* dev; int64_t bytes; };
static MappedRegion g_region = { nullptr, nullptr, 0 };
static const void* g_ok_cache[64];

const void* resolve_weight(const void* W) {
    if (!W) return nullptr;
    if (g_region.host && g_region.dev) {
        const char* p = (const char*)W;
        if (p >= g_region.host && p < g_region.host + g_region.bytes) return g_region.dev + (p - g_region.host);
    }
    const size_t slot = ((uintptr_t)W >> 8) & 63;
    if (g_ok_cache[slot] == W) return W;
    cudaPointerAttributes at{};
    if (cudaPointerGetAttributes(&at, W) != cudaSuccess) { cudaGetLastError(); return nullptr; }
    if (at.type == cudaMemoryTypeDevice || at.type == cudaMemoryTypeManaged) { g_ok_cache[slot] = W; return W; }
    return nullptr;
}

}  // namespace jb

using namespace jb;

extern "C" {

int jllm_b200_init(int device) {
    if (device >= 0) JB_CUDA(cudaSetDevice(device));
    return ctx() ? JB_OK : g_err_code;
}
const char* jllm_b200_last_error(void) { return g_err; }
int  jllm_b200_last_error_code(void) { return g_err_code; }
void jllm_b200_clear_error(void) { g_err[0] = 0; g_err_code = 0; }
int jllm_b200_device_status(void* stream) {
    DeviceCtx* c = ctx();
    if (!c) return g_err_code;
    int h = 0;
    JB_CUDA(cudaMemcpyAsync(&h, c->d_status, sizeof(int), cudaMemcpyDeviceToHost, (cudaStream_t)stream));
    JB_CUDA(cudaStreamSynchronize((cudaStream_t)stream));
    if (h) { cudaMemsetAsync(c->d_status, 0, sizeof(int), (cudaStream_t)stream); set_error(h, "a bounded device-side wait ran out"); }
    return h;
}
long long jllm_b200_launch_count(void) { return g_launches.load(); }
void jllm_b200_set_pdl(int on) { g_pdl.store(on ? 1 : 0); }

const void* jllm_b200_resolve_mapped_weight_device_ptr(const void* p) {
    if (!p || !g_region.host || !g_region.dev) return nullptr;
    const char* c = (const char*)p;
    return (c >= g_region.host && c < g_region.host + g_region.bytes) ? g_region.dev + (c - g_region.host) : nullptr;
}
void jllm_b200_register_mapped_weight_region(const void* hb, const void* db, int64_t bytes) { g_region = { (const char*)hb, (const char*)db, bytes }; }
void jllm_b200_clear_mapped_weight_region(const void* hb) { if (g_region.host == hb) g_region = { nullptr, nullptr, 0 }; }

}  // extern "C"
