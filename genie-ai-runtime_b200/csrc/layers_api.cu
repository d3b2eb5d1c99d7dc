// layers_api.cu — C entry points of the mechanisms of layer-list models, one each, for use outside the decoder session.
#include "../../include/jllm_b200.h"
#include "attention.cuh"
#include "dense.cuh"

using namespace jb;

static bool kind_ok(int kind) { return kind == EK_BF16 || kind == EK_F32; }
#define NEED_KIND(name) do { if (!kind_ok(kind)) return set_error(JB_ERR_TYPE, name ": element kind %d", kind); if (!ctx()) return JB_ERR_STATE; } while (0)

extern "C" {

int jllm_b200_norm_step(void* h, float* x_out, const float* x, const float* y, const int* tokens, const void* embed, const void* y_exp, const int* slots,
                        const float* weights, int top, const float* post_w, const float* post_b, const float* next_w, const float* next_b,
                        float mult, float eps, int rows, int width, int kind, void* stream) {
    NEED_KIND("norm_step");
    NormStep a;
    a.h = h; a.x_out = x_out; a.x = x; a.y = y; a.tokens = tokens; a.embed = embed; a.y_exp = y_exp; a.slots = slots; a.wts = weights; a.top = top;
    a.post_w = post_w; a.post_b = post_b; a.next_w = next_w; a.next_b = next_b; a.mult = mult; a.eps = eps; a.W = width;
    return launch_norm_rows(a, kind, rows, (cudaStream_t)stream);
}
int jllm_b200_sink_attention(void* out, const void* q, const void* k, const void* v, int kind, int n_heads, int n_kv_heads, int head_dim, int v_dim,
                             int n_tokens, int start, int seq_len, float scale, const float* sink, float q_temp_coef, double q_temp_every, int n_splits,
                             void* stream) {
    NEED_KIND("sink_attention");
    AttnCall c;
    c.out = out; c.q = q; c.k = k; c.v = v; c.kv_kind = kind; c.n_heads = n_heads; c.n_kv = n_kv_heads; c.hd = c.chd = head_dim; c.vhd = v_dim;
    c.ldq = pad8(n_heads * head_dim); c.ldo = pad8(n_heads * v_dim); c.scale = scale; c.sink = sink; c.qt_coef = q_temp_coef; c.qt_every = q_temp_every;
    if (n_tokens > 0) { if (start < 0) return set_error(JB_ERR_ARG, "sink_attention: start=%d", start); c.causal_start = start; c.batch = n_tokens; c.n_splits = 1; }
    else              { if (seq_len <= 0) return set_error(JB_ERR_ARG, "sink_attention: %d keys", seq_len); c.seq_len = seq_len; c.n_splits = n_splits; }
    return launch_attention(c, (cudaStream_t)stream);
}
int jllm_b200_moe_route(int* ids, float* weights, int* rank, int* counts, const float* z, const float* correction, int rows, int n_experts, int top,
                        int n_groups, int keep_groups, void* stream) {
    if (!ctx()) return JB_ERR_STATE;
    MoeRoute r;
    r.n_experts = n_experts; r.top = top; r.n_groups = n_groups; r.keep_groups = keep_groups; r.correction = correction;
    JB_CUDA(cudaMemsetAsync(counts, 0, (size_t)(n_experts > 0 ? n_experts : 0) * sizeof(int), (cudaStream_t)stream));
    return launch_moe_topk(z, r, rows, ids, weights, counts, rank, (cudaStream_t)stream);
}
int jllm_b200_dense_matmul(void* y, const void* W, const void* W_up, const void* x, const int* group_offsets, int n_groups, int kind, int out_f32, int M,
                           int N, int K, float softcap, void* stream) {
    NEED_KIND("dense_matmul");
    DenseGemm g;
    g.kind = kind; g.W = W; g.W_up = W_up; g.swiglu = W_up != nullptr; g.M = M; g.N = N; g.K = K; g.x = x; g.softcap = softcap;
    g.off = group_offsets; g.n_groups = n_groups > 0 ? n_groups : 1;
    g.seg[0] = OutSeg{y, out_f32 ? M : pad8(M), M, out_f32, 0};
    return launch_dense_gemm(g, (cudaStream_t)stream);
}
int jllm_b200_dense_matvec(void* y, const void* W, const void* x, int kind, int out_f32, int M, int K, float softcap, void* stream) {
    NEED_KIND("dense_matvec");
    DenseGemv g;
    g.kind = kind; g.W = W; g.M = M; g.K = K; g.x = x; g.softcap = softcap; g.seg[0] = OutSeg{y, M, M, out_f32, 0};
    return launch_dense_gemv(g, (cudaStream_t)stream);
}
int jllm_b200_moe_matvec(void* y, void* act, int* ids, float* weights, const void* W_gate, const void* W_up, const void* W_down, const void* h,
                         const float* z, const float* correction, int kind, int n_experts, int top, int n_groups, int keep_groups, int ff, int width,
                         void* stream) {
    NEED_KIND("moe_matvec");
    DenseGemv u;
    u.mode = GEMV_MOE_UP; u.kind = kind; u.W = W_gate; u.W_up = W_up; u.M = ff; u.K = width; u.x = h; u.z = z; u.ids = ids; u.wts = weights;
    u.route.n_experts = n_experts; u.route.top = top; u.route.n_groups = n_groups; u.route.keep_groups = keep_groups; u.route.correction = correction;
    u.seg[0] = OutSeg{act, pad8(ff), ff, 0, 0};
    const int rc = launch_dense_gemv(u, (cudaStream_t)stream);
    if (rc) return rc;
    DenseGemv d;
    d.mode = GEMV_MOE_DOWN; d.kind = kind; d.W = W_down; d.M = width; d.K = ff; d.x = act; d.ids = ids; d.wts = weights; d.route = u.route;
    d.seg[0] = OutSeg{y, width, width, 1, 0};
    return launch_dense_gemv(d, (cudaStream_t)stream);
}

}  // extern "C"
