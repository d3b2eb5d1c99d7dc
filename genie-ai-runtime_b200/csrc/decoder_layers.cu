// decoder_layers.cu — models described layer by layer (jllm_b200_layered_desc) behind the decoder session.
//
// One decode step is six launches per layer, each product taking the work around it along:
//   [residual step + norm1 + Q/K/V product, K / V rows straight into the cache]  ->  attention  ->  W_o
//   [residual step + norm2 + router product]  ->  [routing + gate / up + SwiGLU of the chosen experts]  ->  [W_down, weighted sum]
// and the residual step of the last sublayer rides in the logits product.  A prompt chunk runs the same steps over all its
// tokens: residual step (layernorm.cu), tensor-core products (dense_tc.cu; fp32: dense_simt.cu), query-tiled attention, and
// experts over expert-major copies of the tokens (moe.cu).
#include "../../include/jllm_b200_api.hpp"
#include "decoder.cuh"
#include "attention.cuh"
#include "dense.cuh"
#include <new>
#include <vector>

using namespace jb;

namespace {

// Activations of `rows` tokens; x ping-pongs between two buffers because the product that applies the residual step reads
// the old row in every CTA while one of them stores the new one.
struct Acts {
    void* slab = nullptr;
    float *x[2] = {nullptr, nullptr}, *y = nullptr, *z = nullptr, *wts = nullptr;
    void *h = nullptr, *q = nullptr, *att = nullptr, *hp = nullptr, *a = nullptr, *ye = nullptr;
    int *ids = nullptr, *rank = nullptr, *slots = nullptr, *counts = nullptr, *off = nullptr, *rows = nullptr;
};

struct LayerDecoder : jllm_b200_decoder {
    jllm_b200_layered_desc m;
    std::vector<jllm_b200_layer_spec> layers;
    std::vector<int> source;                    // layer whose cache rows a layer reads
    jllm::LayeredKVCache kv;
    int kind = EK_BF16;
    int max_q = 0, max_v = 0, max_e = 0, max_top = 0, max_ff = 0, max_heads = 0;
    Acts one, many;                             // decode step, prompt chunk
    int last_x = 0;                             // which x buffer the chunk's residual ended in
    NormStep pending;                           // the last sublayer's exit of the chunk, still to be applied

    ~LayerDecoder() override { if (one.slab) cudaFree(one.slab); if (many.slab) cudaFree(many.slab); kv.destroy(); }
    int alloc_acts(Acts& a, size_t rows, bool chunk);
    NormStep entry(const Acts& a, const float* w, const float* b) const;
    MoeRoute route(const jllm_b200_layer_spec& w) const;
    AttnCall attention_call(int l, const Acts& a) const;
    int enqueue_step(int n_splits, cudaStream_t st) override;
    int reserve_chunk(int tokens) override;
    int enqueue_chunk(const int* dev_tokens, int n, int start, cudaStream_t st) override;
    int enqueue_rows(const int* host_rows, int n, float* out, cudaStream_t st) override;
    int attn_splits(int seq_len) const override {
        if (kind == EK_F32) return attn_splits_for(seq_len);
        int s = 1;
        for (const auto& w : layers) { const int n = attn_bf16_splits(seq_len, w.n_heads, w.n_kv_heads); s = n > s ? n : s; }
        return s;
    }
    void clear_cache() override {}              // rows beyond the position are never read
    const void* buffer(int which) override { return which == 0 ? one.x[0] : which == 7 ? kv.key_ptr(0, 0) : nullptr; }
};

int LayerDecoder::alloc_acts(Acts& a, size_t R, bool chunk) {
    const size_t es = elem_bytes(kind), W = pad8(m.width), T = max_top;
    auto al = [](size_t b) { return (b + 255) & ~(size_t)255; };
    for (int pass = 0; pass < 2; ++pass) {
        size_t at = 0;
        auto take = [&](size_t b) { void* r = (char*)a.slab + at; at += al(b); return r; };
        float* x0 = (float*)take(R * W * 4); float* x1 = (float*)take(R * W * 4); float* y = (float*)take(R * W * 4);
        void* h = take(R * W * es); void* q = take(R * pad8(max_q) * es); void* att = take(R * pad8(max_v) * es);
        float* z = (float*)take(R * max_e * 4); float* wts = (float*)take(R * T * 4);
        int* ids = (int*)take(R * T * 4); void* ga = take(R * T * pad8(max_ff) * es);
        int *rank = nullptr, *slots = nullptr, *counts = nullptr, *off = nullptr, *rows = nullptr; void *hp = nullptr, *ye = nullptr;
        if (chunk) {
            rank = (int*)take(R * T * 4); slots = (int*)take(R * T * 4); counts = (int*)take((size_t)(max_e + 1) * 4); off = (int*)take((size_t)(max_e + 1) * 4);
            rows = (int*)take(R * 4); hp = take(R * T * W * es); ye = take(R * T * W * es);
        }
        if (pass == 0) {
            if (cudaMalloc(&a.slab, at) != cudaSuccess) { cudaGetLastError(); a.slab = nullptr; return set_error(JB_ERR_NOMEM, "decoder: %zu B of activations", at); }
            JB_CUDA(cudaMemset(a.slab, 0, at));           // the padding of every row stays zero
            continue;
        }
        a.x[0] = x0; a.x[1] = x1; a.y = y; a.h = h; a.q = q; a.att = att; a.z = z; a.wts = wts; a.ids = ids; a.a = ga;
        a.rank = rank; a.slots = slots; a.counts = counts; a.off = off; a.rows = rows; a.hp = hp; a.ye = ye;
    }
    return JB_OK;
}

NormStep LayerDecoder::entry(const Acts& a, const float* w, const float* b) const {
    NormStep n;
    n.W = m.width; n.eps = m.eps; n.mult = m.residual_mult; n.next_w = w; n.next_b = b; n.h = a.h;
    return n;
}
MoeRoute LayerDecoder::route(const jllm_b200_layer_spec& w) const {
    MoeRoute r;
    r.n_experts = w.n_experts; r.top = w.top; r.n_groups = w.n_groups > 0 ? w.n_groups : 1; r.keep_groups = w.n_groups > 1 ? w.keep_groups : 1; r.correction = w.correction;
    return r;
}
AttnCall LayerDecoder::attention_call(int l, const Acts& a) const {
    const jllm_b200_layer_spec& w = layers[l];
    AttnCall c;
    c.out = a.att; c.q = a.q; c.k = kv.key_ptr(source[l], 0); c.v = kv.val_ptr(source[l], 0); c.kv_kind = kind;
    c.n_heads = w.n_heads; c.n_kv = w.n_kv_heads; c.hd = c.chd = w.head_dim; c.vhd = w.v_dim; c.ldq = pad8(w.n_heads * w.head_dim); c.ldo = pad8(w.n_heads * w.v_dim);
    c.scale = w.scale; c.sink = w.sink; c.qt_coef = w.q_temp_coef; c.qt_every = w.q_temp_every; c.max_seq = m.max_context;
    return c;
}
// output places of the Q/K/V product: q rows to the activations, k and v rows to the cache at row 0 of `pos`
template <class Args>
void qkv_segments(Args& g, const jllm_b200_layer_spec& w, void* q, void* k, void* v, int at_pos) {
    const int Q = w.n_heads * w.head_dim, K = w.n_kv_heads * w.head_dim, V = w.n_kv_heads * w.v_dim;
    g.seg[0] = OutSeg{q, pad8(Q), Q, 0, 0};
    g.nseg = 1; g.M = Q;
    if (w.kv_from < 0) {
        g.seg[1] = OutSeg{k, K, K, 0, at_pos};
        g.seg[2] = OutSeg{v, V, V, 0, at_pos};
        g.nseg = 3; g.M = Q + K + V;
    }
}

int LayerDecoder::enqueue_step(int n_splits, cudaStream_t st) {
    const long long l0 = jllm_b200_launch_count();
    const Acts& a = one;
    const int* d_pos = state;
    int cur = 0;                                  // x[cur]: residual before the pending exit
    const float *post_w = nullptr, *post_b = nullptr;
    auto norm = [&](const float* w, const float* b) {
        NormStep n = entry(a, w, b);
        if (!post_w) { n.tokens = state + 1; n.embed = m.embed; n.x_out = a.x[cur]; }
        else { n.x = a.x[cur]; n.y = a.y; n.post_w = post_w; n.post_b = post_b; n.x_out = a.x[cur ^ 1]; cur ^= 1; }
        return n;
    };
    for (int l = 0; l < m.n_layers; ++l) {
        const jllm_b200_layer_spec& w = layers[l];
        DenseGemv g;
        g.mode = GEMV_NORM; g.kind = kind; g.W = w.w_qkv; g.K = m.width; g.d_pos = d_pos;
        g.norm = norm(w.norm1_w, w.norm1_b); g.norm.h = nullptr;
        qkv_segments(g, w, a.q, kv.key_ptr(l, 0), kv.val_ptr(l, 0), 1);
        DCHK(launch_dense_gemv(g, st));
        AttnCall c = attention_call(l, a);
        c.d_pos = d_pos; c.n_splits = n_splits;
        DCHK(launch_attention_float(c, st));
        DenseGemv o;
        o.kind = kind; o.W = w.w_o; o.M = m.width; o.K = w.n_heads * w.v_dim; o.x = a.att; o.seg[0] = OutSeg{a.y, pad8(m.width), m.width, 1, 0};
        DCHK(launch_dense_gemv(o, st));
        post_w = w.norm1b_w; post_b = w.norm1b_b;
        if (w.n_experts <= 0) continue;
        DenseGemv r;
        r.mode = GEMV_NORM; r.kind = kind; r.W = w.w_router; r.M = w.n_experts; r.K = m.width; r.norm = norm(w.norm2_w, w.norm2_b);
        r.seg[0] = OutSeg{a.z, w.n_experts, w.n_experts, 1, 0};
        DCHK(launch_dense_gemv(r, st));
        DenseGemv u;
        u.mode = GEMV_MOE_UP; u.kind = kind; u.W = w.w_gate; u.W_up = w.w_up; u.M = w.expert_dim; u.K = m.width; u.x = a.h; u.route = route(w); u.z = a.z;
        u.ids = a.ids; u.wts = a.wts; u.seg[0] = OutSeg{a.a, pad8(w.expert_dim), w.expert_dim, 0, 0};
        DCHK(launch_dense_gemv(u, st));
        DenseGemv d;
        d.mode = GEMV_MOE_DOWN; d.kind = kind; d.W = w.w_down; d.M = m.width; d.K = w.expert_dim; d.x = a.a; d.route = route(w); d.ids = a.ids; d.wts = a.wts;
        d.seg[0] = OutSeg{a.y, pad8(m.width), m.width, 1, 0};
        DCHK(launch_dense_gemv(d, st));
        post_w = w.norm2b_w; post_b = w.norm2b_b;
    }
    DenseGemv f;
    f.mode = GEMV_NORM; f.kind = kind; f.W = m.embed; f.M = m.vocab_size; f.K = m.width; f.norm = norm(m.final_w, m.final_b); f.norm.h = nullptr;
    f.softcap = m.logit_softcap; f.seg[0] = OutSeg{logits, m.vocab_size, m.vocab_size, 1, 0};
    DCHK(launch_dense_gemv(f, st));
    DCHK(launch_argmax_advance(this, st));
    kernels_per_step = (int)(jllm_b200_launch_count() - l0);
    return JB_OK;
}

int LayerDecoder::reserve_chunk(int tokens) {
    if (tokens <= pf_cap) return JB_OK;
    if (many.slab) { JB_CUDA(cudaDeviceSynchronize()); cudaFree(many.slab); many = Acts(); pf_cap = 0; }
    DCHK(alloc_acts(many, tokens, true));
    pf_cap = tokens;
    return JB_OK;
}

int LayerDecoder::enqueue_chunk(const int* dev_tokens, int N, int start, cudaStream_t st) {
    const Acts& a = many;
    int cur = 0;
    NormStep exit;                                // exit of the sublayer before: y (or expert outputs) and its norm
    bool first = true;
    auto norm = [&](const float* w, const float* b) {
        NormStep n = exit;
        const NormStep e = entry(a, w, b);
        n.W = e.W; n.eps = e.eps; n.mult = e.mult; n.next_w = w; n.next_b = b; n.h = a.h;
        if (first) { n = e; n.tokens = dev_tokens; n.embed = m.embed; n.x_out = a.x[cur]; first = false; }
        else { n.x = a.x[cur]; n.x_out = a.x[cur ^ 1]; cur ^= 1; }
        return n;
    };
    for (int l = 0; l < m.n_layers; ++l) {
        const jllm_b200_layer_spec& w = layers[l];
        DCHK(launch_norm_rows(norm(w.norm1_w, w.norm1_b), kind, N, st));
        DenseGemm g;
        g.kind = kind; g.W = w.w_qkv; g.K = m.width; g.N = N; g.x = a.h;
        qkv_segments(g, w, a.q, kv.key_ptr(l, start), kv.val_ptr(l, start), 0);
        DCHK(launch_dense_gemm(g, st));
        AttnCall c = attention_call(l, a);
        c.causal_start = start; c.batch = N; c.n_splits = 1;
        DCHK(launch_attention_float(c, st));
        DenseGemm o;
        o.kind = kind; o.W = w.w_o; o.M = m.width; o.K = w.n_heads * w.v_dim; o.N = N; o.x = a.att; o.seg[0] = OutSeg{a.y, pad8(m.width), m.width, 1, 0};
        DCHK(launch_dense_gemm(o, st));
        exit = NormStep(); exit.y = a.y; exit.post_w = w.norm1b_w; exit.post_b = w.norm1b_b;
        if (w.n_experts <= 0) continue;
        DCHK(launch_norm_rows(norm(w.norm2_w, w.norm2_b), kind, N, st));
        const MoeRoute r = route(w);
        JB_CUDA(cudaMemsetAsync(a.counts, 0, (size_t)w.n_experts * sizeof(int), st));
        DenseGemm z;
        z.kind = kind; z.W = w.w_router; z.M = w.n_experts; z.K = m.width; z.N = N; z.x = a.h; z.seg[0] = OutSeg{a.z, w.n_experts, w.n_experts, 1, 0};
        DCHK(launch_dense_gemm(z, st));
        DCHK(launch_moe_topk(a.z, r, N, a.ids, a.wts, a.counts, a.rank, st));
        DCHK(launch_moe_permute(a.h, a.hp, kind, m.width, r, N, a.ids, a.rank, a.counts, a.slots, a.off, st));
        DenseGemm u;
        u.kind = kind; u.W = w.w_gate; u.W_up = w.w_up; u.swiglu = 1; u.M = w.expert_dim; u.K = m.width; u.N = N * w.top; u.x = a.hp; u.off = a.off; u.n_groups = w.n_experts;
        u.seg[0] = OutSeg{a.a, pad8(w.expert_dim), w.expert_dim, 0, 0};
        DCHK(launch_dense_gemm(u, st));
        DenseGemm d;
        d.kind = kind; d.W = w.w_down; d.M = m.width; d.K = w.expert_dim; d.N = N * w.top; d.x = a.a; d.off = a.off; d.n_groups = w.n_experts;
        d.seg[0] = OutSeg{a.ye, pad8(m.width), m.width, 0, 0};
        DCHK(launch_dense_gemm(d, st));
        exit = NormStep(); exit.y_exp = a.ye; exit.slots = a.slots; exit.wts = a.wts; exit.top = w.top; exit.post_w = w.norm2b_w; exit.post_b = w.norm2b_b;
    }
    pending = exit; last_x = cur;
    return JB_OK;
}

int LayerDecoder::enqueue_rows(const int* rows, int n, float* out, cudaStream_t st) {
    const Acts& a = many;
    JB_CUDA(cudaMemcpyAsync(a.rows, rows, (size_t)n * sizeof(int), cudaMemcpyHostToDevice, st));
    NormStep f = pending;
    f.W = m.width; f.eps = m.eps; f.mult = m.residual_mult; f.next_w = m.final_w; f.next_b = m.final_b; f.h = a.h; f.x = a.x[last_x]; f.row_index = a.rows;
    DCHK(launch_norm_rows(f, kind, n, st));
    DenseGemm g;
    g.kind = kind; g.W = m.embed; g.M = m.vocab_size; g.K = m.width; g.N = n; g.x = a.h; g.softcap = m.logit_softcap;
    g.seg[0] = OutSeg{out, m.vocab_size, m.vocab_size, 1, 0};
    return launch_dense_gemm(g, st);
}

int check_layer(const jllm_b200_layered_desc& m, int l) {
    const jllm_b200_layer_spec& w = m.layers[l];
    if (w.n_heads <= 0 || w.n_kv_heads <= 0 || w.n_heads % w.n_kv_heads || w.head_dim <= 0 || w.head_dim > 512 || w.v_dim <= 0 || w.v_dim > 512)
        return set_error(JB_ERR_ARG, "decoder: layer %d has %d query and %d KV heads of %d / %d", l, w.n_heads, w.n_kv_heads, w.head_dim, w.v_dim);
    if (w.kv_from >= 0) {
        if (w.kv_from >= l) return set_error(JB_ERR_ARG, "decoder: layer %d takes its keys from layer %d", l, w.kv_from);
        const jllm_b200_layer_spec& s = m.layers[w.kv_from];
        if (s.kv_from >= 0 || s.n_kv_heads != w.n_kv_heads || s.head_dim != w.head_dim || s.v_dim != w.v_dim)
            return set_error(JB_ERR_ARG, "decoder: layer %d cannot use the keys of layer %d", l, w.kv_from);
    }
    if (!w.w_qkv || !w.w_o || !w.norm1_w || !w.norm1_b || !w.norm1b_w || !w.norm1b_b) return set_error(JB_ERR_PTR, "decoder: layer %d lacks a mixer tensor", l);
    if (w.n_experts > 0) {
        const int groups = w.n_groups > 1 ? w.n_groups : 1, keep = groups > 1 ? w.keep_groups : 1;
        if (w.n_experts > MOE_MAX_EXPERTS || w.n_experts % groups || keep < 1 || keep > groups || w.top < 1 || w.top > MOE_MAX_TOP || w.top > keep * (w.n_experts / groups) || w.expert_dim <= 0)
            return set_error(JB_ERR_LIMIT, "decoder: layer %d routes to %d of %d experts (%d of %d groups)", l, w.top, w.n_experts, keep, groups);
        if (!w.w_router || !w.w_gate || !w.w_up || !w.w_down || !w.norm2_w || !w.norm2_b || !w.norm2b_w || !w.norm2b_b)
            return set_error(JB_ERR_PTR, "decoder: layer %d lacks an expert tensor", l);
    }
    return JB_OK;
}

}  // namespace

extern "C" jllm_b200_decoder* jllm_b200_decoder_create_layered(const jllm_b200_layered_desc* model, int flags) {
    if (!model || !model->layers || model->n_layers <= 0 || model->width <= 0 || model->vocab_size <= 0 || model->max_context <= 0) { set_error(JB_ERR_ARG, "decoder: empty model description"); return nullptr; }
    if (model->dtype != EK_BF16 && model->dtype != EK_F32) { set_error(JB_ERR_TYPE, "decoder: element kind %d", model->dtype); return nullptr; }
    if (!model->embed || !model->final_w || !model->final_b) { set_error(JB_ERR_PTR, "decoder: null embedding or final norm"); return nullptr; }
    for (int l = 0; l < model->n_layers; ++l) if (check_layer(*model, l)) return nullptr;
    if (!ctx()) return nullptr;
    LayerDecoder* d = new (std::nothrow) LayerDecoder();
    if (!d) return nullptr;
    d->m = *model;
    d->layers.assign(model->layers, model->layers + model->n_layers);
    d->m.layers = d->layers.data();
    d->kind = model->dtype;
    d->use_graph = (flags & 2) != 0; d->batched_prefill = (flags & 16) != 0;
    std::vector<int> kw, vw;
    auto grow = [](int& a, int b) { if (b > a) a = b; };
    d->max_e = d->max_top = d->max_ff = 1;
    for (int l = 0; l < model->n_layers; ++l) {
        const jllm_b200_layer_spec& w = d->layers[l];
        d->source.push_back(w.kv_from >= 0 ? w.kv_from : l);
        kw.push_back(w.n_kv_heads * w.head_dim); vw.push_back(w.n_kv_heads * w.v_dim);
        grow(d->max_q, w.n_heads * w.head_dim); grow(d->max_v, w.n_heads * w.v_dim); grow(d->max_heads, w.n_heads);
        if (w.n_experts > 0) { grow(d->max_e, w.n_experts); grow(d->max_top, w.top); grow(d->max_ff, w.expert_dim); }
    }
    d->vocab = d->vocab_full = model->vocab_size; d->max_context = model->max_context;
    if (!d->kv.init(model->n_layers, kw.data(), vw.data(), d->source.data(), model->max_context, elem_bytes(d->kind))) {
        set_error(JB_ERR_NOMEM, "decoder: KV cache of %d positions", model->max_context); jllm_b200_decoder_destroy(d); return nullptr;
    }
    // scratch that must exist before any graph capture
    int vmax = 0;
    for (const auto& w : d->layers) grow(vmax, w.v_dim);
    if (d->session_alloc() || d->alloc_acts(d->one, 1, false) || !splitk_buffer((size_t)d->max_heads * 64 * (vmax + 2), true)) { jllm_b200_decoder_destroy(d); return nullptr; }
    return d;
}
