// decoder_kquant.cu — the K-quant Llama / Qwen3 family behind the decoder session: one decode step (single GPU and
// tensor-parallel) and the batched prompt prefill.  Order of operations follows the reference engine:
// Engine::decode_step (src/engine/decode.cu:2101-2194), transformer_layer (:1169-1246),
// transformer_layer_attn_compute (:1437-1497), attn/ffn exits (:1499-1522).
#include "../../include/jllm_b200_api.hpp"
#include "decoder.cuh"
#include "gemv.cuh"
#include "elementwise.cuh"
#include "attention.cuh"
#include "mmq.cuh"
#include "tp.cuh"
#include <cfloat>
#include <cstdlib>
#include <new>
#include <vector>

using namespace jb;

namespace {

struct KquantDecoder : jllm_b200_decoder {
    jllm_b200_model_desc m;
    std::vector<jllm_b200_layer_desc> layers;
    jllm::KVCachePool kv;
    bool fused = true, chain = false;
    __half *x = nullptr, *x2 = nullptr, *normed = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *att = nullptr, *gate = nullptr, *up = nullptr, *sw = nullptr;
    void* slab = nullptr;
    // tensor-parallel session: m keeps the full dimensions, the weights are this rank's row slices
    bool tp_on = false, tp_fused = true;
    TpDev tp;
    int tp_off[6] = {0, 0, 0, 0, 0, 0};
    int nh_l = 0, nkv_l = 0, I_l = 0, H_l = 0, V_l = 0;
    uint32_t* seq = nullptr;
    // batched prompt prefill (flag bit 4): activations of up to pf_cap prompt tokens, allocated on first use
    void* pf_slab = nullptr;
    __half *pf_x = nullptr, *pf_x2 = nullptr, *pf_normed = nullptr, *pf_y = nullptr, *pf_q = nullptr, *pf_att = nullptr, *pf_k = nullptr,
           *pf_v = nullptr, *pf_gate = nullptr, *pf_up = nullptr, *pf_sw = nullptr;

    ~KquantDecoder() override {
        if (slab) cudaFree(slab);
        if (pf_slab) cudaFree(pf_slab);
        if (seq) cudaFree(seq);
        kv.destroy();
    }
    int alloc();
    int enqueue_step(int n_splits, cudaStream_t st) override;
    int reserve_chunk(int tokens) override;
    int enqueue_chunk(const int* dev_tokens, int n, int start, cudaStream_t st) override;
    int enqueue_rows(const int* host_rows, int n, float* out, cudaStream_t st) override;
    int attn_splits(int seq_len) const override { return attn_splits_for(seq_len); }
    bool has_chunks() const override { return !tp_on; }
    void clear_cache() override { kv.clear(); }
    const void* buffer(int which) override {
        switch (which) {
            case 0: return x;   case 1: return x2; case 2: return q;  case 3: return k; case 4: return v;
            case 5: return att; case 6: return sw; case 7: return kv.key_ptr(0, 0); case 8: return kv.kv_scale_ptr(0, 0, false);
            default: return nullptr;
        }
    }
};

int KquantDecoder::alloc() {
    // (a tensor-parallel rank could do with slice-sized buffers; the full sizes are a few hundred KB)
    const size_t H = m.hidden_dim, QD = (size_t)m.n_heads * m.head_dim, KVD = (size_t)m.n_kv_heads * m.head_dim, I = m.intermediate_dim;
    auto al = [](size_t b) { return (b + 255) & ~(size_t)255; };
    const size_t total = 3 * al(H * 2) + 2 * al(QD * 2) + 2 * al(KVD * 2) + 3 * al(I * 2);
    if (cudaMalloc(&slab, total) != cudaSuccess) { cudaGetLastError(); return set_error(JB_ERR_NOMEM, "decoder: %zu B of activations", total); }
    cudaMemset(slab, 0, total);
    char* p = (char*)slab;
    auto take = [&](size_t b) { char* r = p; p += al(b); return r; };
    x = (__half*)take(H * 2); x2 = (__half*)take(H * 2); normed = (__half*)take(H * 2);
    q = (__half*)take(QD * 2); att = (__half*)take(QD * 2);
    k = (__half*)take(KVD * 2); v = (__half*)take(KVD * 2);
    gate = (__half*)take(I * 2); up = (__half*)take(I * 2); sw = (__half*)take(I * 2);
    vocab = vocab_full = m.vocab_size; max_context = m.max_context;
    return session_alloc();
}

// Enqueues one decode step that reads position and token from d->state.  n_splits is fixed per
// enqueue (a captured graph keeps the value it was captured with).
static int dec_enqueue_step_tp(KquantDecoder* d, int n_splits, cudaStream_t st);
static int dec_enqueue_step(KquantDecoder* d, int n_splits, cudaStream_t st) {
    if (d->tp_on) return dec_enqueue_step_tp(d, n_splits, st);
    const jllm_b200_model_desc& m = d->m;
    const int H = m.hidden_dim, QD = m.n_heads * m.head_dim, KVD = m.n_kv_heads * m.head_dim, I = m.intermediate_dim;
    const int* d_pos = d->state; const int* d_tok = d->state + 1;
    const float scale = 1.0f / sqrtf((float)m.head_dim);
    const long long l0 = jllm_b200_launch_count();
    DCHK(launch_embed_row(d->x, m.tok_embd, m.embd_type, 0, d_tok, H, st));
    if (d->fused && d->chain) {
        // Q/K/V of layer 0 alone, then per layer: QKV prep, attention, and ONE chained launch for Wo + residual ->
        // norm + gate/up + SwiGLU -> W_down + residual -> norm + Q/K/V of the next layer
        auto triple_args = [&](int l) {
            const jllm_b200_layer_desc& w = d->layers[l];
            GemvArgs a;
            a.nseg = 3;
            a.seg[0] = GemvSeg{ resolve_weight(w.wq), d->q, QD, w.type_wq };
            a.seg[1] = GemvSeg{ resolve_weight(w.wk), d->k, KVD, w.type_wk };
            a.seg[2] = GemvSeg{ resolve_weight(w.wv), d->v, KVD, w.type_wv };
            a.x = d->x; a.K = H; a.xmode = triple_dp4a(w.type_wq, w.type_wk, w.type_wv) ? 0 : 1; a.out_mode = 0;
            a.do_norm = 1; a.norm_w = w.rms_attn; a.norm_w_fp32 = 1; a.eps = m.rms_eps;
            return a;
        };
        { const GemvArgs a0 = triple_args(0); DCHK(launch_gemv(a0, st)); }
        for (int l = 0; l < m.n_layers; ++l) {
            const jllm_b200_layer_desc& w = d->layers[l];
            int8_t* kc = (int8_t*)d->kv.key_ptr(l, 0); int8_t* vc = (int8_t*)d->kv.val_ptr(l, 0);
            float* ks = d->kv.kv_scale_ptr(l, 0, false); float* vs = d->kv.kv_scale_ptr(l, 0, true);
            DCHK(launch_qkv_prep(d->q, d->k, d->v, w.q_norm, w.k_norm, m.rms_eps, kc, vc, ks, vs, m.n_heads, m.n_kv_heads, m.head_dim,
                                 0, d_pos, m.rope_theta, m.rope_neox != 0, true, st));
            AttnCall c;
            c.out = d->att; c.q = d->q; c.k = kc; c.v = vc; c.ks = ks; c.vs = vs; c.n_heads = m.n_heads; c.n_kv = m.n_kv_heads;
            c.hd = m.head_dim; c.chd = m.head_dim; c.d_pos = d_pos; c.scale = scale; c.kv_int8 = 1; c.n_splits = n_splits; c.max_seq = m.max_context;
            DCHK(launch_attention(c, st));
            GemvArgs ph[4];
            int n = 0;
            ph[n].nseg = 1; ph[n].seg[0] = GemvSeg{ resolve_weight(w.wo), d->x2, H, w.type_wo };
            ph[n].x = d->att; ph[n].K = QD; ph[n].xmode = 1; ph[n].out_mode = 2; ph[n].residual = d->x; ++n;
            ph[n].nseg = 2; ph[n].seg[0] = GemvSeg{ resolve_weight(w.w_gate), d->sw, I, w.type_w_gate };
            ph[n].seg[1] = GemvSeg{ resolve_weight(w.w_up), d->sw, I, w.type_w_up };
            ph[n].x = d->x2; ph[n].K = H; ph[n].xmode = (w.type_w_gate == T_Q4K && w.type_w_up == T_Q4K) ? 0 : 1; ph[n].out_mode = 3;
            ph[n].do_norm = 1; ph[n].norm_w = w.rms_ffn; ph[n].norm_w_fp32 = 1; ph[n].eps = m.rms_eps; ++n;
            ph[n].nseg = 1; ph[n].seg[0] = GemvSeg{ resolve_weight(w.w_down), d->x, H, w.type_w_down };
            ph[n].x = d->sw; ph[n].K = I; ph[n].xmode = 1; ph[n].out_mode = 2; ph[n].residual = d->x2; ++n;
            if (l + 1 < m.n_layers) ph[n++] = triple_args(l + 1);
            DCHK(launch_gemv_chain(ph, n, (unsigned int*)(d->state + 200), st));
        }
    } else
    for (int l = 0; l < m.n_layers; ++l) {
        const jllm_b200_layer_desc& w = d->layers[l];
        int8_t* kc = (int8_t*)d->kv.key_ptr(l, 0); int8_t* vc = (int8_t*)d->kv.val_ptr(l, 0);
        float* ks = d->kv.kv_scale_ptr(l, 0, false); float* vs = d->kv.kv_scale_ptr(l, 0, true);
        if (d->fused) {
            DCHK(jllm_b200_norm_gemv_quant_triple(d->q, w.wq, w.type_wq, QD, d->k, w.wk, w.type_wk, KVD, d->v, w.wv, w.type_wv, KVD,
                                                  d->x, w.rms_attn, 1, m.rms_eps, H, st));
            DCHK(launch_qkv_prep(d->q, d->k, d->v, w.q_norm, w.k_norm, m.rms_eps, kc, vc, ks, vs, m.n_heads, m.n_kv_heads, m.head_dim,
                                 0, d_pos, m.rope_theta, m.rope_neox != 0, true, st));
        } else {
            DCHK(launch_rmsnorm(d->normed, d->x, nullptr, w.rms_attn, true, 1, H, m.rms_eps, st));
            DCHK(jllm_b200_gemv_quant_triple(d->q, w.wq, w.type_wq, QD, d->k, w.wk, w.type_wk, KVD, d->v, w.wv, w.type_wv, KVD, d->normed, H, st));
            if (w.q_norm && w.k_norm) {
                DCHK(launch_rmsnorm(d->q, d->q, nullptr, w.q_norm, true, m.n_heads, m.head_dim, m.rms_eps, st));
                DCHK(launch_rmsnorm(d->k, d->k, nullptr, w.k_norm, true, m.n_kv_heads, m.head_dim, m.rms_eps, st));
            }
            DCHK(launch_rope(d->q, d->k, nullptr, nullptr, nullptr, m.n_heads, m.n_kv_heads, m.head_dim, m.head_dim, 0, d_pos, m.rope_theta,
                             m.rope_neox != 0, 1, 0, 0, 0, false, st));
            // K/V rows of this step: one absmax scale per kv head, written at *d_pos (fp16_to_int8 arithmetic;
            // norms and rotation are already applied, so the prep kernel only quantises)
            DCHK(launch_qkv_prep(d->q, d->k, d->v, nullptr, nullptr, m.rms_eps, kc, vc, ks, vs, 0, m.n_kv_heads, m.head_dim, 0, d_pos,
                                 m.rope_theta, m.rope_neox != 0, false, st));
        }
        AttnCall c;
        c.out = d->att; c.q = d->q; c.k = kc; c.v = vc; c.ks = ks; c.vs = vs; c.n_heads = m.n_heads; c.n_kv = m.n_kv_heads;
        c.hd = m.head_dim; c.chd = m.head_dim; c.d_pos = d_pos; c.scale = scale; c.kv_int8 = 1; c.n_splits = n_splits; c.max_seq = m.max_context;
        DCHK(launch_attention(c, st));
        DCHK(jllm_b200_gemv_quant_add(d->x2, w.wo, w.type_wo, d->att, d->x, H, QD, st));
        if (d->fused) {
            DCHK(jllm_b200_norm_gemv_pair_swiglu(d->sw, w.w_gate, w.w_up, w.type_w_gate, I, d->x2, w.rms_ffn, 1, m.rms_eps, H, st));
        } else {
            DCHK(launch_rmsnorm(d->normed, d->x2, nullptr, w.rms_ffn, true, 1, H, m.rms_eps, st));
            DCHK(jllm_b200_gemv_quant_pair(d->gate, w.w_gate, w.type_w_gate, I, d->up, w.w_up, w.type_w_up, I, d->normed, H, st));
            DCHK(launch_glu(d->sw, d->gate, d->up, 1, I, false, st));
        }
        DCHK(jllm_b200_gemv_quant_add(d->x, w.w_down, w.type_w_down, d->sw, d->x2, H, I, st));
    }
    DCHK(launch_rmsnorm(d->normed, d->x, nullptr, m.output_norm, true, 1, H, m.rms_eps, st));
    DCHK(jllm_b200_gemv_quant_f32(d->logits, m.output, m.output_type, d->normed, m.vocab_size, H, st));
    DCHK(launch_argmax_advance(d, st));
    d->kernels_per_step = (int)(jllm_b200_launch_count() - l0);
    return JB_OK;
}


// One decode step of a tensor-parallel rank: the single-GPU sequence on this rank's rows and heads.  The Wo, gate/up
// and W_down kernels send every finished row as a packet to all ranks from their epilogue, the attention output goes
// out through one small push kernel, and each consuming GEMV polls the packets of its own region while it stages
// its activation vector (after its weight prefetch is under way), so an exchange costs one one-way NVLink trip and,
// but for the attention output, no launch.  Plain fp16 copies of this rank's own slices stay local for the residuals.
static int dec_enqueue_step_tp(KquantDecoder* d, int n_splits, cudaStream_t st) {
    const jllm_b200_model_desc& m = d->m;
    const int H = m.hidden_dim, QD = m.n_heads * m.head_dim, I = m.intermediate_dim, hd = m.head_dim;
    const int QD_l = d->nh_l * hd, KVD_l = d->nkv_l * hd, rank = d->tp.rank, world = d->tp.world;
    unsigned char* mine = d->tp.peer[rank];
    const __half* att_pk = (const __half*)(mine + d->tp_off[0]); const __half* x2_pk = (const __half*)(mine + d->tp_off[1]);
    const __half* sw_pk = (const __half*)(mine + d->tp_off[2]);  const __half* x_pk = (const __half*)(mine + d->tp_off[3]);
    const int* d_pos = d->state; const int* d_tok = d->state + 1;
    const float scale = 1.0f / sqrtf((float)hd);
    const long long l0 = jllm_b200_launch_count();
    auto wait_hook = [&](int layer) { GemvTpWait w; w.seq = d->seq; w.epochs_per_step = m.n_layers; w.layer = layer; return w; };
    auto push_hook = [&](int point, int layer, int rows_local) {
        GemvTpPush q;
        for (int r = 0; r < 8; ++r) q.peer[r] = r < world ? d->tp.peer[r] : nullptr;
        q.world = world; q.buf_off = d->tp_off[point]; q.row_off = rank * rows_local;
        q.seq = d->seq; q.epochs_per_step = m.n_layers; q.layer = layer;
        return q;
    };
    // d->normed holds the plain full x of layer 0 (the embedding row, computed by every rank); d->x / d->x2 hold this
    // rank's own slices of x / x2
    DCHK(launch_embed_row(d->normed, m.tok_embd, m.embd_type, 0, d_tok, H, st));
    for (int l = 0; l < m.n_layers; ++l) {
        const jllm_b200_layer_desc& w = d->layers[l];
        int8_t* kc = (int8_t*)d->kv.key_ptr(l, 0); int8_t* vc = (int8_t*)d->kv.val_ptr(l, 0);
        float* ks = d->kv.kv_scale_ptr(l, 0, false); float* vs = d->kv.kv_scale_ptr(l, 0, true);
        auto triple_args = [&](int ll, const GemvTpWait* wh) {
            const jllm_b200_layer_desc& ww = d->layers[ll];
            GemvArgs a;
            a.nseg = 3;
            a.seg[0] = GemvSeg{ resolve_weight(ww.wq), d->q, QD_l, ww.type_wq };
            a.seg[1] = GemvSeg{ resolve_weight(ww.wk), d->k, KVD_l, ww.type_wk };
            a.seg[2] = GemvSeg{ resolve_weight(ww.wv), d->v, KVD_l, ww.type_wv };
            a.x = ll > 0 ? x_pk : d->normed; a.K = H; a.xmode = triple_dp4a(ww.type_wq, ww.type_wk, ww.type_wv) ? 0 : 1; a.out_mode = 0;
            a.do_norm = 1; a.norm_w = ww.rms_attn; a.norm_w_fp32 = 1; a.eps = m.rms_eps;
            a.tp_wait = ll > 0 ? wh : nullptr;
            return a;
        };
        int rc = 0;
        if (l == 0 || !d->chain) {
            const GemvTpWait wh = wait_hook(l - 1);
            const GemvArgs a0 = triple_args(l, &wh);
            DCHK(launch_gemv(a0, st));
        }
        DCHK(launch_qkv_prep(d->q, d->k, d->v, w.q_norm, w.k_norm, m.rms_eps, kc, vc, ks, vs, d->nh_l, d->nkv_l, hd,
                             0, d_pos, m.rope_theta, m.rope_neox != 0, true, st));
        AttnCall c;
        c.out = d->att; c.q = d->q; c.k = kc; c.v = vc; c.ks = ks; c.vs = vs; c.n_heads = d->nh_l; c.n_kv = d->nkv_l;
        c.hd = hd; c.chd = hd; c.d_pos = d_pos; c.scale = scale; c.kv_int8 = 1; c.n_splits = n_splits; c.max_seq = m.max_context;
        DCHK(launch_attention(c, st));
        DCHK(launch_tp_push(d->tp, d->att, QD_l, d->tp_off[0], rank * QD_l, l, st));
        if (d->chain) {
            // Wo -> gate/up -> W_down -> next layer's Q/K/V in one launch; no grid barrier: every input of a later phase
            // (activation vector and residual rows) is read as packets, which carry their own arrival mark
            const GemvTpWait wh = wait_hook(l);
            const GemvTpPush p_x2 = push_hook(TP_POINT_X2, l, d->H_l), p_sw = push_hook(TP_POINT_SW, l, d->I_l), p_x = push_hook(TP_POINT_X, l, d->H_l);
            GemvArgs ph[4];
            int n = 0;
            ph[n].nseg = 1; ph[n].seg[0] = GemvSeg{ resolve_weight(w.wo), d->x2, d->H_l, w.type_wo };
            ph[n].x = att_pk; ph[n].K = QD; ph[n].xmode = 1; ph[n].out_mode = 2;
            ph[n].residual = l > 0 ? d->x : d->normed + (size_t)rank * d->H_l; ph[n].tp_wait = &wh; ph[n].tp_push = &p_x2; ++n;
            ph[n].nseg = 2; ph[n].seg[0] = GemvSeg{ resolve_weight(w.w_gate), d->sw, d->I_l, w.type_w_gate };
            ph[n].seg[1] = GemvSeg{ resolve_weight(w.w_up), d->sw, d->I_l, w.type_w_up };
            ph[n].x = x2_pk; ph[n].K = H; ph[n].xmode = (w.type_w_gate == T_Q4K && w.type_w_up == T_Q4K) ? 0 : 1; ph[n].out_mode = 3;
            ph[n].do_norm = 1; ph[n].norm_w = w.rms_ffn; ph[n].norm_w_fp32 = 1; ph[n].eps = m.rms_eps; ph[n].tp_wait = &wh; ph[n].tp_push = &p_sw; ++n;
            ph[n].nseg = 1; ph[n].seg[0] = GemvSeg{ resolve_weight(w.w_down), d->x, d->H_l, w.type_w_down };
            ph[n].x = sw_pk; ph[n].K = I; ph[n].xmode = 1; ph[n].out_mode = 2;
            ph[n].residual_pk = reinterpret_cast<const uint2*>(x2_pk) + (size_t)rank * d->H_l; ph[n].tp_wait = &wh; ph[n].tp_push = &p_x; ++n;
            if (l + 1 < m.n_layers) ph[n++] = triple_args(l + 1, &wh);
            DCHK(launch_gemv_chain(ph, n, nullptr, st));
            continue;
        }
        {
            const GemvTpWait wh = wait_hook(l); const GemvTpPush ph = push_hook(TP_POINT_X2, l, d->H_l);
            gemv_set_tp_hooks(&wh, &ph);
            const __half* resid = l > 0 ? d->x : d->normed + (size_t)rank * d->H_l;
            rc = jllm_b200_gemv_quant_add(d->x2, w.wo, w.type_wo, att_pk, resid, d->H_l, QD, st);
            gemv_set_tp_hooks(nullptr, nullptr);
            DCHK(rc);
        }
        {
            const GemvTpWait wh = wait_hook(l); const GemvTpPush ph = push_hook(TP_POINT_SW, l, d->I_l);
            gemv_set_tp_hooks(&wh, &ph);
            rc = jllm_b200_norm_gemv_pair_swiglu(d->sw, w.w_gate, w.w_up, w.type_w_gate, d->I_l, x2_pk, w.rms_ffn, 1, m.rms_eps, H, st);
            gemv_set_tp_hooks(nullptr, nullptr);
            DCHK(rc);
        }
        {
            const GemvTpWait wh = wait_hook(l); const GemvTpPush ph = push_hook(TP_POINT_X, l, d->H_l);
            gemv_set_tp_hooks(&wh, &ph);
            rc = jllm_b200_gemv_quant_add(d->x, w.w_down, w.type_w_down, sw_pk, d->x2, d->H_l, I, st);
            gemv_set_tp_hooks(nullptr, nullptr);
            DCHK(rc);
        }
    }
    DCHK(launch_tp_unpack(d->tp, d->gate, H, d->tp_off[3], m.n_layers - 1, st));          // d->gate: free scratch of at least H halves
    DCHK(launch_rmsnorm(d->normed, d->gate, nullptr, m.output_norm, true, 1, H, m.rms_eps, st));
    DCHK(jllm_b200_gemv_quant_f32(d->logits, m.output, m.output_type, d->normed, d->V_l, H, st));
    DCHK(launch_tp_argmax(d->tp, d->logits, d->V_l, d->state, d->out_tokens, d->out_cap, st));
    d->kernels_per_step = (int)(jllm_b200_launch_count() - l0);
    return JB_OK;
}

// ── batched prompt prefill: the reference's Engine::transformer_prefill (src/engine/decode.cu:1760-1884) for a chunk of
// N >= 2 prompt tokens at positions start .. start+N-1: RMSNorm over rows, batched K-quant products (prefill arithmetic),
// QK-norm + RoPE + INT8 KV store for all tokens in one launch, query-tiled causal attention, Wo, residual, RMSNorm,
// gate/up, SwiGLU, W_down, residual.  After the last chunk: final norm and logits of the last token only, greedy token.
int KquantDecoder::reserve_chunk(int cap) {
    if (cap <= pf_cap) return JB_OK;
    if (pf_slab) { cudaFree(pf_slab); pf_slab = nullptr; pf_cap = 0; }
    const size_t N = (size_t)cap, H = m.hidden_dim, QD = (size_t)m.n_heads * m.head_dim, KVD = (size_t)m.n_kv_heads * m.head_dim, I = m.intermediate_dim;
    auto al = [](size_t b) { return (b + 255) & ~(size_t)255; };
    const size_t total = 4 * al(N * H * 2) + 2 * al(N * QD * 2) + 2 * al(N * KVD * 2) + 3 * al(N * I * 2);
    if (cudaMalloc(&pf_slab, total) != cudaSuccess) { cudaGetLastError(); return set_error(JB_ERR_NOMEM, "decoder: %zu B of prefill activations", total); }
    char* p = (char*)pf_slab;
    auto take = [&](size_t b) { char* r = p; p += al(b); return r; };
    pf_x = (__half*)take(N * H * 2); pf_x2 = (__half*)take(N * H * 2); pf_normed = (__half*)take(N * H * 2); pf_y = (__half*)take(N * H * 2);
    pf_q = (__half*)take(N * QD * 2); pf_att = (__half*)take(N * QD * 2);
    pf_k = (__half*)take(N * KVD * 2); pf_v = (__half*)take(N * KVD * 2);
    pf_gate = (__half*)take(N * I * 2); pf_up = (__half*)take(N * I * 2); pf_sw = (__half*)take(N * I * 2);
    pf_cap = cap;
    return JB_OK;
}

int KquantDecoder::enqueue_chunk(const int* dev_tokens, int N, int start, cudaStream_t st) {
    const int H = m.hidden_dim, QD = m.n_heads * m.head_dim, KVD = m.n_kv_heads * m.head_dim, I = m.intermediate_dim;
    const float scale = 1.0f / sqrtf((float)m.head_dim);
    DCHK(launch_embed_rows(pf_x, m.tok_embd, m.embd_type, dev_tokens, N, H, st));
    for (int l = 0; l < m.n_layers; ++l) {
        const jllm_b200_layer_desc& w = layers[l];
        int8_t* kc = (int8_t*)kv.key_ptr(l, 0); int8_t* vc = (int8_t*)kv.val_ptr(l, 0);
        float* ks = kv.kv_scale_ptr(l, 0, false); float* vs = kv.kv_scale_ptr(l, 0, true);
        DCHK(launch_rmsnorm(pf_normed, pf_x, nullptr, w.rms_attn, true, N, H, m.rms_eps, st));
        DCHK(launch_mmq(pf_q, resolve_weight(w.wq), w.type_wq, pf_normed, QD, N, H, nullptr, st));
        DCHK(launch_mmq_ex(pf_k, resolve_weight(w.wk), w.type_wk, pf_normed, KVD, N, H, nullptr, true, st));      // the operand of the product before
        DCHK(launch_mmq_ex(pf_v, resolve_weight(w.wv), w.type_wv, pf_normed, KVD, N, H, nullptr, true, st));      // the operand of the product before
        DCHK(launch_qkv_prep_tokens(pf_q, pf_k, pf_v, w.q_norm, w.k_norm, m.rms_eps, kc, vc, ks, vs, N, m.n_heads, m.n_kv_heads,
                                    m.head_dim, start, m.rope_theta, m.rope_neox != 0, st));
        AttnCall c;
        c.out = pf_att; c.q = pf_q; c.k = kc; c.v = vc; c.ks = ks; c.vs = vs; c.n_heads = m.n_heads; c.n_kv = m.n_kv_heads;
        c.hd = m.head_dim; c.chd = m.head_dim; c.scale = scale; c.kv_int8 = 1; c.causal_start = start; c.batch = N; c.n_splits = 1;
        DCHK(attention_prefill_fast_applies(c) ? launch_attention_prefill_fast(c, st) : launch_attention_general(c, st));
        DCHK(launch_mmq(pf_y, resolve_weight(w.wo), w.type_wo, pf_att, H, N, QD, nullptr, st));
        DCHK(launch_add_half(pf_x2, pf_x, pf_y, (long long)N * H, st));
        DCHK(launch_rmsnorm(pf_normed, pf_x2, nullptr, w.rms_ffn, true, N, H, m.rms_eps, st));
        DCHK(launch_mmq_pair(pf_gate, pf_up, resolve_weight(w.w_gate), w.type_w_gate, resolve_weight(w.w_up), w.type_w_up, pf_normed, I, I, N, H, st));
        DCHK(launch_glu(pf_sw, pf_gate, pf_up, N, I, false, st));
        DCHK(launch_mmq(pf_y, resolve_weight(w.w_down), w.type_w_down, pf_sw, H, N, I, nullptr, st));
        DCHK(launch_add_half(pf_x, pf_x2, pf_y, (long long)N * H, st));
    }
    return JB_OK;
}
// logits of single rows of the chunk (src/engine/decode.cu:2019-2050 computes them for the last prompt token only)
int KquantDecoder::enqueue_rows(const int* rows, int n, float* out, cudaStream_t st) {
    const int H = m.hidden_dim;
    for (int i = 0; i < n; ++i) {
        DCHK(launch_rmsnorm(normed, pf_x + (size_t)rows[i] * H, nullptr, m.output_norm, true, 1, H, m.rms_eps, st));
        DCHK(jllm_b200_gemv_quant_f32(out + (size_t)i * m.vocab_size, m.output, m.output_type, normed, m.vocab_size, H, st));
    }
    return JB_OK;
}
int KquantDecoder::enqueue_step(int n_splits, cudaStream_t st) { return dec_enqueue_step(this, n_splits, st); }

}  // namespace

extern "C" {

jllm_b200_decoder* jllm_b200_decoder_create(const jllm_b200_model_desc* model, int flags) {
    if (!model || !model->layers || model->n_layers <= 0) { set_error(JB_ERR_ARG, "decoder: empty model description"); return nullptr; }
    if (model->hidden_dim % QK_K || model->intermediate_dim % QK_K || (model->n_heads * model->head_dim) % QK_K) {
        set_error(JB_ERR_ARG, "decoder: hidden/intermediate/q dims must be multiples of 256"); return nullptr;
    }
    if (!ctx()) return nullptr;
    KquantDecoder* d = new (std::nothrow) KquantDecoder();
    if (!d) return nullptr;
    d->m = *model;
    d->layers.assign(model->layers, model->layers + model->n_layers);
    d->m.layers = d->layers.data();
    d->fused = (flags & 1) != 0; d->use_graph = (flags & 2) != 0; d->chain = (flags & 8) != 0; d->batched_prefill = (flags & 16) != 0;
    jllm::KVCachePool::Config c = { model->n_layers, model->n_kv_heads, model->head_dim, model->max_context, 0, 1 };
    if (!d->kv.init(c) || !d->kv.kv_scale_ptr(0, 0, false)) { set_error(JB_ERR_NOMEM, "decoder: KV pool allocation failed"); jllm_b200_decoder_destroy(d); return nullptr; }
    if (d->alloc()) { jllm_b200_decoder_destroy(d); return nullptr; }
    // scratch that must exist before any graph capture
    splitk_buffer((size_t)model->n_heads * 64 * (model->head_dim + 4), true);
    return d;
}

jllm_b200_decoder* jllm_b200_decoder_create_tp(const jllm_b200_model_desc* model, int flags, int rank, int world, void* const* regions) {
    if (!model || !model->layers || model->n_layers <= 0 || !regions) { set_error(JB_ERR_ARG, "decoder: empty model description"); return nullptr; }
    if (world < 2 || world > TP_MAX_WORLD || rank < 0 || rank >= world) { set_error(JB_ERR_ARG, "decoder: rank %d of %d", rank, world); return nullptr; }
    const int hd = model->head_dim;
    if (model->n_heads % world || model->n_kv_heads % world || model->intermediate_dim % world || model->hidden_dim % world || model->vocab_size % world ||
        ((model->n_heads / world) * hd * 2) % 16 || ((model->hidden_dim / world) * 2) % 16 || ((model->intermediate_dim / world) * 2) % 16) {
        set_error(JB_ERR_ARG, "decoder: heads, hidden, intermediate and vocabulary sizes must split evenly over %d ranks in 16-byte slices", world); return nullptr;
    }
    if (model->hidden_dim % QK_K || model->intermediate_dim % QK_K || (model->n_heads * hd) % QK_K || model->intermediate_dim < model->hidden_dim) {
        set_error(JB_ERR_ARG, "decoder: hidden/intermediate/q dims must be multiples of 256, intermediate >= hidden"); return nullptr;
    }
    // every sharded product pushes its rows from the epilogue of the streaming GEMV, which exists for Q4_K and Q6_K only
    for (int l = 0; l < model->n_layers; ++l) {
        const jllm_b200_layer_desc& w = model->layers[l];
        const int ts[7] = { w.type_wq, w.type_wk, w.type_wv, w.type_wo, w.type_w_gate, w.type_w_up, w.type_w_down };
        for (int t : ts)
            if (t != T_Q4K && t != T_Q6K) { set_error(JB_ERR_TYPE, "decoder: ggml type %d in layer %d has no tensor-parallel path (Q4_K and Q6_K only)", t, l); return nullptr; }
    }
    if (model->output_type != T_Q4K && model->output_type != T_Q6K) { set_error(JB_ERR_TYPE, "decoder: output type %d has no tensor-parallel path", model->output_type); return nullptr; }
    if (!ctx()) return nullptr;
    // This rank's own region may hold the packets of an earlier session, whose epochs would pass for fresh ones: clear it.
    // (The caller must let every rank finish its create before any rank runs a step: a barrier, as TPDecoder does.)
    if (cudaMemset(regions[rank], 0, jllm_b200_tp_region_bytes(model->hidden_dim, model->n_heads * hd, model->intermediate_dim)) != cudaSuccess ||
        cudaDeviceSynchronize() != cudaSuccess) { cuda_error(cudaGetLastError(), "cudaMemset(exchange region)"); return nullptr; }
    KquantDecoder* d = new (std::nothrow) KquantDecoder();
    if (!d) return nullptr;
    d->m = *model;
    d->layers.assign(model->layers, model->layers + model->n_layers);
    d->m.layers = d->layers.data();
    d->fused = true; d->use_graph = (flags & 2) != 0; d->chain = (flags & 8) != 0;
    d->tp_on = true;
    d->nh_l = model->n_heads / world; d->nkv_l = model->n_kv_heads / world; d->I_l = model->intermediate_dim / world;
    d->H_l = model->hidden_dim / world; d->V_l = model->vocab_size / world;
    tp_region_layout(model->hidden_dim, model->n_heads * hd, model->intermediate_dim, d->tp_off);
    for (int r = 0; r < TP_MAX_WORLD; ++r) d->tp.peer[r] = r < world ? (unsigned char*)regions[r] : nullptr;
    d->tp.rank = rank; d->tp.world = world; d->tp.flags_off = d->tp_off[4]; d->tp.argmax_off = d->tp_off[5];
    d->tp.epochs_per_step = model->n_layers; d->tp.status = ctx()->d_status;
    if (cudaMalloc(&d->seq, 256) != cudaSuccess) { cudaGetLastError(); set_error(JB_ERR_NOMEM, "decoder: step counter"); jllm_b200_decoder_destroy(d); return nullptr; }
    cudaMemset(d->seq, 0, 256);
    d->tp.seq = d->seq;
    jllm::KVCachePool::Config c = { model->n_layers, d->nkv_l, hd, model->max_context, 0, 1 };
    if (!d->kv.init(c) || !d->kv.kv_scale_ptr(0, 0, false)) { set_error(JB_ERR_NOMEM, "decoder: KV pool allocation failed"); jllm_b200_decoder_destroy(d); return nullptr; }
    if (d->alloc()) { jllm_b200_decoder_destroy(d); return nullptr; }
    d->vocab = d->V_l;                     // logits of this rank's vocabulary slice
    splitk_buffer((size_t)d->nh_l * 64 * (hd + 4), true);
    return d;
}

}  // extern "C"
