// attention.cu — which attention kernel serves a call.
#include "attention.cuh"

namespace jb {

int launch_attention(const AttnCall& c, cudaStream_t st) {
    if (c.n_heads <= 0 || c.n_kv <= 0 || c.n_heads % c.n_kv) return set_error(JB_ERR_ARG, "attention: n_heads=%d n_kv_heads=%d", c.n_heads, c.n_kv);
    if (!c.out || !c.q) return set_error(JB_ERR_PTR, "attention: null q/out");
    if (!c.k_list && (!c.k || !c.v)) return set_error(JB_ERR_PTR, "attention: null cache pointer");
    // INT8 / head_dim 128 with a known cache extent (a length, a device-side position with its bound, or a plan of tensor
    // maps for a ragged batch): 2-D TMA tiles on the tensor cores; everything else — FP16 caches, other head sizes, sliding
    // windows, pointer lists that live in device memory — goes to the general kernel
    if (c.kind() == EK_BF16 || c.kind() == EK_F32) return launch_attention_float(c, st);
    if (c.causal_start >= 0) return attention_prefill_fast_applies(c) ? launch_attention_prefill_fast(c, st) : launch_attention_general(c, st);
    return attention_tma_applies(c) ? launch_attention_tma(c, st) : launch_attention_general(c, st);
}

}  // namespace jb
