"""K-quant Llama / Qwen3 models in a model folder: config.json carries the sizes, model.safetensors the GGUF block images.

Matrices are uint8 [rows, bytes per row] under `blk.<i>.wq|wk|wv|wo|gate|up|down`, `tok_embd` and `output`; the block format
(Q4_K, Q5_K, Q6_K) follows from the bytes of a row.  Norm vectors are float32: `blk.<i>.rms_attn|rms_ffn|q_norm|k_norm` (the
last two optional) and `out_norm`."""
from __future__ import annotations

from . import Q4_K, Q5_K, Q6_K
from .decoder import Decoder, FUSED, GRAPH, PREFILL
from .registry import register, ConfigError

_BLOCK_BYTES = {144: Q4_K, 176: Q5_K, 210: Q6_K}


def _matrix(tensors, name, K):
    t = tensors[name]
    kind = _BLOCK_BYTES.get(t.shape[1] * 256 // K)
    if kind is None or K % 256 or t.shape[1] % (K // 256):
        raise ConfigError(f"{name}: rows of {t.shape[1]} bytes for {K} weights")
    return t.cuda().contiguous(), kind


@register("Qwen3KQuant", dtypes=("float16",))
def _kquant(config, tensors, dtype):
    cfg = {k: config[k] for k in ("n_layers", "hidden", "n_heads", "n_kv_heads", "head_dim", "ffn", "vocab", "rope_theta", "eps")}
    H, QD, I = cfg["hidden"], cfg["n_heads"] * cfg["head_dim"], cfg["ffn"]
    inner = dict(wq=H, wk=H, wv=H, wo=QD, gate=H, up=H, down=I)
    weights = dict(tok_embd=_matrix(tensors, "tok_embd", H), output=_matrix(tensors, "output", H), out_norm=tensors["out_norm"].cuda(), layers=[])
    for i in range(cfg["n_layers"]):
        p = f"blk.{i}."
        lw = {k: _matrix(tensors, p + k, K) for k, K in inner.items()}
        lw.update({k: tensors[p + k].cuda() for k in ("rms_attn", "rms_ffn", "q_norm", "k_norm") if p + k in tensors})
        weights["layers"].append(lw)
    return lambda max_context, flags=FUSED | GRAPH | PREFILL: Decoder(cfg, weights, max_context, flags)
