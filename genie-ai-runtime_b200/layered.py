"""Models described layer by layer: configuration, weight loading and the decoder session (jllm_b200_decoder_create_layered).

A configuration lists the layers; each names its mixer ("attention": grouped-query attention without rotation, with a query
temperature and a softmax sink, optionally over an earlier layer's keys and values) and its feed-forward part (None or a
mixture of SwiGLU experts).  Every size and constant is a parameter of the layer.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

from . import lib, check, JllmError, last_error  # noqa: F401
from .decoder import Session, GRAPH, PREFILL
from .registry import register, ConfigError

DTYPES = {"bfloat16": 2, "float32": 3}


@dataclass
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    kv_from: int = -1
    q_temp_coef: float = 0.0
    q_temp_every: float = 0.0        # 0: no temperature


@dataclass
class MoeSpec:
    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1


@dataclass
class LayerSpec:
    mixer: AttentionSpec
    mlp: MoeSpec | None


@dataclass
class LayeredConfig:
    vocab: int
    width: int
    layers: list
    eps: float
    residual_mult: float
    logit_softcap: float

    @classmethod
    def parse(cls, cfg):
        """From a parsed config.json; raises ConfigError on a part that no layer here implements."""
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            if entry["type"] != "attention":
                raise ConfigError(f"layer {i}: mixer {entry['type']!r}")
            m = entry["mixer"]
            t = m.get("q_temp") or {}
            src = m.get("kv_from")
            mixer = AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                                  kv_from=-1 if src is None else src, q_temp_coef=float(t.get("coef", 0.0)), q_temp_every=float(t.get("every", 0.0)))
            mlp = None
            if entry.get("mlp") is not None:
                f = entry["mlp"]
                if f["kind"] != "moe":
                    raise ConfigError(f"layer {i}: feed-forward {f['kind']!r}")
                r = f["router"]
                g = r.get("groups") or {"count": 1, "keep": 1}
                mlp = MoeSpec(experts=r["experts"], top=r["top"], ff=f["expert"]["ff"], groups=g["count"], keep=g["keep"])
            layers.append(LayerSpec(mixer, mlp))
        return cls(vocab=cfg["vocab"], width=cfg["width"], layers=layers, eps=float(cfg["norm"]["eps"]), residual_mult=float(cfg["residual_mult"]),
                   logit_softcap=float(cfg.get("logit_softcap") or 0.0))


class CLayer(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("n_heads", "n_kv_heads", "head_dim", "v_dim", "kv_from")] + \
               [("scale", C.c_float), ("q_temp_coef", C.c_float), ("q_temp_every", C.c_double)] + \
               [(n, C.c_void_p) for n in ("w_qkv", "w_o", "sink", "norm1_w", "norm1_b", "norm1b_w", "norm1b_b")] + \
               [(n, C.c_int) for n in ("n_experts", "top", "n_groups", "keep_groups", "expert_dim")] + \
               [(n, C.c_void_p) for n in ("w_router", "correction", "w_gate", "w_up", "w_down", "norm2_w", "norm2_b", "norm2b_w", "norm2b_b")]


class CModel(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("n_layers", "width", "vocab_size", "max_context", "dtype")] + \
               [(n, C.c_float) for n in ("eps", "residual_mult", "logit_softcap")] + \
               [(n, C.c_void_p) for n in ("embed", "final_w", "final_b")] + [("layers", C.POINTER(CLayer))]


class LayeredWeights:
    """Device tensors of a model in the layout the kernels read, by C field name: `layers[i]` and `top`.  `tensors` maps
    names to torch tensors (any device); matrices become `dtype` rows padded to a multiple of 8, vectors fp32."""

    def __init__(self, cfg: LayeredConfig, tensors, dtype="bfloat16", device="cuda"):
        import torch
        self.cfg, self.dtype = cfg, dtype
        dt = getattr(torch, dtype)
        pad8 = lambda n: (n + 7) // 8 * 8

        def shaped(name, *shape):
            t = tensors[name]
            if tuple(t.shape) != shape:
                raise ConfigError(f"{name} is {tuple(t.shape)}, the configuration says {shape}")
            return t

        def matrix(parts):
            t = torch.cat([p.to(device) for p in parts]) if len(parts) > 1 else parts[0].to(device)
            out = torch.zeros((t.shape[0], pad8(t.shape[1])), dtype=dt, device=device)
            out[:, :t.shape[1]] = t.to(dt)
            return out

        def vector(name, n):
            out = torch.zeros(pad8(n), dtype=torch.float32, device=device)
            out[:n] = shaped(name, n).to(device).float()
            return out

        W = cfg.width
        norm = lambda field, name: {field + "_w": vector(name, W), field + "_b": vector(name + ".b", W)}
        self.top = {"embed": matrix([shaped("embed", cfg.vocab, W)]), **norm("final", "final.norm")}
        self.layers = []
        for i, layer in enumerate(cfg.layers):
            p, a = f"l{i}.", layer.mixer
            rows = [shaped(p + "mix.q", a.heads * a.dim, W)]
            if a.kv_from < 0:
                rows += [shaped(p + "mix.k", a.kv_heads * a.dim, W), shaped(p + "mix.v", a.kv_heads * a.vdim, W)]
            d = {"w_qkv": matrix(rows), "w_o": matrix([shaped(p + "mix.o", W, a.heads * a.vdim)]), "sink": vector(p + "mix.sink", a.heads),
                 **norm("norm1", p + "norm1"), **norm("norm1b", p + "norm1b")}
            if layer.mlp is not None:
                f = layer.mlp
                each = lambda part, *shape: matrix([shaped(f"{p}mlp.e{e}.{part}", *shape) for e in range(f.experts)])
                d.update(w_router=matrix([shaped(p + "mlp.router", f.experts, W)]), w_gate=each("gate", f.ff, W), w_up=each("up", f.ff, W),
                         w_down=each("down", W, f.ff), **norm("norm2", p + "norm2"), **norm("norm2b", p + "norm2b"))
                if p + "mlp.correction" in tensors:
                    d["correction"] = vector(p + "mlp.correction", f.experts)
            self.layers.append(d)


class LayeredDecoder(Session):
    """Session of a layer-list model.  Several sessions may share one LayeredWeights."""

    def __init__(self, weights: LayeredWeights, max_context, flags=GRAPH | PREFILL):
        cfg = weights.cfg
        self._keep = weights
        self._layers = (CLayer * len(cfg.layers))()
        for c, spec, w in zip(self._layers, cfg.layers, weights.layers):
            a = spec.mixer
            c.n_heads, c.n_kv_heads, c.head_dim, c.v_dim, c.kv_from = a.heads, a.kv_heads, a.dim, a.vdim, a.kv_from
            c.scale, c.q_temp_coef, c.q_temp_every = a.scale, a.q_temp_coef, a.q_temp_every
            if spec.mlp is not None:
                f = spec.mlp
                c.n_experts, c.top, c.n_groups, c.keep_groups, c.expert_dim = f.experts, f.top, f.groups, f.keep, f.ff
            for k, t in w.items():
                setattr(c, k, t.data_ptr())
        m = CModel()
        m.n_layers, m.width, m.vocab_size, m.max_context, m.dtype = len(cfg.layers), cfg.width, cfg.vocab, max_context, DTYPES[weights.dtype]
        m.eps, m.residual_mult, m.logit_softcap = cfg.eps, cfg.residual_mult, cfg.logit_softcap
        for k, t in weights.top.items():
            setattr(m, k, t.data_ptr())
        m.layers = self._layers
        self.cfg, self.vocab, self.max_context = cfg, cfg.vocab, max_context
        lib.jllm_b200_decoder_create_layered.restype = C.c_void_p
        import torch
        torch.cuda.synchronize()             # the weights were written on torch's stream
        self._h = lib.jllm_b200_decoder_create_layered(C.byref(m), C.c_int(flags))
        if not self._h:
            raise JllmError(-1, last_error())


@register("Ramilorn", dtypes=tuple(DTYPES))
def _ramilorn(config, tensors, dtype):
    weights = LayeredWeights(LayeredConfig.parse(config), tensors, dtype)
    return lambda max_context, flags=GRAPH | PREFILL: LayeredDecoder(weights, max_context, flags)
