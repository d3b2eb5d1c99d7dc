"""Small random models described layer by layer, for the tests: configurations, weights and model folders."""
import json
import os

import numpy as np


def attn(heads, kv_heads, dim, vdim, scale=None, kv_from=None, q_temp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale if scale is not None else dim ** -0.5)
    if kv_from is not None:
        m["kv_from"] = kv_from
    if q_temp is not None:
        m["q_temp"] = dict(coef=q_temp[0], every=q_temp[1])
    return m


def moe(experts, top, ff, groups=None):
    r = dict(experts=experts, top=top)
    if groups is not None:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    return dict(kind="moe", expert=dict(ff=ff), router=r)


def config(vocab, width, layers, eps=1e-4, mult=0.8, softcap=25.0):
    c = dict(architecture="Ramilorn", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult,
             layers=[dict(type="attention", mixer=m, mlp=f) for m, f in layers])
    if softcap is not None:
        c["logit_softcap"] = softcap
    return c


CONFIGS = {
    # layers that differ in everything, a layer without feed-forward part, keys of layer 0 under another temperature
    "mixed": config(149, 72, [(attn(6, 2, 24, 40, q_temp=(0.3, 7)), moe(12, 3, 40, (3, 2))),
                              (attn(4, 4, 16, 16), None),
                              (attn(6, 2, 24, 40, scale=0.31, kv_from=0, q_temp=(0.8, 50)), moe(6, 6, 24)),
                              (attn(3, 1, 136, 8, q_temp=(0.5, 1)), moe(5, 1, 100))], mult=0.7, softcap=12.0),
    # nothing is a multiple of 8; two readers of one layer's keys, one of them across a layer with keys of its own
    "odd": config(101, 50, [(attn(4, 2, 10, 14, q_temp=(0.4, 5)), moe(9, 2, 21, (3, 1))),
                            (attn(2, 1, 33, 7), moe(4, 2, 13, (2, 1))),
                            (attn(4, 2, 10, 14, kv_from=0), None),
                            (attn(4, 2, 10, 14, kv_from=0, q_temp=(1.0, 3)), moe(8, 4, 30, (4, 3)))], eps=1e-3, mult=1.0, softcap=None),
    # many query heads per KV head, wide heads
    "wide": config(203, 320, [(attn(40, 2, 64, 48, q_temp=(0.2, 16)), moe(64, 6, 72, (8, 3))),
                              (attn(5, 5, 256, 200), moe(16, 2, 136, (4, 2))),
                              (attn(5, 5, 256, 200, kv_from=1, q_temp=(0.6, 11)), moe(3, 2, 56))], mult=0.3, softcap=50.0),
}


def weights(cfg, seed, sharp=1.0, clear_routing=False):
    """Random tensors (float32, values that bf16 holds exactly).  `sharp` scales queries and keys, so that single keys stand
    out; the sinks are large enough to matter.  clear_routing: corrections so far apart that they decide the choice alone."""
    rng = np.random.Generator(np.random.PCG64(seed))
    W = cfg["width"]

    def bf16(a):
        u = np.ascontiguousarray(a, np.float32).view(np.uint32)
        return ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)
    mat = lambda o, i, g=1.0: bf16(rng.standard_normal((o, i)) * g / np.sqrt(i))
    out = {"embed": bf16(rng.standard_normal((cfg["vocab"], W)))}

    def norm(name):
        out[name] = bf16(1.0 + 0.3 * rng.standard_normal(W))
        out[name + ".b"] = bf16(0.3 * rng.standard_normal(W))
    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, a = f"l{i}.", layer["mixer"]
        norm(p + "norm1")
        norm(p + "norm1b")
        out[p + "mix.q"] = mat(a["heads"] * a["dim"], W, sharp)
        if a.get("kv_from") is None:
            out[p + "mix.k"] = mat(a["kv_heads"] * a["dim"], W, sharp)
            out[p + "mix.v"] = mat(a["kv_heads"] * a["vdim"], W)
        out[p + "mix.sink"] = bf16(1.0 + 1.5 * rng.standard_normal(a["heads"]))
        out[p + "mix.o"] = mat(W, a["heads"] * a["vdim"])
        if layer.get("mlp"):
            r, ff = layer["mlp"]["router"], layer["mlp"]["expert"]["ff"]
            norm(p + "norm2")
            norm(p + "norm2b")
            out[p + "mlp.router"] = mat(r["experts"], W, 2.0)
            out[p + "mlp.correction"] = bf16(-0.3 + 0.4 * rng.standard_normal(r["experts"]))
            if clear_routing:
                out[p + "mlp.correction"] = bf16(4.0 * (rng.permutation(r["experts"]) - r["experts"] // 2))
            for e in range(r["experts"]):
                q = f"{p}mlp.e{e}."
                out[q + "gate"], out[q + "up"], out[q + "down"] = mat(ff, W, 1.5), mat(ff, W), mat(W, ff)
    return out


def save(folder, cfg, w):
    """A model folder: config.json and bf16 model.safetensors."""
    import torch
    from __graft_entry__ import load_package
    import importlib
    jb = load_package()
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    st = importlib.import_module(jb.__name__ + ".safetensors")
    st.save_file({k: torch.from_numpy(np.ascontiguousarray(v)).to(torch.bfloat16) for k, v in w.items()}, os.path.join(folder, "model.safetensors"))
    return str(folder)


def logit_error(got, want):
    """Per position: RMS over the vocabulary of the difference (mean taken off), relative to the RMS of the logits."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=1, keepdims=True)
    c = want - want.mean(axis=1, keepdims=True)
    return np.sqrt((d ** 2).mean(axis=1)) / np.sqrt((c ** 2).mean())
