"""Plain restatement of the layer-list decoder models (Ramilorn), one function per mechanism, in float64 numpy.

The oracle of the layer-list path: slow, no cache, no batching, nothing shared with the library.  A model is its
configuration dict (the parsed config.json) and a dict of tensors by name.  All functions take and return float64
arrays; a sequence is a [tokens, width] array.
"""
import numpy as np


def layer_norm(x, w, b, eps):
    mu = x.mean(axis=-1, keepdims=True)
    var = ((x - mu) ** 2).mean(axis=-1, keepdims=True)
    return (x - mu) / np.sqrt(var + eps) * w + b


def query_temperature(pos, coef, every):
    """Factor of the queries at each position: grows by coef * ln n at the start of every n-th run of `every` positions."""
    return 1.0 + coef * np.log(np.floor((np.asarray(pos, np.float64) + 1.0) / every) + 1.0)


def sink_softmax(scores, sink):
    """Softmax over the last axis with one extra term exp(sink) in the denominator; -inf scores are masked keys."""
    top = np.maximum(scores.max(axis=-1), sink)
    e = np.exp(scores - top[..., None])
    return e / (e.sum(axis=-1) + np.exp(sink - top))[..., None]


def attention(q, k, v, sink, scale, positions, q_temp=None):
    """Causal attention of queries at `positions` over keys at 0..len(k)-1.  q [T, H, dim], k [S, G, dim], v [S, G, vdim]."""
    T, H, _ = q.shape
    S, G, _ = k.shape
    positions = np.asarray(positions)
    if q_temp is not None:
        q = q * query_temperature(positions, q_temp["coef"], q_temp["every"])[:, None, None]
    seen = np.arange(S)[None, :] <= positions[:, None]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(seen, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        out[:, h] = sink_softmax(s, np.float64(sink[h])) @ v[:, g]
    return out.reshape(T, -1)


def silu(z):
    return z / (1.0 + np.exp(-z))


def expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def choose_experts(z, correction, top, groups=None):
    """Router logits [T, E] -> (indices [T, top], weights [T, top])."""
    s = 1.0 / (1.0 + np.exp(-z))
    choice = s if correction is None else s + correction
    T, E = z.shape
    ids = np.zeros((T, top), np.int64)
    for t in range(T):
        c = choice[t].copy()
        if groups is not None:
            n = E // groups["count"]
            two = [np.sort(c[g * n:(g + 1) * n])[::-1][:2].sum() for g in range(groups["count"])]
            kept = np.argsort(-np.asarray(two), kind="stable")[:groups["keep"]]
            for g in range(groups["count"]):
                if g not in kept:
                    c[g * n:(g + 1) * n] = -np.inf
        ids[t] = np.argsort(-c, kind="stable")[:top]
    return ids, np.take_along_axis(s, ids, axis=1)


def moe(h, w, prefix, mlp):
    r = mlp["router"]
    ids, wt = choose_experts(h @ w[prefix + "router"].T, w.get(prefix + "correction"), r["top"], r.get("groups"))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(r["top"]):
            e = f"{prefix}e{ids[t, j]}."
            out[t] += wt[t, j] * expert(h[t], w[e + "gate"], w[e + "up"], w[e + "down"])
    return out


def project_kv(h, w, prefix, mixer):
    T = h.shape[0]
    return ((h @ w[prefix + "k"].T).reshape(T, mixer["kv_heads"], mixer["dim"]),
            (h @ w[prefix + "v"].T).reshape(T, mixer["kv_heads"], mixer["vdim"]))


def mix(h, w, prefix, mixer, kv):
    T = h.shape[0]
    q = (h @ w[prefix + "q"].T).reshape(T, mixer["heads"], mixer["dim"])
    a = attention(q, kv[0], kv[1], w[prefix + "sink"], mixer["scale"], np.arange(T), mixer.get("q_temp"))
    return a @ w[prefix + "o"].T


def softcap(z, cap):
    return z if not cap else cap * np.tanh(z / cap)


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; appends the residual stream after every layer to layers_out."""
    w = {k: np.asarray(v, np.float64) for k, v in w.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    norm = lambda name, z: layer_norm(z, w[name], w[name + ".b"], eps)
    x = w["embed"][np.asarray(tokens)]
    store = {}
    for i, layer in enumerate(cfg["layers"]):
        p, mixer = f"l{i}.", layer["mixer"]
        h = norm(p + "norm1", x)
        src = mixer.get("kv_from")
        if src is None:
            src = i
            store[i] = project_kv(h, w, p + "mix.", mixer)
        x = x + m * norm(p + "norm1b", mix(h, w, p + "mix.", mixer, store[src]))
        if layer.get("mlp"):
            x = x + m * norm(p + "norm2b", moe(norm(p + "norm2", x), w, p + "mlp.", layer["mlp"]))
        if layers_out is not None:
            layers_out.append(x)
    return softcap(norm("final.norm", x) @ w["embed"].T, cfg.get("logit_softcap"))
