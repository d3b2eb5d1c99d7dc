"""Layer-list models on the GPU against the plain oracle: every mechanism alone, then whole models in both number formats —
prompts against token-by-token decoding, portions of several sizes, sessions that are used again, long decoding, and greedy
generation through the engine and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import layered_models as lm
from gpu_util import pkg
from oracle import layered as orc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL, BF16_TOL = 5e-5, 0.04


def pad8(n):
    return (n + 7) // 8 * 8


def rng(seed):
    return np.random.Generator(np.random.PCG64(seed))


def up(a, dtype="float32", pad=False):
    """numpy -> CUDA tensor of a number format, rows padded to a multiple of 8 with zeros when `pad`."""
    import torch
    t = torch.from_numpy(np.ascontiguousarray(a))
    if t.is_floating_point():
        t = t.to(getattr(torch, dtype))
    if pad and t.shape[-1] % 8:
        z = torch.zeros((*t.shape[:-1], pad8(t.shape[-1])), dtype=t.dtype)
        z[..., :t.shape[-1]] = t
        t = z
    return t.cuda()


def as_np(t):
    import torch
    torch.cuda.synchronize()
    return t.float().cpu().numpy().astype(np.float64)


def rounded(a, dtype):
    import torch
    return torch.from_numpy(np.ascontiguousarray(a, np.float32)).to(getattr(torch, dtype)).float().numpy().astype(np.float64)


# ── the mechanisms alone ─────────────────────────────────────────────────
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [5, 64, 250, 1111])
def test_residual_step(width, dtype):
    import torch
    jb, r = pkg(), rng(width)
    rows, eps, mult = 7, 1e-3, 0.37
    vec = lambda: r.standard_normal(width) + 0.5
    pw, pb, nw, nb = vec(), vec(), vec(), vec()
    x, y = 3 * r.standard_normal((rows, width)) + 2, 5 * r.standard_normal((rows, width)) - 9
    emb = r.standard_normal((11, width))
    tok = r.integers(0, 11, rows)
    top, slots = 3, r.permutation(rows * 3).reshape(rows, 3)
    ye, wt = rounded(r.standard_normal((rows * 3, width)), dtype), r.random((rows, 3))
    tol = 2e-6 if dtype == "float32" else 5e-3
    v = {k: up(a.astype(np.float32), pad=True) for k, a in dict(pw=pw, pb=pb, nw=nw, nb=nb, x=x, y=y).items()}
    embd = up(emb, dtype, True)

    def run(**kw):
        h = torch.zeros((rows, pad8(width)), dtype=getattr(torch, dtype), device="cuda")
        xo = torch.zeros((rows, pad8(width)), dtype=torch.float32, device="cuda")
        jb.norm_step(h, xo, v["nw"], v["nb"], eps, width, mult=mult, **kw)
        return as_np(h)[:, :width], as_np(xo)[:, :width]
    for kw, want_x in ((dict(tokens=up(tok.astype(np.int32)), embed=embd), rounded(emb, dtype)[tok]),
                       (dict(x=v["x"], y=v["y"], post_w=v["pw"], post_b=v["pb"]), x + mult * orc.layer_norm(y, pw, pb, eps)),
                       (dict(x=v["x"], y_exp=up(ye, dtype, True), slots=up(slots.astype(np.int32)), weights=up(wt.astype(np.float32)), post_w=v["pw"], post_b=v["pb"]),
                        x + mult * orc.layer_norm((wt[:, :, None] * ye[slots]).sum(1), pw, pb, eps))):
        h, xo = run(**kw)
        assert np.abs(xo - want_x).max() < 1e-5 * np.abs(want_x).max()
        want_h = orc.layer_norm(want_x, nw, nb, eps)
        assert np.abs(h - want_h).max() < tol * max(1.0, np.abs(want_h).max())


HEADS = [(8, 4, 64, 64), (6, 2, 48, 32), (5, 5, 40, 72), (20, 1, 16, 24), (3, 1, 128, 96), (4, 2, 256, 200), (2, 2, 12, 20), (34, 2, 8, 8), (2, 1, 300, 264)]


def _planted(r, T, S, H, G, dim, vdim, start, dtype):
    """Random q / k / v in which some queries have one key that stands out: the first, the last they may see, and keys in
    between, at and around multiples of 16 and 64."""
    q, k, v = r.standard_normal((T, H, dim)), r.standard_normal((S, G, dim)), r.standard_normal((S, G, vdim))
    for t in range(T):
        p = start + t
        places = [0, p, p // 2, max(0, p // 16 * 16 - 1), p // 16 * 16, max(0, p // 64 * 64 - 1), p // 64 * 64, max(0, p - 1)]
        j = places[t % len(places)]
        for h in range(H):
            if (t + h) % 3 == 0:
                kk = k[j, h // (H // G)]
                q[t, h] = kk * (6.0 * np.sqrt(dim) / (kk @ kk))
    return rounded(q, dtype), rounded(k, dtype), rounded(v, dtype)


def _attend(jb, q, k, v, dtype, scale, start, sink, temp, decode_splits=None):
    import torch
    T, H, dim = q.shape
    _, G, vdim = v.shape
    qd = up(q.reshape(T, -1), dtype, True)
    out = torch.zeros((T, pad8(H * vdim)), dtype=qd.dtype, device="cuda")
    kd, vd = up(k.reshape(k.shape[0], -1), dtype), up(v.reshape(v.shape[0], -1), dtype)
    kw = dict(sink=None if sink is None else up(sink.astype(np.float32)), q_temp=temp or (0.0, 0.0))
    if decode_splits is None:
        jb.sink_attention(out, qd, kd, vd, H, G, dim, vdim, scale, n_tokens=T, start=start, **kw)
    else:
        jb.sink_attention(out, qd, kd, vd, H, G, dim, vdim, scale, seq_len=start + 1, n_splits=decode_splits, **kw)
    return as_np(out)[:, :H * vdim]


def _want(q, k, v, scale, start, sink, temp):
    T, H, _ = q.shape
    s = np.full(H, -np.inf) if sink is None else sink
    with np.errstate(invalid="ignore"):
        return orc.attention(q, k, v, s, scale, start + np.arange(T), None if temp is None else dict(coef=temp[0], every=temp[1]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dim,vdim", HEADS)
def test_prompt_attention(H, G, dim, vdim, dtype):
    jb, r = pkg(), rng(H * 1000 + dim)
    sink = r.standard_normal(H) + 1
    tol = 3e-6 if dtype == "float32" else 1.5e-2
    for start, T, sk, temp in ((0, 1, sink, None), (0, 2, sink, (0.5, 3)), (0, 130, sink, (0.3, 16)), (37, 65, sink, None), (63, 2, None, (0.7, 64)), (127, 200, sink, (0.4, 100))):
        q, k, v = _planted(r, T, start + T, H, G, dim, vdim, start, dtype)
        scale = 1.7 / np.sqrt(dim)
        got, want = _attend(jb, q, k, v, dtype, scale, start, sk, temp), _want(q, k, v, scale, start, sk, temp)
        assert np.abs(got - want).max() < tol * max(1.0, np.abs(want).max()), (start, T)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dim,vdim", HEADS)
def test_decode_attention_and_its_slices(H, G, dim, vdim, dtype):
    jb, r = pkg(), rng(H * 77 + dim)
    sink = r.standard_normal(H) + 1
    tol = 3e-6 if dtype == "float32" else 1.5e-2
    for n in (1, 2, 15, 16, 17, 63, 64, 65, 255, 256, 257, 700):
        q, k, v = _planted(r, 1, n, H, G, dim, vdim, n - 1, dtype)
        if n % 2:                                             # a far key for the decoded query
            kk = k[n // 3, 0]
            q[0, 0] = rounded(kk * (6.0 * np.sqrt(dim) / (kk @ kk)), dtype)
        scale = 1.7 / np.sqrt(dim)
        want = _want(q, k, v, scale, n - 1, sink, (0.4, 32))
        for splits in (0, 1, 2, 7, 16):
            got = _attend(jb, q, k, v, dtype, scale, n - 1, sink, (0.4, 32), splits)
            assert np.abs(got - want).max() < tol * max(1.0, np.abs(want).max()), (n, splits)


def test_a_large_sink_silences_a_head():
    jb, r = pkg(), rng(3)
    for dtype in ("float32", "bfloat16"):
        q, k, v = _planted(r, 9, 9, 4, 2, 32, 32, 0, dtype)
        sink = np.array([200.0, -200.0, 0.0, 3.0])
        got = _attend(jb, q, k, v, dtype, 0.2, 0, sink, None).reshape(9, 4, 32)
        assert not got[:, 0].any() and np.isfinite(got).all()
        want = _want(q, k, v, 0.2, 0, sink, None).reshape(9, 4, 32)
        assert np.abs(got - want).max() < 1.5e-2 * np.abs(want).max()


@pytest.mark.parametrize("E,top,groups", [(12, 3, (3, 2)), (5, 1, None), (6, 6, None), (64, 6, (8, 3)), (40, 7, (20, 5)), (100, 9, (4, 1)), (1, 1, None), (256, 8, (8, 4)), (7, 2, (7, 3))])
def test_router(E, top, groups):
    import torch
    jb, r = pkg(), rng(E)
    rows = 67
    z = (2 * r.standard_normal((rows, E))).astype(np.float32)
    for corr in (None, (-0.6 + 0.5 * r.standard_normal(E)).astype(np.float32)):
        want_ids, want_w = orc.choose_experts(z.astype(np.float64), None if corr is None else corr.astype(np.float64), top, groups and dict(count=groups[0], keep=groups[1]))
        ids, rank = (torch.full((rows, top), -1, dtype=torch.int32, device="cuda") for _ in range(2))
        wts = torch.zeros((rows, top), dtype=torch.float32, device="cuda")
        counts = torch.zeros(E, dtype=torch.int32, device="cuda")
        jb.moe_route(ids, wts, rank, counts, up(z), top, *(groups or (1, 1)), correction=None if corr is None else up(corr))
        ids, rank = ids.cpu().numpy(), rank.cpu().numpy()
        assert np.array_equal(ids, want_ids)
        assert np.abs(as_np(wts) - want_w).max() < 1e-6
        assert np.array_equal(counts.cpu().numpy(), np.bincount(want_ids.ravel(), minlength=E))
        for e in range(E):                                    # ranks are a permutation of the places of each expert
            assert sorted(rank[ids == e]) == list(range((ids == e).sum()))


def test_router_limits_are_errors():
    import torch
    jb = pkg()
    i, f = torch.zeros((1, 8), dtype=torch.int32, device="cuda"), torch.zeros((1, 9), dtype=torch.float32, device="cuda")
    for top, groups in ((0, (1, 1)), (8, (3, 1)), (2, (2, 1)), (2, (3, 0))):
        with pytest.raises(jb.JllmError):
            jb.moe_route(i, f, i, torch.zeros(9, dtype=torch.int32, device="cuda"), f, top, *groups)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M,N,K", [(1, 2, 8), (130, 33, 50), (128, 257, 64), (77, 1, 200), (300, 600, 72), (512, 40, 1000), (2000, 300, 136)])
def test_dense_product(M, N, K, dtype):
    import torch
    jb, r = pkg(), rng(M + N)
    W, V, x = (rounded(r.standard_normal(s), dtype) for s in ((M, K), (M, K), (N, K)))
    dev = lambda a: up(a, dtype, True)
    tol = 1e-5 if dtype == "float32" else 1e-2
    y = torch.zeros((N, M), dtype=torch.float32, device="cuda")
    jb.dense_matmul(y, dev(W), dev(x), M, N, K, softcap=20.0)
    want = orc.softcap(x @ W.T, 20.0)
    assert np.abs(as_np(y) - want).max() < 1e-5 * np.sqrt(K)
    ya = torch.zeros((N, M if dtype == "float32" else pad8(M)), dtype=getattr(torch, dtype), device="cuda")      # fp32 rows are not padded
    jb.dense_matmul(ya, dev(W), dev(x), M, N, K, W_up=dev(V))
    want = orc.silu(x @ W.T) * (x @ V.T)
    assert np.abs(as_np(ya)[:, :M] - want).max() < tol * np.abs(want).max() and not as_np(ya)[:, M:].any()
    y1 = torch.zeros(M, dtype=torch.float32, device="cuda")
    jb.dense_matvec(y1, dev(W), dev(x)[0], M, K)
    assert np.abs(as_np(y1) - W @ x[0]).max() < 1e-5 * np.sqrt(K)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_grouped_product_with_empty_and_uneven_groups(dtype):
    import torch
    jb, r = pkg(), rng(9)
    for M, K, counts in ((72, 56, [0, 3, 0, 130, 1, 31, 32, 33, 0]), (200, 24, [64, 0, 65]), (136, 40, [1] * 40), (8, 8, [0, 0, 5])):
        N, G = sum(counts), len(counts)
        off = np.concatenate([[0], np.cumsum(counts)]).astype(np.int32)
        W, V, x = (rounded(r.standard_normal(s), dtype) for s in ((G * M, K), (G * M, K), (N, K)))
        y = torch.full((N + 4, M), 7.0, dtype=torch.float32, device="cuda")
        ya = torch.zeros((N, M if dtype == "float32" else pad8(M)), dtype=getattr(torch, dtype), device="cuda")
        jb.dense_matmul(y, up(W, dtype, True), up(x, dtype, True), M, N, K, group_offsets=up(off), n_groups=G)
        jb.dense_matmul(ya, up(W, dtype, True), up(x, dtype, True), M, N, K, W_up=up(V, dtype, True), group_offsets=up(off), n_groups=G)
        got, gota = as_np(y), as_np(ya)
        assert (got[N:] == 7).all()
        for g in range(G):
            s, w = slice(off[g], off[g + 1]), slice(g * M, (g + 1) * M)
            a, b = x[s] @ W[w].T, x[s] @ V[w].T
            assert np.abs(got[s] - a).max(initial=0) < 1e-5 * np.sqrt(K)
            want = orc.silu(a) * b
            assert np.abs(gota[s, :M] - want).max(initial=0) <= (1e-5 if dtype == "float32" else 1e-2) * np.abs(want).max(initial=0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,top,groups,ff,width", [(12, 3, (3, 2), 40, 72), (5, 1, None, 21, 50), (6, 6, None, 8, 320), (64, 8, (8, 4), 136, 256)])
def test_experts_of_one_token(E, top, groups, ff, width, dtype):
    import torch
    jb, r = pkg(), rng(E + ff)
    gate, upw, down, h = (rounded(r.standard_normal(s) / np.sqrt(s[-1]), dtype) for s in ((E, ff, width), (E, ff, width), (E, width, ff), (1, width)))
    h = rounded(h * np.sqrt(width), dtype)
    z = (2 * r.standard_normal((1, E))).astype(np.float32)
    corr = (0.4 * r.standard_normal(E) - 0.2).astype(np.float32)
    ids, wt = orc.choose_experts(z.astype(np.float64), corr.astype(np.float64), top, groups and dict(count=groups[0], keep=groups[1]))
    want = sum(wt[0, k] * orc.expert(h[0], gate[e], upw[e], down[e]) for k, e in enumerate(ids[0]))
    dt = getattr(torch, dtype)
    y = torch.zeros(width, dtype=torch.float32, device="cuda")
    act = torch.zeros((top, pad8(ff)), dtype=dt, device="cuda")
    gi, gw = torch.zeros(top, dtype=torch.int32, device="cuda"), torch.zeros(top, dtype=torch.float32, device="cuda")
    jb.moe_matvec(y, act, gi, gw, up(gate.reshape(-1, width), dtype, True), up(upw.reshape(-1, width), dtype, True), up(down.reshape(-1, ff), dtype, True),
                  up(h[0], dtype, True), up(z), top, ff, width, *(groups or (1, 1)), correction=up(corr))
    assert np.array_equal(gi.cpu().numpy(), ids[0])
    assert np.abs(as_np(y) - want).max() < (2e-6 if dtype == "float32" else 1e-2) * max(1.0, np.abs(want).max())


# ── whole models ─────────────────────────────────────────────────────────
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """(name, number format) -> configuration, weights, folder.  In bf16 the corrections are spread so far that no routing
    decision hangs on the rounding of the router's input, and the attention is not sharpened (bf16 queries alone would move
    its logits by a few percent); fp32 has both, the mechanism tests have both in bf16."""
    out = {}
    for name, cfg in lm.CONFIGS.items():
        for dtype in ("float32", "bfloat16"):
            w = lm.weights(cfg, 100 + len(name), sharp=1.6, clear_routing=False) if dtype == "float32" else lm.weights(cfg, 100 + len(name), clear_routing=True)
            out[name, dtype] = (cfg, w, lm.save(tmp_path_factory.mktemp(name), cfg, w))
    return out


_forward_cache = {}


def oracle_logits(name, dtype, cfg, w, tokens):
    key = (name, dtype, tuple(int(t) for t in tokens))
    if key not in _forward_cache:
        _forward_cache[key] = orc.forward(cfg, w, tokens)
    return _forward_cache[key]


def check_logits(got, want, dtype):
    err = lm.logit_error(got, want)
    assert err.max() < (F32_TOL if dtype == "float32" else BF16_TOL), (err.max(), int(err.argmax()))


def fed(engine, rid, tokens, cuts):
    got, at = [], 0
    for c in cuts:
        c = min(c, len(tokens) - at)
        if c <= 0:
            break
        got.append(engine.feed(rid, tokens[at:at + c], range(c)))
        at += c
    assert at == len(tokens)
    engine.end(rid)
    return np.concatenate(got)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(lm.CONFIGS))
def test_prompt_decoding_and_portions(models, name, dtype):
    cfg, w, folder = models[name, dtype]
    tokens = [int(t) for t in rng(17).integers(0, cfg["vocab"], 150)]
    want = oracle_logits(name, dtype, cfg, w, tokens)
    e = pkg().engine.Engine(folder, dtype, 160)
    for cuts in ([150], [1] * 150, [2] * 75, [3] * 50, [64, 1, 1, 63, 2, 1, 18], [7, 100, 1, 42], [149, 1], [1, 149]):
        check_logits(fed(e, "r", tokens, cuts), want, dtype)       # one session, used again and again
    assert len(e._free) == 1
    e.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompts_are_chunked_inside_the_session(models, dtype):
    cfg, w, folder = models["mixed", dtype]
    tokens = [int(t) for t in rng(18).integers(0, cfg["vocab"], 150)]
    _, open_session = pkg().registry.open_model(folder, dtype)
    s = open_session(160)
    for chunk in (2, 5, 149):
        s.prefill(tokens, 0, chunk=chunk)
        last = as_np(s.logits())[None]
        s.reset()
        got = s.feed(tokens, 0, range(150))
        check_logits(got, oracle_logits("mixed", dtype, cfg, w, tokens), dtype)
        check_logits(last, oracle_logits("mixed", dtype, cfg, w, tokens)[-1:], dtype)
        s.reset()
    s.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_interleaved_requests_equal_each_alone(models, dtype):
    cfg, w, folder = models["mixed", dtype]
    e = pkg().engine.Engine(folder, dtype, 64)
    reqs = {f"q{i}": [int(t) for t in rng(30 + i).integers(0, cfg["vocab"], n)] for i, n in enumerate((40, 1, 23, 9))}
    alone = {k: fed(e, k, t, [len(t)]) for k, t in reqs.items()}
    at, got = {k: 0 for k in reqs}, {k: [] for k in reqs}
    step = 0
    while any(at[k] < len(t) for k, t in reqs.items()):
        for i, (k, t) in enumerate(reqs.items()):
            c = min((step + i) % 4 + 1, len(t) - at[k])
            if c > 0:
                got[k].append(e.feed(k, t[at[k]:at[k] + c], range(c)))
                at[k] += c
                if at[k] == len(t):
                    e.end(k)
        step += 1
    for k, t in reqs.items():
        check_logits(np.concatenate(got[k]), alone[k].astype(np.float64), dtype)
        check_logits(np.concatenate(got[k]), oracle_logits("mixed", dtype, cfg, w, t), dtype)
    e.close()


def test_long_decoding_crosses_the_slice_counts(models):
    """700 positions, the last 460 decoded one by one: KV slices 1, 2 and 4 of the bf16 attention, and the fp32 path's."""
    for dtype in ("float32", "bfloat16"):
        cfg, w, folder = models["mixed", dtype]
        tokens = [int(t) for t in rng(77).integers(0, cfg["vocab"], 700)]
        want = oracle_logits("mixed", dtype, cfg, w, tokens)
        e = pkg().engine.Engine(folder, dtype, 700)
        check_logits(fed(e, "r", tokens, [240] + [1] * 460), want, dtype)
        e.close()


def greedy(cfg, w, prompt, n):
    """Greedy continuation by the oracle, with the margin of each choice."""
    seq, margins = list(prompt), []
    for _ in range(n):
        lg = orc.forward(cfg, w, seq)[-1]
        order = np.argsort(-lg)
        seq.append(int(order[0]))
        margins.append(float(lg[order[0]] - lg[order[1]]))
    return seq[len(prompt):], margins


def test_greedy_generation_through_the_engine_and_the_command_line(models):
    cfg, w, folder = models["odd", "float32"]
    prompts = [[5, 17, 3, 99, 4], [42], [int(t) for t in rng(4).integers(0, cfg["vocab"], 33)]]
    want = [greedy(cfg, w, p, 12) for p in prompts]
    jb = pkg()
    e = jb.engine.Engine(folder, "float32", 64)
    got = e.generate(prompts, 12)
    again = e.generate(prompts[::-1], 12)[::-1]
    e.close()
    assert got == again
    for g, (t, margins) in zip(got, want):
        upto = next((i for i, m in enumerate(margins) if m < 1e-3), 12)
        assert g[:upto] == t[:upto], (g, t, margins)
    r = subprocess.run([sys.executable, os.path.join(ROOT, "genie-ai-runtime_b200", "generate.py"), "--model", folder, "--dtype", "float32", "--new", "12"] +
                       [",".join(map(str, p)) for p in prompts], capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-800:]
    assert [json.loads(l)["tokens"] for l in r.stdout.splitlines()] == got


def test_trace_command(models, tmp_path):
    cfg, w, folder = models["odd", "float32"]
    tokens = [int(t) for t in rng(8).integers(0, cfg["vocab"], 20)]
    steps = [dict(step=0, entries=[dict(id="x", tokens=tokens[:15], want=[0, 14])], end=[]),
             dict(step=1, entries=[dict(id="x", tokens=tokens[15:16], want=[])], end=[]),
             dict(step=2, entries=[dict(id="x", tokens=tokens[16:], want=[1, 3])], end=["x"]),
             dict(step=3, entries=[dict(id="y", tokens=tokens[:1], want=[0])], end=["y"])]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "20"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-800:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    want = oracle_logits("odd", "float32", cfg, w, tokens)
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"])
    check_logits(read(0), want[[0, 14]], "float32")
    check_logits(read(2), want[[17, 19]], "float32")
    check_logits(read(3), want[:1], "float32")
    assert not (tmp_path / "1.f32").exists()


def test_session_limits_are_errors(models):
    cfg, w, folder = models["odd", "float32"]
    jb = pkg()
    _, open_session = jb.registry.open_model(folder, "bfloat16")
    s = open_session(8)
    with pytest.raises(jb.JllmError):
        s.feed(list(range(9)), 0, [])
    with pytest.raises(jb.JllmError):
        s.feed([cfg["vocab"]], 0, [0])
    with pytest.raises(jb.JllmError):
        s.feed([1, 2], 0, [1, 0])
    assert s.feed([1, 2], 0, [1]).shape == (1, cfg["vocab"])
    s.close()


def test_kquant_model_folder_opens_through_the_registry(tmp_path):
    """The K-quant family through the same registry, engine and feed call as the session it already had."""
    import importlib
    import torch
    from oracle import oracle as kq
    jb = pkg()
    m = kq.gen_model(42, n_layers=2, hidden=512, n_heads=8, n_kv=2, hd=128, ffn=1024, vocab=1000)
    t = {}
    rows = dict(wq=1024, wk=256, wv=256, wo=512, gate=1024, up=1024, down=512)
    img = lambda a, n: torch.from_numpy(np.ascontiguousarray(a).view(np.uint8).reshape(n, -1).copy())
    for i, lw in enumerate(m["layers"]):
        for k, v in lw.items():
            t[f"blk.{i}.{k}"] = img(v[0], rows[k]) if isinstance(v, tuple) else torch.from_numpy(v)
    t["tok_embd"], t["output"], t["out_norm"] = img(m["tok_embd"][0], 1000), img(m["output"][0], 1000), torch.from_numpy(m["out_norm"])
    importlib.import_module(jb.__name__ + ".safetensors").save_file(t, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(dict(m["cfg"], architecture="Qwen3KQuant")))
    e = jb.engine.Engine(str(tmp_path), None, 64)
    prompt = [int(x) for x in rng(2).integers(0, 1000, 12)]
    d = jb.decoder.Decoder(m["cfg"], jb.decoder.upload(m), 64, jb.decoder.FUSED | jb.decoder.GRAPH | jb.decoder.PREFILL)
    assert e.generate([prompt], 8)[0] == [int(x) for x in d.generate(prompt, 8)]
    d.reset()
    d.prefill(prompt)
    assert np.array_equal(e.feed("a", prompt, [11])[0], d.logits().cpu().numpy())
    nxt = d.last_token()
    one = e.feed("a", [nxt], [0])
    d.step(nxt, 12)
    assert np.array_equal(one[0], d.logits().cpu().numpy())
    e.end("a")
    e.close()
    d.close()
