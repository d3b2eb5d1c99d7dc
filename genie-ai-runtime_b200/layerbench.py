"""Throughput of layer-list models at sizes that resemble real layers, beside the K-quant decoder at equal size.

    python bench.py --workload ramilorn [--sizes base,small,large] [--no-kernels]

Random weights.  Equal size: the K-quant model has the same width, heads, layers and vocabulary and a dense feed-forward as
wide as the experts a token uses together (top * ff).  Decode steps are timed with CUDA events over self-feeding steps
(captured graph, everything resident), prompts over the chunk path; every step streams far more weight bytes than the L2
holds.  Kernels are timed as a CUDA graph of launches over operand copies rotated past the L2.  Fractions are of the
measured copy bandwidth and of the sustained bf16 rate.
"""
from __future__ import annotations

import importlib
import json

import numpy as np

L2_BYTES = 126 << 20
SIZES = {
    "base": dict(width=2560, heads=32, kv_heads=8, dim=128, vdim=128, experts=64, top=8, ff=1216, groups=8, keep=4, n_layers=8, vocab=151936),
    "small": dict(width=1024, heads=16, kv_heads=4, dim=128, vdim=128, experts=32, top=4, ff=768, groups=4, keep=3, n_layers=16, vocab=65536),
    "large": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, experts=64, top=8, ff=1536, groups=8, keep=4, n_layers=4, vocab=131072),
}


def _mod(jb, name):
    return importlib.import_module(jb.__name__ + "." + name)


def random_model(jb, s, dev, seed=7):
    """(LayeredWeights with random tensors drawn on the GPU, its configuration); every second layer reads the keys of the one before."""
    import torch
    L = _mod(jb, "layered")
    g = torch.Generator(device=dev)
    g.manual_seed(seed)
    dt = torch.bfloat16
    mat = lambda o, i: (torch.randn((o, i), device=dev, generator=g, dtype=dt) / i ** 0.5)
    vec = lambda n, c: c + 0.1 * torch.randn(n, device=dev, generator=g)
    W = s["width"]
    w = L.LayeredWeights.__new__(L.LayeredWeights)
    layers = [L.LayerSpec(L.AttentionSpec(s["heads"], s["kv_heads"], s["dim"], s["vdim"], s["dim"] ** -0.5, -1, 0.1, 4096.0),
                          L.MoeSpec(s["experts"], s["top"], s["ff"], s["groups"], s["keep"])) for _ in range(s["n_layers"])]
    w.cfg = L.LayeredConfig(vocab=s["vocab"], width=W, layers=layers, eps=1e-6, residual_mult=0.6, logit_softcap=40.0)
    w.dtype = "bfloat16"
    norm = lambda f: {f + "_w": vec(W, 1.0), f + "_b": vec(W, 0.0)}
    w.top = {"embed": torch.randn((s["vocab"], W), device=dev, generator=g, dtype=dt), **norm("final")}
    w.layers = []
    for _ in layers:
        E, ff = s["experts"], s["ff"]
        w.layers.append({"w_qkv": mat(s["heads"] * s["dim"] + s["kv_heads"] * (s["dim"] + s["vdim"]), W), "w_o": mat(W, s["heads"] * s["vdim"]),
                         "sink": vec(s["heads"], 0.0), "w_router": mat(E, W), "correction": vec(E, 0.0), "w_gate": mat(E * ff, W), "w_up": mat(E * ff, W),
                         "w_down": mat(E * W, ff), **norm("norm1"), **norm("norm1b"), **norm("norm2"), **norm("norm2b")})
    return w


def step_bytes(s):
    """Weight bytes a decode step must read: attention, router, chosen experts, output matrix (bf16)."""
    W = s["width"]
    attn = (s["heads"] * s["dim"] + s["kv_heads"] * (s["dim"] + s["vdim"])) * W + W * s["heads"] * s["vdim"]
    return 2 * (s["n_layers"] * (attn + s["experts"] * W + 3 * s["top"] * s["ff"] * W) + s["vocab"] * W)


def matmul_params(s):
    W = s["width"]
    return s["n_layers"] * ((s["heads"] * s["dim"] + s["kv_heads"] * (s["dim"] + s["vdim"])) * W + W * s["heads"] * s["vdim"] + s["experts"] * W + 3 * s["top"] * s["ff"] * W)


def time_session(torch, d, s, stream, prompt, steps, repeats=3):
    """(decode ms per step after `prompt`, {prompt length: ms}) of a session opened with the chunk path."""
    out = {}
    with torch.cuda.stream(stream):
        for n in (33, 512, 2048):
            t = prompt[:n]
            for _ in range(2):
                d.reset(); d.prefill(t, 0, stream)
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record(stream)
            for _ in range(repeats):
                d.prefill(t, 0, stream)
            e1.record(stream)
            torch.cuda.synchronize()
            out[n] = e0.elapsed_time(e1) / repeats
        d.reset(); d.prefill(prompt[:512], 0, stream)
        for _ in range(4):
            d.step_device(stream)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record(stream)
        for _ in range(steps):
            d.step_device(stream)
        e1.record(stream)
        torch.cuda.synchronize()
    return e0.elapsed_time(e1) / steps, out


def graph_us(torch, calls, st, iters):
    """Microseconds per call of `iters` rotating calls replayed as one CUDA graph."""
    with torch.cuda.stream(st):
        for c in calls:
            c()
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g, stream=st):
            for i in range(iters):
                calls[i % len(calls)]()
        g.replay()
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record(st)
        g.replay()
        e1.record(st)
        torch.cuda.synchronize()
    return e0.elapsed_time(e1) * 1e3 / iters


def kernel_records(jb, torch, dev, peak_gbs, peak_tf, only=None):
    """The kernels of the layer-list path at the `base` sizes, with their fraction of the roofline."""
    s = SIZES["base"]
    W, QD = s["width"], s["heads"] * s["dim"]
    st = torch.cuda.Stream(device=dev)
    bf = lambda *shape: torch.randn(shape, device=dev, dtype=torch.bfloat16)
    out = {}

    def rotate(make, nbytes):
        return [make() for _ in range(max(2, -(-3 * L2_BYTES // nbytes)))]

    def hbm(name, calls, nbytes, iters=100):
        us = graph_us(torch, calls, st, iters)
        out[name] = {"us": round(us, 2), "bytes": nbytes, "GBps": round(nbytes / us / 1e3, 1), "frac": round(nbytes / us / 1e3 / peak_gbs, 4)}

    def tensor(name, calls, flops, iters=20):
        us = graph_us(torch, calls, st, iters)
        out[name] = {"us": round(us, 2), "TFLOPs": round(flops / us / 1e6, 1), "frac": round(flops / us / 1e6 / peak_tf, 4)}

    def want(group):
        return only is None or group in only
    if want("gemv"):
        for name, M, K in (("gemv_qkv", QD + 2 * s["kv_heads"] * s["dim"], W), ("gemv_wo", W, QD), ("gemv_logits", s["vocab"], W)):
            x, y = bf(K), torch.zeros(M, device=dev)
            ws = rotate(lambda: bf(M, K), 2 * M * K)
            hbm(name, [lambda w=w: jb.dense_matvec(y, w, x, M, K, stream=st) for w in ws], 2 * M * K + 2 * K + 4 * M)
        E, ff, top = s["experts"], s["ff"], s["top"]
        gate, upw, down = bf(E * ff, W), bf(E * ff, W), bf(E * W, ff)
        h, y, act = bf(W), torch.zeros(W, device=dev), bf(top, ff)
        ids, wts = torch.zeros(top, dtype=torch.int32, device=dev), torch.zeros(top, device=dev)
        zs = [torch.randn(E, device=dev) for _ in range(16)]
        hbm("moe_up_and_down_one_token", [lambda z=z: jb.moe_matvec(y, act, ids, wts, gate, upw, down, h, z, top, ff, W, s["groups"], s["keep"], stream=st) for z in zs],
            3 * top * ff * W * 2)
        del gate, upw, down
    if want("attn"):
        scale = s["dim"] ** -0.5
        sink = torch.zeros(s["heads"], device=dev)
        for L in (1024, 4096, 8192, 32768):
            nb = 2 * L * s["kv_heads"] * s["dim"] * 2 + 4 * QD
            q, o = bf(1, QD), bf(1, QD)
            kv = rotate(lambda: (bf(L, s["kv_heads"] * s["dim"]), bf(L, s["kv_heads"] * s["dim"])), nb)
            hbm(f"attn_decode_L{L}", [lambda k=k, v=v: jb.sink_attention(o, q, k, v, s["heads"], s["kv_heads"], s["dim"], s["vdim"], scale, seq_len=L, sink=sink, stream=st)
                                      for k, v in kv], nb)
        for N in (512, 2048):
            q, o, k, v = bf(N, QD), bf(N, QD), bf(N, s["kv_heads"] * s["dim"]), bf(N, s["kv_heads"] * s["dim"])
            tensor(f"attn_prefill_N{N}", [lambda: jb.sink_attention(o, q, k, v, s["heads"], s["kv_heads"], s["dim"], s["vdim"], scale, n_tokens=N, sink=sink, stream=st)],
                   4.0 * QD * N * (N + 1) / 2)
    if want("gemm"):
        for name, M, K in (("gemm_qkv", QD + 2 * s["kv_heads"] * s["dim"], W), ("gemm_wo", W, QD)):
            for N in (33, 512, 2048, 8192):
                x, y = bf(N, K), torch.zeros((N, M), device=dev, dtype=torch.bfloat16)
                ws = rotate(lambda: bf(M, K), 2 * M * K)
                tensor(f"{name}_N{N}", [lambda w=w: jb.dense_matmul(y, w, x, M, N, K, stream=st) for w in ws], 2.0 * M * N * K)
        E, ff, top = s["experts"], s["ff"], s["top"]
        gate, upw, down = bf(E * ff, W), bf(E * ff, W), bf(E * W, ff)
        for T in (512, 2048):
            N = T * top
            cnt = np.bincount(np.random.Generator(np.random.PCG64(1)).integers(0, E, N), minlength=E)
            off = torch.from_numpy(np.concatenate([[0], np.cumsum(cnt)]).astype(np.int32)).to(dev)
            x, a, y = bf(N, W), bf(N, ff), bf(N, W)
            tensor(f"experts_up_T{T}", [lambda: jb.dense_matmul(a, gate, x, ff, N, W, W_up=upw, group_offsets=off, n_groups=E, stream=st)], 4.0 * N * ff * W)
            tensor(f"experts_down_T{T}", [lambda: jb.dense_matmul(y, down, a, W, N, ff, group_offsets=off, n_groups=E, stream=st)], 2.0 * N * ff * W)
    assert jb.device_status(st) == 0
    return out


def run(jb, torch, dev, bench, sizes, steps=64, kernels=True, peaks=None):
    peaks = peaks or {}
    gbs, tf = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops_sustained", 1400.0))
    stream = torch.cuda.Stream(device=dev)
    rec = {}
    for name in sizes:
        s = SIZES[name]
        prompt = np.random.Generator(np.random.PCG64(3)).integers(0, s["vocab"], 2048).astype(np.int32)
        L, D = _mod(jb, "layered"), jb.decoder
        w = random_model(jb, s, dev)
        d = L.LayeredDecoder(w, 2304, D.GRAPH | D.PREFILL)
        l0 = jb.launch_count()
        ms, pf = time_session(torch, d, s, stream, prompt, steps)
        launches = jb.launch_count() - l0
        r = {"sizes": s, "decode": {"ms_per_step": round(ms, 4), "tok_s": round(1e3 / ms, 1), "kernels_per_step": d.kernels_per_step(),
                                    "weight_bytes_per_step": step_bytes(s), "frac_of_hbm": round(step_bytes(s) / ms / 1e6 / gbs, 4)},
             "prefill": {str(n): {"ms": round(t, 3), "tok_s": round(n / t * 1e3), "TFLOPs_matmul": round(2.0 * n * matmul_params(s) / t / 1e9, 1)} for n, t in pf.items()},
             "gpu_launches": int(launches), "device_status": jb.device_status(stream)}
        d.close()
        del d, w
        torch.cuda.empty_cache()
        kc = dict(n_layers=s["n_layers"], hidden=s["width"], n_heads=s["heads"], n_kv_heads=s["kv_heads"], head_dim=s["dim"], ffn=s["top"] * s["ff"], vocab=s["vocab"],
                  rope_theta=1e6, eps=1e-6)
        kw = bench.gen_model_gpu(dev, kc)
        kd = D.Decoder(kc, kw, 2304, D.FUSED | D.GRAPH | D.PREFILL)
        kms, kpf = time_session(torch, kd, s, stream, prompt, steps)
        kb = bench.weight_bytes_per_token(kc)
        r["kquant_equal_size"] = {"decode": {"ms_per_step": round(kms, 4), "tok_s": round(1e3 / kms, 1), "kernels_per_step": kd.kernels_per_step(),
                                             "weight_bytes_per_step": kb, "frac_of_hbm": round(kb / kms / 1e6 / gbs, 4)},
                                  "prefill": {str(n): {"ms": round(t, 3), "tok_s": round(n / t * 1e3)} for n, t in kpf.items()}}
        kd.close()
        del kd, kw
        torch.cuda.empty_cache()
        rec[name] = r
    out = {"metric": "layer_list_decode_tok_s", "unit": "tok/s", "value": rec[sizes[0]]["decode"]["tok_s"], "higher_is_better": True, "data": "synthetic",
           "dtype": "bf16", "n_gpus": 1, "steps": steps, "config": {"model": "Ramilorn layers, random weights", "sizes": list(sizes)}, "models": rec}
    if kernels:
        out["kernels"] = kernel_records(jb, torch, dev, gbs, tf)
        mb, k = _mod(jb, "microbench"), {}
        for name, argv in (("gemv_q4k_triple_norm", ["triple", "--norm", "--K", 2560]), ("gemv_q4k_wo", ["add", "--type", 12, "--M", 2560, "--K", 4096]),
                           ("gemv_pair_swiglu_norm", ["pair", "--swiglu", "--norm"]), ("gemv_q6k_down", ["add", "--type", 14, "--M", 2560, "--K", 9728]),
                           ("gemv_q6k_logits", ["f32", "--type", 14, "--M", 151936, "--K", 2560]), ("attn_L1024", ["attn", "--L", 1024]), ("attn_L4096", ["attn", "--L", 4096]),
                           ("attn_L8192", ["attn", "--L", 8192]), ("attn_L32768", ["attn", "--L", 32768]), ("attn_prefill_N512", ["pattn", "--N", 512]),
                           ("attn_prefill_N2048", ["pattn", "--N", 2048])) + tuple((f"mmq_q4k_4096x2560_N{n}", ["mmq", "--type", 12, "--M", 4096, "--K", 2560, "--N", n, "--iters", 20])
                                                                                  for n in (33, 512, 2048, 8192)):
            r = mb.measure(jb, argv)
            k[name] = {"us": round(r["us_per_launch"], 2), **({"TFLOPs": round(r["TFLOPs"], 1), "frac": round(r["TFLOPs"] / tf, 4)} if "TFLOPs" in r else
                                                              {"GBps": round(r["GBps"], 1), "frac": round(r["GBps"] / gbs, 4)})}
        out["kquant_kernels"] = k
    return out


def main(bench, a):
    import os
    import torch
    from __graft_entry__ import load_package
    jb = load_package()
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    try:
        peaks = json.load(open(os.path.join(bench.ROOT, "MEASURED_PEAKS.json")))
    except Exception:
        peaks = {}
    with bench.ClockSampler(0) as clk:
        line = run(jb, torch, dev, bench, a.sizes.split(","), steps=max(1, min(a.steps, 512)), kernels=not a.no_kernels, peaks=peaks)
    line["clocks"] = clk.summary()
    line["peaks"] = {"hbm_gbs": peaks.get("hbm_gbs", 6650.0), "bf16_tflops_sustained": peaks.get("bf16_tflops_sustained", 1400.0), "source": "measured" if peaks else "fallback"}
    print(json.dumps(line))
