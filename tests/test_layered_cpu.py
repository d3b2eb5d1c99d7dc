"""Layer-list models without a GPU: configuration and registry, the safetensors reader, the oracle's mechanisms, and that a
wrong mechanism would show in the logits the GPU tests compare."""
import copy
import importlib
import json
import os
import struct

import numpy as np
import pytest

import layered_models as lm
from gpu_util import pkg
from oracle import layered as orc


def sub(name):
    return importlib.import_module(pkg().__name__ + "." + name)


def test_registry_names_the_architectures_and_refuses_others():
    reg = sub("registry")
    assert {"Ramilorn", "Qwen3KQuant"} <= set(reg.ARCHITECTURES)
    assert reg.check_config({"architecture": "Ramilorn"})[1] == "bfloat16"
    assert reg.check_config({"architecture": "Ramilorn"}, "float32")[1] == "float32"
    with pytest.raises(reg.DtypeError):
        reg.check_config({"architecture": "Qwen3KQuant"}, "float32")
    with pytest.raises(reg.ConfigError):
        reg.check_config({"architecture": "Nobody"})


def test_configuration_is_read_layer_by_layer():
    L = sub("layered")
    c = L.LayeredConfig.parse(lm.CONFIGS["mixed"])
    assert [l.mixer.kv_from for l in c.layers] == [-1, -1, 0, -1]
    assert [l.mlp is None for l in c.layers] == [False, True, False, False]
    assert (c.layers[0].mlp.groups, c.layers[0].mlp.keep, c.layers[2].mlp.groups) == (3, 2, 1)
    assert c.layers[1].mixer.q_temp_every == 0 and c.layers[3].mixer.q_temp_every == 1
    assert L.LayeredConfig.parse(lm.CONFIGS["odd"]).logit_softcap == 0
    for path, value in ((("layers", 0, "type"), "recurrent"), (("layers", 0, "mlp", "kind"), "dense")):
        bad = copy.deepcopy(lm.CONFIGS["mixed"])
        d = bad
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(sub("registry").ConfigError):
            L.LayeredConfig.parse(bad)


def test_weights_are_padded_and_checked(tmp_path):
    import torch
    L, st = sub("layered"), sub("safetensors")
    cfg = lm.CONFIGS["odd"]
    w = lm.weights(cfg, 3)
    f = st.SafetensorsFile(os.path.join(lm.save(tmp_path / "m", cfg, w), "model.safetensors"))
    c = L.LayeredConfig.parse(cfg)
    got = L.LayeredWeights(c, f, "float32", "cpu")
    qkv = got.layers[0]["w_qkv"]
    assert qkv.shape == (40 + 20 + 28, 56) and not qkv[:, 50:].any()
    assert np.array_equal(qkv[:, :50].numpy(), np.concatenate([w["l0.mix.q"], w["l0.mix.k"], w["l0.mix.v"]]))
    assert got.layers[2]["w_qkv"].shape == (40, 56)                                   # queries only
    assert np.array_equal(got.layers[0]["w_down"].reshape(9, 50, 24)[4, :, :21].numpy(), w["l0.mlp.e4.down"])
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["mlp"]["expert"]["ff"] = 22
    with pytest.raises(sub("registry").ConfigError):
        L.LayeredWeights(L.LayeredConfig.parse(bad), f, "float32", "cpu")
    assert torch.equal(f["embed"].float(), torch.from_numpy(w["embed"]))


def test_safetensors_refuses_broken_files(tmp_path):
    st = sub("safetensors")
    for n, head in ((1 << 40, b"{}"), (2, b"{}"), (None, json.dumps({"a": {"dtype": "BF16", "shape": [4], "data_offsets": [0, 8]}}).encode()),
                    (None, json.dumps({"a": {"dtype": "F8", "shape": [1], "data_offsets": [0, 1]}}).encode())):
        p = tmp_path / "x.safetensors"
        p.write_bytes(struct.pack("<Q", n if n is not None else len(head)) + head)
        if n == 2:
            assert not list(st.SafetensorsFile(str(p)).keys())
        else:
            with pytest.raises(ValueError):
                st.SafetensorsFile(str(p))


def test_router_groups_rank_by_their_two_best_and_weights_ignore_the_correction():
    z = np.array([[3.0, -3.0, 1.0, 1.0, 0.5, 0.9]])
    corr = np.array([0.0, 0.0, 0.0, 0.0, -0.9, 0.0])
    ids, wt = orc.choose_experts(z, corr, 2, dict(count=3, keep=1))
    assert sorted(ids[0]) == [2, 3]                            # 0.73 + 0.73 beats 0.95 + 0.05
    assert np.allclose(wt, 1 / (1 + np.exp(-1.0)))
    ids, wt = orc.choose_experts(z, corr, 6)
    assert ids[0, -1] == 4 and np.isclose(wt[0, -1], 1 / (1 + np.exp(-0.5)))       # chosen last, weighted by its score


def test_query_temperature_steps_at_every_run():
    t = orc.query_temperature(np.arange(10), 0.5, 4)
    assert np.allclose(t, 1 + 0.5 * np.log([1, 1, 1, 2, 2, 2, 2, 3, 3, 3]))


def test_sink_takes_weight_and_is_not_a_key():
    p = orc.sink_softmax(np.array([0.0, 0.0, -np.inf]), np.log(2.0))
    assert np.allclose(p, [0.25, 0.25, 0.0])
    assert np.allclose(orc.sink_softmax(np.array([-2000.0]), 900.0), 0.0)


def _drop_sink(o, m):
    m.setattr(o, "sink_softmax", lambda s, sink: np.exp(s - s.max(-1, keepdims=True)) / np.exp(s - s.max(-1, keepdims=True)).sum(-1, keepdims=True))


def _late_temperature(o, m):
    f = o.query_temperature
    m.setattr(o, "query_temperature", lambda pos, c, e: f(np.asarray(pos) - 1, c, e))


def _corrected_weights(o, m):
    f = o.choose_experts

    def g(z, corr, *a, **k):
        ids, wt = f(z, corr, *a, **k)
        return ids, wt + corr[ids]
    m.setattr(o, "choose_experts", g)


def _ungrouped(o, m):
    f = o.choose_experts
    m.setattr(o, "choose_experts", lambda z, c, t, groups=None: f(z, c, t))


def _uncorrected(o, m):
    f = o.choose_experts
    m.setattr(o, "choose_experts", lambda z, c, t, groups=None: f(z, None, t, groups))


def _rms_only(o, m):
    m.setattr(o, "layer_norm", lambda x, w, b, eps: x / np.sqrt((x ** 2).mean(-1, keepdims=True) + eps) * w + b)


def _no_cap(o, m):
    m.setattr(o, "softcap", lambda z, cap: z)


def _lost_first_key(o, m):
    f = o.attention

    def g(q, k, v, *a, **kw):
        k = k.copy()
        k[0] = 0
        return f(q, k, v, *a, **kw)
    m.setattr(o, "attention", g)


@pytest.mark.parametrize("mistake", [_drop_sink, _late_temperature, _corrected_weights, _ungrouped, _uncorrected, _rms_only, _no_cap, _lost_first_key])
def test_a_wrong_mechanism_shows_in_the_logits(mistake, monkeypatch):
    """The bounds of the GPU tests (5e-5 in fp32, 0.04 in bf16) catch each of these.  (A common factor on the expert weights
    would not show: the norm behind the experts takes it out.  The router tests compare the weights themselves.)"""
    cfg = lm.CONFIGS["mixed"]
    w = lm.weights(cfg, 11, sharp=2.0)
    tokens = np.random.Generator(np.random.PCG64(5)).integers(0, cfg["vocab"], 40)
    want = orc.forward(cfg, w, tokens)
    mistake(orc, monkeypatch)
    err = lm.logit_error(orc.forward(cfg, w, tokens), want)
    assert err.max() > 0.05, err.max()


def test_trace_replay_orders_rows_and_ends_requests(tmp_path):
    class Fake:
        def __init__(self):
            self.log = []

        def feed(self, rid, tokens, want):
            self.log.append((rid, list(tokens)))
            return np.array([[tokens[k], k] for k in want], np.float32).reshape(len(want), 2)

        def end(self, rid):
            self.log.append(("end", rid))
    e, said = Fake(), []
    lines = [json.dumps(dict(step=0, entries=[dict(id="a", tokens=[5, 6, 7], want=[0, 2])], end=[])),
             json.dumps(dict(step=1, entries=[dict(id="a", tokens=[8], want=[])], end=["a"]))]
    sub("trace").replay(e, lines, str(tmp_path), said.append)
    assert said == ["done 0", "done 1"] and e.log == [("a", [5, 6, 7]), ("a", [8]), ("end", "a")]
    assert np.array_equal(np.fromfile(tmp_path / "0.f32", "<f4"), [5, 0, 7, 2]) and not (tmp_path / "1.f32").exists()


def test_trace_refuses_a_number_format_with_code_3(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(dict(architecture="Qwen3KQuant")))
    assert sub("trace").main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "8"]) == 3
