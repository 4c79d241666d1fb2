"""Sigalorn without a GPU: configuration reading, the registry and build group, the synthetic checkpoints, and properties of the float64 oracle that the GPU
tests rely on."""
import importlib.util
import json
import os

import pytest
import torch

import candle_vllm_b200 as pkg
from candle_vllm_b200 import _lib, registry, synthetic as S
from candle_vllm_b200.mixers import yarn_rotary_tables
from candle_vllm_b200.sigalorn import SigalornConfig
from oracle import sigalorn as O

F64 = torch.float64


def _cfg():
    return S.sigalorn_config(48, 37, [S.sigalorn_gla_layer(3, 8, 6, tau=4.0, ff=20), S.sigalorn_attention_layer(4, 2, 8, 6, chunk=5, rot_dims=4, ff=12),
                                      S.sigalorn_attention_layer(2, 2, 8, 6, chunk=7, rot_dims=4, kv_from=1)], softcap=11.0)


def test_registered_with_a_build_group_of_its_own(tmp_path):
    assert "Sigalorn" in registry.registered()
    (tmp_path / "config.json").write_text(json.dumps(_cfg()))
    group = registry.build_group_of(str(tmp_path))
    assert group == "talking" and set(_lib.GROUP_SYMBOLS[group]) <= set(_lib.SYMBOLS)
    spec = importlib.util.spec_from_file_location("b200_build", os.path.join(os.path.dirname(_lib.__file__), "build.py"))
    b = importlib.util.module_from_spec(spec); spec.loader.exec_module(b)
    assert all(os.path.exists(os.path.join(b.CSRC, n + ".cu")) for n in b.GROUPS[group])


def test_config_is_read_and_checked():
    cfg = SigalornConfig.from_dict(_cfg())
    assert (cfg.vocab, cfg.width, len(cfg.layers), cfg.softcap, cfg.embedding_scale) == (37, 48, 3, 11.0, 1.0)
    d = _cfg(); d.pop("logit_softcap"); d.pop("embedding"); d["layers"][1]["mlp"] = None
    cfg = SigalornConfig.from_dict(d)
    assert cfg.softcap == 0.0 and cfg.embedding_scale == 1.0
    for breaker, text in [(lambda d: d["layers"][0].update(type="conv"), "unknown mixer"), (lambda d: d["layers"][0]["mixer"].pop("tau"), "lacks"),
                          (lambda d: d["layers"][0]["mixer"].update(tau=0.0), "tau"), (lambda d: d["layers"][1]["mixer"].pop("scale"), "lacks"),
                          (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "feed-forward kind"), (lambda d: d["layers"][2]["mixer"].update(kv_from=0), "earlier attention"),
                          (lambda d: d["layers"][2]["mixer"].update(kv_from=2), "earlier attention"), (lambda d: d["layers"][2]["mixer"].update(vdim=8), "must equal"),
                          (lambda d: d["layers"][2]["mixer"]["rot"].update(base=3.0), "must equal"), (lambda d: d.pop("norm"), "lacks")]:
        d = json.loads(json.dumps(_cfg()))
        breaker(d)
        with pytest.raises(pkg.BackendError, match=text):
            SigalornConfig.from_dict(d)


def test_synthetic_checkpoint_through_the_oracle():
    cfg = _cfg()
    w = S.sigalorn_weights(cfg, 0, rank=5)
    assert w["l0.mix.a1"].shape == (5, 48) and w["l0.mix.a2"].shape == (24, 5) and w["l1.mix.talk"].shape == (4, 4) and "l2.mix.k" not in w and "l2.mlp.up" not in w
    trace = []
    lg = O.forward(cfg, w, list(range(20)), trace)
    assert lg.shape == (20, 37) and len(trace) == 3 and bool(torch.isfinite(lg).all()) and float(lg.abs().max()) < 11.0
    # causal: a later token changes no earlier row
    lg2 = O.forward(cfg, w, list(range(19)) + [5])
    assert float((lg[:19] - lg2[:19]).abs().max()) < 1e-12 and float((lg[19] - lg2[19]).abs().max()) > 1e-3


def test_chunks_are_counted_from_the_start_of_the_sequence():
    seen = [[j for j in range(12) if O.sees(i, j, 5)] for i in range(12)]
    assert seen[4] == [0, 1, 2, 3, 4] and seen[5] == [5] and seen[9] == [5, 6, 7, 8, 9] and seen[11] == [10, 11]
    assert [j for j in range(12) if O.sees(7, j, 0)] == list(range(8))


def test_softmax_with_one_in_the_denominator():
    s = torch.tensor([[-700.0, 2.0, 0.5], [800.0, 799.0, -3.0], [-5.0, -6.0, -7.0]], dtype=F64)
    p = O.softmax_with_one(s)
    plain = torch.exp(s[2]) / (1.0 + torch.exp(s[2]).sum())
    assert float((p[2] - plain).abs().max()) < 1e-15 and float(p[2].sum()) < 0.02
    assert bool(torch.isfinite(p).all()) and abs(float(p[1].sum()) - 1.0) < 1e-12


def test_values_turned_forth_and_back_depend_on_the_distance_only():
    g = torch.Generator().manual_seed(0)
    v = torch.randn(1, 2, 10, generator=g, dtype=F64)
    at = lambda i, j: O.rotate_halves(O.rotate_halves(v, torch.tensor([j]), 10, 300.0), torch.tensor([i]), 10, 300.0, back=True)
    assert float((at(40, 33) - at(7, 0)).abs().max()) < 1e-10 and float((at(5, 5) - v).abs().max()) < 1e-12 and float((at(7, 0) - v).abs().max()) > 0.1
    cos, sin = yarn_rotary_tables(10, 300.0, 50, None, device="cpu")
    got = torch.cat([v[..., :5] * cos[33].to(F64) - v[..., 5:] * sin[33].to(F64), v[..., 5:] * cos[33].to(F64) + v[..., :5] * sin[33].to(F64)], -1)
    assert float((got - O.rotate_halves(v, torch.tensor([33]), 10, 300.0)).abs().max()) < 1e-6


def test_recurrence_equals_the_sum_over_decayed_keys():
    """the state form against the explicit double sum with products of decays, strong ones included"""
    g = torch.Generator().manual_seed(1)
    T, H, dk, dv = 9, 2, 3, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=F64) for n in (dk, dk, dv))
    a = O.decay_per_key(torch.randn(T, H, dk, generator=g, dtype=F64) * 20, 2.0)
    out = O.gated_linear_recurrence(q, k, v, a)
    for t in range(T):
        want = sum((q[t] * k[j] * torch.prod(a[j + 1:t + 1], 0)).sum(-1, keepdim=True) * v[j] for j in range(t + 1))
        assert float((out[t] - want).abs().max()) < 1e-12


def test_xielu_is_continuous_with_slope_one_half_at_zero():
    z = torch.tensor([-1e-6, 0.0, 1e-6, -30.0, 3.0], dtype=F64)
    y = O.xielu(z, 0.3, -0.2)
    assert abs(float(y[0]) + 5e-7) < 1e-11 and float(y[1]) == 0.0 and abs(float(y[2]) - 5e-7) < 1e-11
    sp = lambda a: torch.log1p(torch.exp(torch.tensor(a, dtype=F64)))
    assert abs(float(y[4] - (sp(0.3) * 9 + 1.5))) < 1e-12 and abs(float(y[3] - ((0.5 + sp(-0.2)) * 29 - 15.0))) < 1e-9
