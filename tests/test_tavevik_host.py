"""Tavevik without a GPU: configuration reading, the registry and build group, the synthetic checkpoints, and properties of the float64 oracle that the GPU tests
rely on."""
import importlib.util
import json
import os

import pytest
import torch

import candle_vllm_b200 as pkg
from candle_vllm_b200 import _lib, registry, synthetic as S
from candle_vllm_b200.mixers import ParallelSumMixer
from candle_vllm_b200.tavevik import TavevikConfig
from oracle import tavevik as O

F64 = torch.float64


def _cfg():
    return S.tavevik_config(24, 37, [S.tavevik_shift_layer(4, 2, 8, 6, 3, 5, window=7, keep_first=2, rot_dims=4, ff=20), S.tavevik_delta_layer(3, 1, 8, 6, 4, 2, 6, 5, 3, window=5, ff=12)])


def test_registered_with_a_build_group_of_its_own(tmp_path):
    assert "Tavevik" in registry.registered()
    (tmp_path / "config.json").write_text(json.dumps(_cfg()))
    group = registry.build_group_of(str(tmp_path))
    assert group == "sliding" and set(_lib.GROUP_SYMBOLS[group]) <= set(_lib.SYMBOLS)
    spec = importlib.util.spec_from_file_location("b200_build", os.path.join(os.path.dirname(_lib.__file__), "build.py"))
    b = importlib.util.module_from_spec(spec); spec.loader.exec_module(b)
    assert all(os.path.exists(os.path.join(b.CSRC, n + ".cu")) for n in b.GROUPS[group])


def test_config_is_read_and_checked():
    cfg = TavevikConfig.from_dict(_cfg())
    assert (cfg.vocab, cfg.width, len(cfg.layers), cfg.eps) == (37, 24, 2, 1e-6)
    d = _cfg(); d["layers"][1]["mlp"] = None; d["layers"][0]["mixer"]["left"].pop("rot"); d["layers"][0]["mixer"]["left"].pop("mask")
    TavevikConfig.from_dict(d)
    for breaker, text in [(lambda d: d["layers"][0].update(type="conv"), "unknown mixer"), (lambda d: d["layers"][0]["mixer"].pop("left_scale"), "lacks"),
                          (lambda d: d["layers"][0]["mixer"]["left"].pop("scale"), "lacks"), (lambda d: d["layers"][1]["mixer"]["right"].pop("conv"), "lacks"),
                          (lambda d: d["layers"][0]["mixer"]["left"]["mask"].pop("size"), "without a window"), (lambda d: d["layers"][0]["mlp"].pop("limit"), "lacks"),
                          (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "feed-forward kind"), (lambda d: d.pop("norm"), "lacks")]:
        d = json.loads(json.dumps(_cfg()))
        breaker(d)
        with pytest.raises(pkg.BackendError, match=text):
            TavevikConfig.from_dict(d)


def test_synthetic_checkpoint_through_the_oracle():
    cfg = _cfg()
    w = S.tavevik_weights(cfg, 0, (5, 3, 4))
    assert w["l0.mix.right.w2"].shape == (15, 5) and w["l1.mix.right.a2"].shape == (24, 3) and w["l1.mix.right.g2"].shape == (20, 4) and w["l0.mix.left.g"].shape == (24, 24)
    assert "l0.mix.left.q.b" not in w and "l1.mix.left.o.b" in w and "l1.mix.left.sink" in w and "head" not in w
    trace = []
    lg = O.forward(cfg, w, list(range(20)), trace)
    assert lg.shape == (20, 37) and len(trace) == 2 and bool(torch.isfinite(lg).all())
    # causal: a later token changes no earlier row
    lg2 = O.forward(cfg, w, list(range(19)) + [5])
    assert float((lg[:19] - lg2[:19]).abs().max()) < 1e-12 and float((lg[19] - lg2[19]).abs().max()) > 1e-3


def test_what_a_query_sees():
    see = lambda i, win, keep: [j for j in range(30) if O.sees(i, j, win, keep)]
    assert see(9, 4, 0) == [6, 7, 8, 9] and see(9, 4, 2) == [0, 1, 6, 7, 8, 9] and see(3, 4, 2) == [0, 1, 2, 3] and see(4, 4, 1) == [0, 1, 2, 3, 4]
    assert see(5, 4, 1) == [0, 2, 3, 4, 5] and see(6, 1, 9) == list(range(7)) and see(12, 1, 9) == list(range(9)) + [12] and see(7, 0, 0) == list(range(8))


def test_softmax_with_a_sink_and_capped_scores():
    s = torch.tensor([-700.0, 2.0, 0.5], dtype=F64)
    assert abs(float(O.softmax_with_sink(s, None).sum()) - 1.0) < 1e-12
    p = O.softmax_with_sink(s, torch.tensor(3.0, dtype=F64))
    e = torch.exp(s)
    assert float((p - e / (e.sum() + torch.exp(torch.tensor(3.0, dtype=F64)))).abs().max()) < 1e-15
    assert float(O.softmax_with_sink(s, torch.tensor(900.0, dtype=F64)).sum()) < 1e-300
    c = O.cap_scores(torch.tensor([1e-6, 1000.0, -1000.0, 5.0], dtype=F64), 5.0)
    assert abs(float(c[0]) - 1e-6) < 1e-15 and float(c[1]) == 5.0 and float(c[2]) == -5.0 and 3.7 < float(c[3]) < 3.9


def test_bonus_recurrence_equals_its_sum_over_decayed_keys():
    """the state form against the explicit double sum: products of the decays strictly between two tokens, the token itself with the bonus"""
    g = torch.Generator().manual_seed(1)
    T, H, dk, dv = 9, 2, 3, 4
    r, k, v = (torch.randn(T, H, n, generator=g, dtype=F64) for n in (dk, dk, dv))
    w, u = O.double_exponential_decay(torch.randn(T, H, dk, generator=g, dtype=F64) * 2), torch.randn(H, dk, generator=g, dtype=F64)
    out = O.bonus_recurrence(r, k, v, w, u)
    for t in range(T):
        want = (r[t] * u * k[t]).sum(-1, keepdim=True) * v[t]
        for j in range(t):
            want = want + (r[t] * k[j] * torch.prod(w[j + 1:t], 0)).sum(-1, keepdim=True) * v[j]
        assert float((out[t] - want).abs().max()) < 1e-12


def test_delta_rule_over_a_chunk_equals_the_triangular_system():
    """the token-by-token rule against the form the chunked kernel solves: (I + diag(beta) strict(M)) U = diag(beta) (V - K_P S0)"""
    g = torch.Generator().manual_seed(2)
    T, dk, dv = 11, 4, 3
    q, k = (O.unit(torch.randn(T, 1, dk, generator=g, dtype=F64)) for _ in range(2))
    v, b, d = torch.randn(T, 1, dv, generator=g, dtype=F64), torch.sigmoid(torch.randn(T, 1, generator=g, dtype=F64)), torch.rand(T, 1, dk, generator=g, dtype=F64)
    out = O.delta_recurrence(q, k, v, b, d)[:, 0]
    n = 4                                            # the chunk starts at token 4; the state before it from the rule itself
    S0 = torch.zeros(dk, dv, dtype=F64)
    for t in range(n):
        S0 = S0 * d[t, 0][:, None]
        S0 = S0 + k[t, 0][:, None] * (b[t] * (v[t, 0] - S0.T @ k[t, 0]))[None, :]
    C = T - n
    P = torch.cumprod(d[n:, 0], 0)
    R = lambda t, s: torch.prod(d[n + s + 1:n + t + 1, 0], 0)
    M = torch.tensor([[float((k[n + t, 0] * R(t, s) * k[n + s, 0]).sum()) if s < t else 0.0 for s in range(C)] for t in range(C)], dtype=F64)
    N = torch.tensor([[float((q[n + t, 0] * R(t, s) * k[n + s, 0]).sum()) if s <= t else 0.0 for s in range(C)] for t in range(C)], dtype=F64)
    B = torch.linalg.solve(torch.eye(C, dtype=F64) + b[n:] * M, torch.diag(b[n:, 0]))
    U = B @ v[n:, 0] - (B @ (P * k[n:, 0])) @ S0
    assert float(((P * q[n:, 0]) @ S0 + N @ U - out[n:]).abs().max()) < 1e-12
    assert float(B.abs().max()) <= 1.0 + 1e-12       # responses of a contraction


def test_shifted_rows_and_clamped_activation():
    h = torch.arange(12, dtype=F64).view(4, 3)
    assert torch.equal(O.previous_rows(h)[0], torch.zeros(3, dtype=F64)) and torch.equal(O.previous_rows(h)[1:], h[:3])
    assert torch.equal(O.shift_mix(h, torch.tensor([0.0, 1.0, 0.5], dtype=F64))[2], torch.tensor([6.0, 4.0, 6.5], dtype=F64))
    y = O.clamped_glu(torch.tensor([9.0, -50.0, 1.0], dtype=F64), torch.tensor([9.0, -9.0, 0.0], dtype=F64), 2.0)
    sg = lambda z: 1 / (1 + torch.exp(-torch.tensor(1.702 * z, dtype=F64)))
    assert abs(float(y[0] - 2 * sg(2.0) * 3)) < 1e-12 and abs(float(y[1])) < 1e-30 and abs(float(y[2] - sg(1.0))) < 1e-12


def test_scales_of_the_two_sides():
    """the factor that enters the right side's norm weight times the scale applied to the sum gives the right scale back, whatever the left one is"""
    for ls, rs in ((1.5, 0.5), (-0.25, 2.0), (0.0, 0.7), (1e-3, 1.0), (2.0, 0.0)):
        out_scale = ls if ls else 1.0
        assert abs(ParallelSumMixer.right_factor(ls, rs) * out_scale - rs) < 1e-12
