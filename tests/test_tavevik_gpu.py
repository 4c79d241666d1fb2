"""Tavevik on the GPU against the plain float64 restatement in oracle/tavevik.py: every mechanism alone, then whole models through the runner (portions down to
two tokens, decoding, unequal batches, pages and state slots handed from finished requests to new ones) and greedy generation through LLMEngine.
Configurations are small and made here; sizes that one model might happen to make equal or 1 (kv heads == heads, one kv head, value size == key size, rotation
over part of the head or none, a one-tap convolution, equal scales, layers of different head counts, a layer without feed-forward or window) differ between them.
Faults that random weights would hide are made loud: a single key with a large score at a window's edge, among the first tokens or at a page border, scores far
beyond the cap, scores so low that the sink carries the row, one memory written far back."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import candle_vllm_b200 as pkg
from candle_vllm_b200 import seq_ops as ops, synthetic as S
from candle_vllm_b200.engine import LLMEngine, ModelRunner
from candle_vllm_b200.inputs import prepare_step
from candle_vllm_b200.mixers import ChannelDecayDeltaMixer, GatedMlp, PagedAttentionMixer, ParallelSumMixer, TokenShiftLinearAttention
from candle_vllm_b200.tavevik import TavevikConfig, TavevikModel
from oracle import tavevik as O

pytestmark = pytest.mark.gpu
DEV = "cuda"
F64 = torch.float64


def dev(t, dt=torch.float32):
    return t.to(dt).to(DEV).contiguous()


def batch_of(entries, block_size=64):
    return ops.StepBatch.from_host(prepare_step(entries, block_size), DEV)


def close(got, want, tol, what=""):
    got, want = got.detach().cpu().to(F64), want.detach().cpu().to(F64)
    assert bool(torch.isfinite(got).all()), f"{what}: not finite"
    err = float((got - want).abs().max()) / max(float(want.abs().max()), 1e-30)
    assert err < tol, f"{what}: max-err/max = {err:.3e} (tolerance {tol})"


def _portions(total, sizes):
    out, at, i = [], 0, 0
    while at < total:
        n = min(sizes[i % len(sizes)], total - at)
        out.append((at, n)); at += n; i += 1
    return out


# ----------------------------------------------------------------------------------------------------------------------
# row-wise pieces
# ----------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("n", [5, 96, 321, 2048, 4100, 8200])
@pytest.mark.parametrize("scale,biased", [(1.0, False), (0.37, True), (-1.6, True)])
def test_norm_after_a_scaled_sublayer_output(n, scale, biased):
    g = torch.Generator().manual_seed(n)
    T, eps = 7, 1e-3
    x, y = torch.randn(T, n, generator=g) * 3, torch.randn(T, n + 4, generator=g) * 0.2
    yb = torch.randn(n, generator=g) * 0.3 if biased else None
    wp, w = 1 + torch.randn(n, generator=g) * 0.3, 1 + torch.randn(n, generator=g) * 0.3
    new = x.to(F64) + O.rms(y[:, :n].to(F64) * scale + (yb.to(F64) if biased else 0), eps) * wp.to(F64)
    bias = None if yb is None else dev(yb)
    for yd in (dev(y)[:, :n], dev(y[:, :n])):
        for cd in (torch.float32, torch.bfloat16):
            xd, copy = dev(x), torch.zeros(T, n, dtype=cd, device=DEV)
            assert ops.post_norm_add_rms_norm(xd, yd, dev(wp), None, eps, y_bias=bias, y_scale=scale, copy=copy) is None
            close(xd, new, 1e-6, "the stream")
            assert torch.equal(copy, xd.to(cd)), "the copy is the stream in the compute dtype"
        xd = dev(x)
        out = ops.post_norm_add_rms_norm(xd, yd, dev(wp), dev(w), eps, torch.float32, y_bias=bias, y_scale=scale)
        close(xd, new, 1e-6, "the stream beside an opening norm")
        close(out, O.rms(new, eps) * w.to(F64), 2e-6, "opening norm")
        xd, rows = dev(x), torch.tensor([6, 0, 3], dtype=torch.int32, device=DEV)
        out = ops.post_norm_add_rms_norm(xd, yd, dev(wp), dev(w), eps, torch.float32, y_bias=bias, y_scale=scale, row_index=rows)
        assert torch.equal(xd, dev(x))
        close(out, (O.rms(new, eps) * w.to(F64))[[6, 0, 3]], 2e-6, "selected rows")


@pytest.mark.parametrize("ff,limit", [(3, 1.0), (64, 2.5), (257, 7.0), (1024, 0.3)])
def test_clamped_feed_forward(ff, limit):
    g = torch.Generator().manual_seed(ff)
    D, T = 24, 9
    w = {"gate": torch.randn(ff, D, generator=g), "up": torch.randn(ff, D, generator=g), "down": torch.randn(D, ff, generator=g) * ff ** -0.5}
    h = torch.randn(T, D, generator=g)
    mlp = GatedMlp({k: dev(v) for k, v in w.items()}, torch.float32, act="clamped", limit=limit)
    w64, h64 = {k: v.to(F64) for k, v in w.items()}, h.to(F64)
    gate, up = h64 @ w64["gate"].T, h64 @ w64["up"].T
    assert bool((gate > limit).any()) and bool((gate < -limit).any()) and bool((up > limit).any()) and bool((up < -limit).any())
    close(mlp.forward(dev(h)), O.dense_mlp(h64, w64, limit), 1e-5, "feed-forward")
    z = torch.cat([gate, up], 1).float()
    for dt, tol in ((torch.float32, 1e-6), (torch.bfloat16, 5e-3)):
        close(ops.glu_packed(dev(z), "clamped", dt, limit), O.clamped_glu(gate.float().to(F64), up.float().to(F64), limit), tol, "activation")
        close(ops.glu_packed(dev(torch.cat([z, z[:, :3]], 1))[:, :2 * ff], "clamped", dt, limit), O.clamped_glu(gate.float().to(F64), up.float().to(F64), limit), tol, "strided")


@pytest.mark.parametrize("T", [1, 7, 300])
@pytest.mark.parametrize("H,n,R", [(1, 7, 1), (3, 20, 5), (2, 64, 24), (5, 103, 33)])
def test_low_rank_maps(T, H, n, R):
    g = torch.Generator().manual_seed(n)
    N = H * n
    y, w, b, lr = torch.randn(T, R + 3, generator=g), torch.randn(N, R, generator=g), torch.randn(N, generator=g) * 3, torch.randn(H, generator=g)
    b[0], b[1] = -25.0, 12.0                     # a decay that keeps everything, one that kills at once
    y64, w64 = y[:, :R].to(F64), w.to(F64)
    for tanh in (False, True):
        z = (torch.tanh(y64) if tanh else y64) @ w64.T + b.to(F64)
        call = lambda form, **k: ops.low_rank_map(dev(y)[:, :R], dev(w), dev(b), form, in_tanh=tanh, **k).cpu().to(F64)
        close(call("plain"), z, 1e-6, "plain")
        assert float((call("double_exp") - O.double_exponential_decay(z)).abs().max()) < 5e-6
        want = torch.exp(-torch.exp(lr.to(F64)).repeat_interleave(n) * O.softplus(z))
        got = call("softplus_exp", log_rate=dev(lr))
        assert float((got - want).abs().max()) < 5e-6
        near = want > 0.999                      # decays next to one, what a long memory depends on: right to the last place
        assert bool(near.any()) and float((got - want).abs()[near].max()) < 1.3e-7
    assert float((ops.low_rank_map(dev(y)[:, :R], dev(w), None, "double_exp").cpu().to(F64) - O.double_exponential_decay(y64 @ w64.T)).abs().max()) < 5e-6


@pytest.mark.parametrize("D", [5, 48, 130, 1028])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_token_shift_in_unequal_batches(D, dtype):
    g = torch.Generator().manual_seed(D)
    lens, M = [23, 1, 40, 9, 300], 5
    xs, mu = [torch.randn(n, D, generator=g) for n in lens], torch.rand(M, D, generator=g) * 1.4 - 0.2
    want = [torch.stack([O.shift_mix(x.to(F64), m.to(F64)) for m in mu]) for x in xs]
    plans = [[5, 2, 1, 15], [1], [2, 1, 37], [9], [290, 1, 9]]
    state = torch.full((6, D), 1e9, device=DEV)                       # what a slot held before is not read
    slots, fed, pi, got = [4, 0, 2, 5, 1], [0] * 5, [0] * 5, [[] for _ in lens]
    while any(f < n for f, n in zip(fed, lens)):
        live = [i for i in range(5) if fed[i] < lens[i]]
        take = [min(plans[i][pi[i]], lens[i] - fed[i]) for i in live]
        b = batch_of([dict(tokens=[0] * n, start=fed[i], block_table=list(range(5)), state_slot=slots[i], want=[]) for i, n in zip(live, take)])
        x = torch.cat([xs[i][fed[i]:fed[i] + n] for i, n in zip(live, take)])
        wide = dev(torch.cat([x, x[:, :4]], 1))[:, :D] if len(live) % 2 else dev(x)
        out = torch.full((M, sum(take) + 3, D), 7.0, dtype=dtype, device=DEV)
        ops.token_shift_mix(wide, dev(mu), state, b, out)
        assert bool((out[:, sum(take):] == 7.0).all()), "padding rows stay as they are"
        at = 0
        for i, n in zip(live, take):
            got[i].append(out[:, at:at + n]); at += n; fed[i] += n; pi[i] += 1
    for i in range(5):
        close(torch.cat(got[i], 1), want[i], 1e-6 if dtype == torch.float32 else 5e-3, f"sequence {i}")
        assert torch.equal(state[slots[i]].cpu(), xs[i][-1])


@pytest.mark.parametrize("C,K", [(8, 1), (36, 2), (33, 3), (512, 4), (20, 6), (7, 8), (12, 11)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_convolution_over_steps_of_many_rows(C, K, dtype):
    g = torch.Generator().manual_seed(C)
    lens, plans = [700, 3, 41, 290, 1], [[300, 1, 399], [2, 1], [5, 36], [1, 289], [1]]
    xs, taps = [torch.randn(n, C, generator=g) for n in lens], torch.randn(C, K, generator=g)
    want = [O.silu(O.short_conv(x.to(F64), taps.to(F64))) for x in xs]
    ib, ob = torch.randn(C, generator=g), torch.randn(C, generator=g)
    want2 = [O.short_conv(x.to(F64) + ib.to(F64), taps.to(F64)) + ob.to(F64) + x.to(F64) + ib.to(F64) for x in xs]
    for plain in (True, False):
        state, fed, pi, got = torch.full((6, max(K - 1, 1), C), 1e9, device=DEV), [0] * 5, [0] * 5, [[] for _ in lens]
        while any(f < n for f, n in zip(fed, lens)):
            live = [i for i in range(5) if fed[i] < lens[i]]
            take = [min(plans[i][pi[i]], lens[i] - fed[i]) for i in live]
            b = batch_of([dict(tokens=[0] * n, start=fed[i], block_table=list(range(11)), state_slot=5 - i, want=[]) for i, n in zip(live, take)])
            x = dev(torch.cat([torch.cat([xs[i][fed[i]:fed[i] + n]] * 2, 1) for i, n in zip(live, take)]))[:, :C]
            y = ops.causal_conv(x, dev(taps), state, b, out_dtype=dtype, act="silu") if plain else ops.causal_conv(x, dev(taps), state, b, dtype, dev(ib), dev(ob), add_input=True)
            at = 0
            for i, n in zip(live, take):
                got[i].append(y[at:at + n]); at += n; fed[i] += n; pi[i] += 1
        for i in range(5):
            close(torch.cat(got[i]), (want if plain else want2)[i], 2e-6 if dtype == torch.float32 else 5e-3, f"sequence {i}")


# ----------------------------------------------------------------------------------------------------------------------
# the two recurrences
# ----------------------------------------------------------------------------------------------------------------------
def _decays(T, H, dk, g, kind):
    if kind == "mild":
        return torch.exp(-torch.exp(torch.randn(T, H, dk, generator=g) - 4))
    if kind == "wide":
        return torch.exp(-torch.exp(torch.randn(T, H, dk, generator=g) * 3 - 2))
    a = torch.exp(-torch.rand(T, H, dk, generator=g) * 30)                     # strong decays with exact zeros and ones among them
    r = torch.rand(T, H, dk, generator=g)
    a[r < 0.1], a[r > 0.8] = 0.0, 1.0
    return a


SHAPES = [(1, 5, 3), (3, 20, 12), (2, 32, 40), (2, 64, 64), (1, 100, 33), (2, 128, 70), (1, 160, 20)]
LENS = [200, 1, 67, 129, 3]
PLANS = [[64, 1, 2, 70, 1, 62], [1], [2, 65], [128, 1], [1, 2]]


def walk(lens, plans, nslots, step):
    """advance unequal sequences together by their plans; step(live, take, fed, slots) -> rows; returns the rows per sequence"""
    slots = list(range(nslots - 1, nslots - 1 - len(lens), -1))
    fed, pi, got = [0] * len(lens), [0] * len(lens), [[] for _ in lens]
    while any(f < n for f, n in zip(fed, lens)):
        live = [i for i in range(len(lens)) if fed[i] < lens[i]]
        take = [min(plans[i][pi[i] % len(plans[i])], lens[i] - fed[i]) for i in live]
        b = batch_of([dict(tokens=[0] * n, start=fed[i], block_table=list(range(8)), state_slot=slots[i], want=[]) for i, n in zip(live, take)])
        rows = step(b, live, take, fed)
        at = 0
        for i, n in zip(live, take):
            got[i].append(rows[at:at + n].clone()); at += n; fed[i] += n; pi[i] += 1
    return [torch.cat(r) for r in got], slots


@pytest.mark.parametrize("H,dk,dv", SHAPES)
@pytest.mark.parametrize("kind", ["mild", "wide", "harsh"])
def test_bonus_recurrence_on_all_kernels_in_unequal_batches(H, dk, dv, kind):
    g = torch.Generator().manual_seed(dk)
    seqs = [dict(r=torch.randn(n, H, dk, generator=g), k=torch.randn(n, H, dk, generator=g) * dk ** -0.5, v=torch.randn(n, H, dv, generator=g), w=_decays(n, H, dk, g, kind)) for n in LENS]
    u = torch.randn(H, dk, generator=g) * 2
    want = [O.bonus_recurrence(*(s[x].to(F64) for x in "rkvw"), u.to(F64)) for s in seqs]
    for plans, kernel in ((PLANS, None), ([[n] for n in LENS], "token"), ([[n] for n in LENS], "chunked"), ([[1]] * 5, "step"), ([[90, 1, 3, 64]] * 5, "chunked")):
        state = torch.full((7, H, dv, dk), 1e6, device=DEV)

        def step(b, live, take, fed):
            cat = lambda x: torch.cat([seqs[i][x][fed[i]:fed[i] + n].reshape(n, -1) for i, n in zip(live, take)])
            if kernel == "token":                # operands as columns of one matrix
                p = dev(torch.cat([cat("v"), cat("r"), cat("k")], 1))
                return ops.linear_attention_channel(p, H * dv, H * (dv + dk), 0, dev(cat("w")), state, b, H, dk, dv, kernel=kernel, bonus=dev(u))
            n = max(dk, dv) * H                  # or as slabs of one with a common pitch
            T, Tp = sum(take), sum(take) + 2
            p = torch.zeros(3 * Tp, n)
            p[:T, :H * dk], p[Tp:Tp + T, :H * dk], p[2 * Tp:2 * Tp + T, :H * dv] = cat("r"), cat("k"), cat("v")
            return ops.linear_attention_channel(dev(p), 0, Tp * n, 2 * Tp * n, dev(cat("w")), state, b, H, dk, dv, kernel=kernel, bonus=dev(u), rows=T)
        got, slots = walk(LENS, plans, 7, step)
        for i in range(len(LENS)):
            close(got[i].view(-1, H, dv), want[i], 2e-5, f"{kernel} sequence {i}")
        assert bool((state[[s for s in range(7) if s not in slots]] == 1e6).all()), "slots of no entry stay as they are"


def test_the_output_is_read_before_decay_and_write():
    """one key, one value: the token that writes sees them with the bonus weight alone, the next one undecayed, the one after that decayed once"""
    H, dk, dv, T = 1, 4, 4, 5
    r, k, v, w = torch.ones(T, H, dk), torch.zeros(T, H, dk), torch.zeros(T, H, dv), torch.full((T, H, dk), 0.5)
    k[1], v[1] = 1.0, torch.tensor([1.0, 2.0, 3.0, 4.0])
    u = torch.full((H, dk), -3.0)
    want = torch.tensor([0.0, -12.0, 4.0, 2.0, 1.0])[:, None] * v[1]
    assert torch.allclose(O.bonus_recurrence(*(x.to(F64) for x in (r, k, v, w, u))).view(T, dv), want.to(F64))
    for kernel in ("token", "chunked"):
        state = torch.zeros(1, H, dv, dk, device=DEV)
        b = batch_of([dict(tokens=[0] * T, start=0, block_table=[0], state_slot=0, want=[])])
        p = dev(torch.cat([r.view(T, -1), k.view(T, -1), v.view(T, -1)], 1))
        close(ops.linear_attention_channel(p, 0, 4, 8, dev(w.view(T, -1)), state, b, H, dk, dv, kernel=kernel, bonus=dev(u)), want, 1e-6, kernel)


DELTA = [(1, 1, 5, 3), (4, 2, 20, 12), (2, 2, 32, 40), (3, 1, 64, 64), (2, 1, 100, 33), (2, 1, 128, 70), (1, 1, 160, 20)]


@pytest.mark.parametrize("H,G,dk,dv", DELTA)
@pytest.mark.parametrize("kind", ["mild", "wide", "harsh"])
def test_delta_rule_on_all_kernels_in_unequal_batches(H, G, dk, dv, kind):
    g = torch.Generator().manual_seed(dk + H)
    seqs = []
    for n in LENS:
        k = torch.randn(n, G, dk, generator=g)
        if kind == "mild":                       # keys that nearly repeat: the triangular system is far from the identity
            k = torch.randn(1, G, dk, generator=g) + 0.3 * k
        seqs.append(dict(q=torch.randn(n, G, dk, generator=g), k=k, v=torch.randn(n, H, dv, generator=g), b=torch.randn(n, H, generator=g) * 2 + (2 if kind == "mild" else 0),
                         g=_decays(n, H, dk, g, kind)))
    rep = H // G
    want = [O.delta_recurrence((O.unit(s["q"].to(F64)) * dk ** -0.5).repeat_interleave(rep, 1), O.unit(s["k"].to(F64)).repeat_interleave(rep, 1), s["v"].to(F64),
                               torch.sigmoid(s["b"].to(F64)), s["g"].to(F64)) for s in seqs]
    runs = [(PLANS, None), ([[n] for n in LENS], "token"), ([[1]] * 5, "step")]
    if dk <= 128:
        runs += [([[n] for n in LENS], "chunked"), ([[90, 1, 3, 64]] * 5, "chunked")]
    for plans, kernel in runs:
        state = torch.full((7, H, dv, dk), 1e6, device=DEV)

        def step(b, live, take, fed):
            cat = lambda x: torch.cat([seqs[i][x][fed[i]:fed[i] + n].reshape(n, -1) for i, n in zip(live, take)])
            proj = dev(torch.cat([cat("b") * 0 + 9, cat("b")], 1))
            return ops.gated_delta_rule_channel(dev(torch.cat([cat("q"), cat("k"), cat("v")], 1)), proj, H, dev(cat("g")), state, b, H, G, dk, dv, kernel=kernel)
        got, slots = walk(LENS, plans, 7, step)
        for i in range(len(LENS)):
            close(got[i].view(-1, H, dv), want[i], 4e-5, f"{kernel} sequence {i}")
        assert bool((state[[s for s in range(7) if s not in slots]] == 1e6).all()), "slots of no entry stay as they are"


@pytest.mark.parametrize("kernel", ["token", "chunked"])
def test_a_memory_written_far_back(kernel):
    """One key and value 2000 tokens back: found again where the decays are slow, gone from the key rows where one decay in between was fast, and (delta rule)
    replaced where its key was written again"""
    H, dk, dv, T = 1, 32, 16, 2100
    g = torch.Generator().manual_seed(3)
    k = torch.zeros(T, H, dk); q = torch.zeros(T, H, dk); v = torch.zeros(T, H, dv)
    k[10, 0, :4] = 1.0; v[10] = torch.randn(dv, generator=g) * 3
    k[11:, :, 8:] = torch.randn(T - 11, H, dk - 8, generator=g) * 0.05; v[11:] = torch.randn(T - 11, H, dv, generator=g) * 0.1
    q[-3:, 0, :4] = torch.tensor([[1.0, 1, 0, 0], [0, 0, 1, 1], [1, 1, 1, 1]])
    w = torch.full((T, H, dk), 0.9997)
    w[1000, 0, 2:4] = 1e-9                       # rows 2 and 3 forget
    b = batch_of([dict(tokens=[0] * T, start=0, block_table=list(range(40)), state_slot=0, want=[])])
    u = torch.zeros(H, dk)
    want = O.bonus_recurrence(*(x.to(F64) for x in (q, k, v, w, u)))
    p = dev(torch.cat([x.view(T, -1) for x in (q, k, v)], 1))
    got = ops.linear_attention_channel(p, 0, dk, 2 * dk, dev(w.view(T, -1)), torch.zeros(1, H, dv, dk, device=DEV), b, H, dk, dv, kernel=kernel, bonus=dev(u)).cpu()
    close(got.view(T, H, dv)[-3:], want[-3:], 6e-5, "last rows")           # two thousand equal factors round the same way
    assert float(want[-3].abs().max()) > 1.0 and float(want[-2].abs().max()) < 1e-3
    beta = torch.zeros(T, H) + 30.0              # sigmoid -> 1
    k[1500] = 0; k[1500, 0, :4] = 2.0; v[1500] = 5.0
    wd = w.clone(); wd[1000] = 0.9997
    for rewrite in (False, True):
        bb = beta.clone()
        if not rewrite:
            bb[1500] = -60.0                     # sigmoid -> 0: nothing is written
        want = O.delta_recurrence(O.unit(q.to(F64)) * dk ** -0.5, O.unit(k.to(F64)), v.to(F64), torch.sigmoid(bb.to(F64)), wd.to(F64))
        got = ops.gated_delta_rule_channel(p_cat(q, k, v), dev(bb), 0, dev(wd.view(T, -1)), torch.zeros(1, H, dv, dk, device=DEV), b, H, 1, dk, dv, kernel=kernel).cpu()
        close(got.view(T, H, dv)[-1], want[-1], 6e-5, f"rewritten {rewrite}")
        assert float((want[-1] / want[-1].mean()).std()) < 0.2 if rewrite else float((want[-1] / want[-1].mean()).std()) > 0.2


def p_cat(q, k, v):
    return dev(torch.cat([x.view(x.shape[0], -1) for x in (q, k, v)], 1))


# ----------------------------------------------------------------------------------------------------------------------
# attention
# ----------------------------------------------------------------------------------------------------------------------
TABLE = [7, 2, 9, 0, 5, 11, 3, 8]


def left_case(H, G, dk, dv, window, keep, rot, cap, sink, gate, bias, T, seed=0, D=40, scale=None):
    """(layer's left config, tensors, input rows, oracle's [T, D])"""
    L = (S.tavevik_shift_layer(H, G, dk, dv, 1, 8, window, keep, rot, 700.0, scale, cap) if gate else
         S.tavevik_delta_layer(H, G, dk, dv, 1, 1, 8, 8, 2, window, rot, 700.0, scale))
    m = L["mixer"]["left"]
    if not gate and window and keep:
        m["mask"]["keep_first"] = keep
    if not gate and cap:
        m["softcap"] = cap
    w = {k[12:]: v for k, v in S.tavevik_weights(S.tavevik_config(D, 9, [L]), seed).items() if k.startswith("l0.mix.left.")}
    if not sink:
        w.pop("sink", None)
    elif "sink" not in w:
        w["sink"] = torch.randn(H, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16)
    if not bias:
        w = {k: v for k, v in w.items() if not k.endswith(".b")}
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(seed + 5)).to(torch.bfloat16).float()
    return m, w, h


def left_mixer(m, w, dtype, **kw):
    mask = m.get("mask") or {}
    return PagedAttentionMixer({k: v.to(DEV) for k, v in w.items()}, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], 1e-5, dtype, rot=m.get("rot"),
                               window=mask.get("size", 0), keep_first=mask.get("keep_first", 0), softcap=m.get("softcap", 0.0), gate="element", head_norm="before", max_pos=64, **kw)


def oracle_left(m, w, h):
    return O.attention_part(h.to(F64), {k: v.to(F64) for k, v in w.items()}, m, 1e-5)


def run_left(mix, h, sizes, dtype, bs=64, table=TABLE, pitch=0):
    """one sequence in portions -> the output projection of what `attend` leaves in a slice of a wider buffer"""
    G, dk, dv = mix.cache_shape()
    cache = (torch.full((12, bs, G, dk), float("nan"), dtype=dtype, device=DEV), torch.full((12, bs, G, dv), float("nan"), dtype=dtype, device=DEV))
    out = []
    for at, n in _portions(h.shape[0], sizes):
        b = batch_of([dict(tokens=[0] * n, start=at, block_table=table, state_slot=0, want=[])], bs)
        z = torch.full((n, mix.H * dv + pitch), 3.0, dtype=dtype, device=DEV)
        mix.attend(dev(h[at:at + n], dtype), b, cache, out=z[:, :mix.H * dv])
        assert bool((z[:, mix.H * dv:] == 3.0).all())
        y = ops.linear(z[:, :mix.H * dv].contiguous(), mix.w_o)
        out.append(y if mix.out_bias is None else y + mix.out_bias)
    return torch.cat(out)


#       H  G  dk  dv  window keep rot cap   sink  gate  bias
LEFT = [(6, 2, 14, 10, 37, 5, 8, 12.0, False, True, False), (4, 4, 16, 24, 70, 0, 0, 0.0, True, False, True), (3, 1, 9, 6, 0, 0, 4, 3.0, False, True, False),
        (5, 1, 20, 33, 1, 1, 20, 0.0, True, False, True), (2, 2, 40, 40, 64, 70, 6, 0.0, True, True, False), (8, 2, 12, 8, 100, 3, 12, 0.5, True, False, False)]


@pytest.mark.parametrize("case", LEFT)
@pytest.mark.parametrize("sizes", [[230], [2], [61, 1, 1, 2, 70, 3]])
def test_attention_f32(case, sizes):
    m, w, h = left_case(*case, T=230)
    mix = left_mixer(m, w, torch.float32)
    close(run_left(mix, h, sizes, torch.float32, pitch=3), oracle_left(m, w, h), 3e-5, f"portions {sizes}")


WIDE = [(8, 1, 64, 128, 90, 7, 64, 20.0, False, True, False), (6, 2, 64, 64, 130, 0, 16, 0.0, True, False, True), (4, 2, 128, 128, 100, 70, 128, 8.0, True, True, False),
        (4, 1, 128, 40, 0, 0, 32, 0.0, True, False, True), (20, 1, 24, 72, 65, 3, 24, 5.0, False, True, False), (34, 2, 8, 8, 64, 64, 4, 0.0, True, True, False),
        (3, 3, 72, 120, 200, 130, 10, 0.0, False, False, True), (4, 2, 96, 16, 33, 1, 0, 2.0, False, True, False)]


@pytest.mark.parametrize("case", WIDE)
def test_attention_on_the_tensor_core_kernels(case):
    m, w, h = left_case(*case, T=260)
    want = oracle_left(m, w, h)
    mix = left_mixer(m, w, torch.bfloat16)
    assert mix.selected_tc
    ref = None
    for sizes, pitch in (([260], 0), ([260], 1), ([1], 2), ([3, 1, 2, 7], 0), ([90, 8, 1, 2], 5)):
        got = run_left(mix, h, sizes, torch.bfloat16, pitch=pitch)
        close(got, want, 3e-2, f"portions {sizes}")
        ref = got if ref is None else ref
        close(got, ref, 2e-2, f"portions {sizes} against the whole prompt")
    # the row kernel with the visible keys in one or several runs
    real = ops.paged_attention_selected
    try:
        for splits in (1, 2, 5):
            ops.paged_attention_selected = lambda *a, **k: real(*a, **{**k, "splits": splits})
            close(run_left(mix, h, [100, 160], torch.bfloat16), ref, 2e-2, f"{splits} runs")
    finally:
        ops.paged_attention_selected = real
    # f32 queries on the kernel in f32 arithmetic over the same 16-bit cache
    mix.selected_tc = False
    close(run_left(mix, h, [260], torch.bfloat16), ref, 2e-2, "plain kernel")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window,keep", [(50, 6), (64, 64), (100, 1), (20, 0), (0, 0)])
def test_one_loud_key_at_the_edges_of_window_kept_tokens_and_pages(dtype, window, keep):
    """Every key is orthogonal to every query except one; its value is the only large one.  Rows that see it return it, rows that do not return next to nothing."""
    H, G, dk, dv, D, T = 4, 2, 16, 24, 24, 210
    m, w, _ = left_case(H, G, dk, dv, window, keep, 0, 0.0, False, False, False, T, D=D, scale=1.0)
    w = {k: torch.zeros_like(v) for k, v in w.items()}
    w["q"].view(H, dk, D)[:, 0, 0] = 1.0                                     # queries point along entry 0
    w["k"].view(G, dk, D)[:, 0, 1], w["k"].view(G, dk, D)[:, 1, 2] = 1.0, 1.0        # keys along entry 1, the loud one along entry 0
    w["v"].view(G, dv, D)[:, :, 1] = 1.0
    w["q.norm"], w["k.norm"] = torch.full((dk,), 3.0).to(torch.bfloat16), torch.full((dk,), 3.0).to(torch.bfloat16)
    w["o"] = torch.eye(D, H * dv).to(torch.bfloat16)
    mix = left_mixer(m, w, dtype)
    for loud in sorted({0, 1, max(keep - 1, 0), keep, keep + 1, 63, 64, 65, 127, 128, 150}):
        h = torch.zeros(T, D)
        h[:, 0], h[:, 2] = 1.0, 1.0
        h[loud, 1], h[loud, 2] = 8.0, 0.0
        sees = torch.tensor([O.sees(i, loud, window, keep) for i in range(T)])
        for sizes in ([T], [1], [64, 1, 1, 40, 2]):
            got = run_left(mix, h, sizes, dtype).float().cpu()[:, 0]
            assert bool((got[sees] > 7.9).all()), (loud, sizes, [i for i in range(T) if sees[i] and got[i] < 7.9][:5])
            assert bool((got[~sees].abs() < 1e-3).all()), (loud, sizes, [i for i in range(T) if not sees[i] and abs(got[i]) > 1e-3][:5])
        if window:
            edge = loud + window
            assert edge >= T or (bool(sees[edge - 1]) and bool(sees[edge]) == (loud < keep))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_kept_tokens_keep_their_true_distance(dtype):
    """rotation over the whole head: what a far query sees of a kept token depends on the true distance between them"""
    m, w, h = left_case(2, 1, 16, 16, 30, 4, 16, 0.0, False, True, False, 250)
    w = {k: (v.float() * (3 if k in ("q.norm", "k.norm") else 1)).to(torch.bfloat16) for k, v in w.items()}
    want = oracle_left(m, w, h)
    w64 = {k: v.to(F64) for k, v in w.items()}
    real = O.rotate_halves
    near = lambda x, pos, dims, base: real(x, torch.clamp(pos, max=60), dims, base)       # positions that stop counting give something else
    O.rotate_halves = near
    try:
        wrong = O.attention_part(h.to(F64), w64, m, 1e-5)
    finally:
        O.rotate_halves = real
    assert float((wrong - want)[200:].abs().max() / want.abs().max()) > 0.2
    for sizes in ([250], [1]):
        close(run_left(left_mixer(m, w, dtype), h, sizes, dtype), want, 3e-5 if dtype == torch.float32 else 4e-2, f"portions {sizes}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_scores_far_beyond_the_cap(dtype):
    """scores of +-60 under a cap of 2: weights between e^-2 and e^2, so no key takes a row for itself"""
    m, w, h = left_case(4, 2, 16, 16, 90, 3, 4, 2.0, False, True, False, 150, scale=8.0)
    want = oracle_left(m, w, h)
    plain = dict(m); plain.pop("softcap")
    assert float((oracle_left(plain, w, h) - want).abs().max() / want.abs().max()) > 0.5
    for sizes in ([150], [1], [40, 2, 1]):
        close(run_left(left_mixer(m, w, dtype), h, sizes, dtype), want, 5e-5 if dtype == torch.float32 else 4e-2, f"portions {sizes}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_sink_that_carries_the_row(dtype):
    H = 4
    m, w, h = left_case(H, 2, 16, 16, 40, 0, 4, 0.0, True, False, False, 120)
    w["sink"] = torch.tensor([7.0, -9.0, 4.0, 0.0]).to(torch.bfloat16)
    want = oracle_left(m, w, h)
    bare = {k: v for k, v in w.items() if k != "sink"}
    assert float((oracle_left(m, bare, h) - want).abs().max() / want.abs().max()) > 0.3
    mix = left_mixer(m, w, dtype)
    for sizes in ([120], [1], [30, 2, 1]):
        close(run_left(mix, h, sizes, dtype), want, 3e-5 if dtype == torch.float32 else 4e-2, f"portions {sizes}")
    if dtype == torch.bfloat16:                  # several runs of keys: the sink counts once
        real = ops.paged_attention_selected
        try:
            ops.paged_attention_selected = lambda *a, **k: real(*a, **{**k, "splits": 3})
            close(run_left(mix, h, [1], dtype), want, 4e-2, "three runs")
        finally:
            ops.paged_attention_selected = real


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_entries_of_a_batch_do_not_see_each_other(dtype):
    m, w, _ = left_case(6, 2, 16, 24, 50, 4, 8, 9.0, True, True, False, 1)
    mix = left_mixer(m, w, dtype)
    g = torch.Generator().manual_seed(8)
    lens, starts = [100, 1, 30, 66, 1], [0, 70, 5, 64, 0]
    hs = [torch.randn(s + n, 40, generator=g).to(torch.bfloat16).float() for n, s in zip(lens, starts)]
    G, dk, dv = mix.cache_shape()
    cache = tuple(torch.full((12, 64, G, d), float("nan"), dtype=dtype, device=DEV) for d in (dk, dv))
    tables = [[3, 8], [1, 6], [10], [0, 11, 4], [7]]
    for h, s, t in zip(hs, starts, tables):
        if s:
            mix.attend(dev(h[:s], dtype), batch_of([dict(tokens=[0] * s, start=0, block_table=t, state_slot=0, want=[])]), cache, out=torch.empty(s, 6 * dv, dtype=dtype, device=DEV))
    for pick in ([0, 1, 2, 3, 4], ):
        b = batch_of([dict(tokens=[0] * lens[i], start=starts[i], block_table=tables[i], state_slot=0, want=[]) for i in pick])
        x = torch.cat([hs[i][starts[i]:] for i in pick])
        z = torch.empty(x.shape[0], 6 * dv, dtype=dtype, device=DEV)
        mix.attend(dev(x, dtype), b, cache, out=z)
        y = ops.linear(z, mix.w_o)
        at = 0
        for i in pick:
            close(y[at:at + lens[i]], oracle_left(m, w, hs[i])[starts[i]:], 3e-5 if dtype == torch.float32 else 4e-2, f"entry {i}")
            at += lens[i]


# ----------------------------------------------------------------------------------------------------------------------
# the mixers
# ----------------------------------------------------------------------------------------------------------------------
def mixer_tensors(L, D, seed, ranks):
    cfg = S.tavevik_config(D, 9, [L])
    return {k[7:]: v for k, v in S.tavevik_weights(cfg, seed, ranks).items() if k.startswith("l0.mix.")}


def run_state_mixer(mix, x, sizes, dtype, kernel=None):
    state = tuple(torch.full((3,) + s, 1e4, device=DEV) for s in mix.state_shapes())
    mix.kernel = kernel
    out = []
    for at, n in _portions(x.shape[0], sizes):
        b = batch_of([dict(tokens=[0] * n, start=at, block_table=list(range(8)), state_slot=1, want=[])])
        xs = dev(x[at:at + n])
        out.append(mix.forward(xs if isinstance(mix, TokenShiftLinearAttention) else xs.to(dtype), b, state))
    return torch.cat(out)


@pytest.mark.parametrize("D,H,n,R", [(40, 3, 12, 7), (33, 1, 9, 1), (64, 2, 32, 16), (128, 4, 64, 20)])
@pytest.mark.parametrize("sizes", [[130], [2], [1], [70, 1, 3, 26]])
def test_token_shift_linear_attention_mixer(D, H, n, R, sizes):
    L = S.tavevik_shift_layer(1, 1, 8, 8, H, n)
    w = {k[6:]: v for k, v in mixer_tensors(L, D, n, (R, 1, 1)).items() if k.startswith("right.")}
    x = torch.randn(130, D, generator=torch.Generator().manual_seed(1)) * 1.5
    want = O.time_mix_part(x.to(F64), {k: v.to(F64) for k, v in w.items()}, L["mixer"]["right"], 1e-5)
    for dtype, tol in ((torch.float32, 3e-5), (torch.bfloat16, 4e-2)):
        mix = TokenShiftLinearAttention({k: v.to(DEV) for k, v in w.items()}, H, n, 1e-5, dtype)
        assert mix.grouped == (dtype == torch.bfloat16 and D % 8 == 0 and D >= 64 and H * n >= 64)
        close(run_state_mixer(mix, x, sizes, dtype), want, tol, f"{dtype}")


@pytest.mark.parametrize("D,H,G,dk,dv,taps,ra,rg", [(40, 4, 2, 12, 20, 4, 7, 5), (33, 1, 1, 9, 6, 1, 1, 3), (64, 2, 2, 32, 32, 2, 16, 24), (128, 3, 1, 64, 64, 6, 16, 72)])
@pytest.mark.parametrize("sizes", [[130], [2], [1], [70, 1, 3, 26]])
def test_channel_decay_delta_mixer(D, H, G, dk, dv, taps, ra, rg, sizes):
    L = S.tavevik_delta_layer(1, 1, 8, 8, H, G, dk, dv, taps)
    w = {k[6:]: v for k, v in mixer_tensors(L, D, dk, (1, ra, rg)).items() if k.startswith("right.")}
    h = torch.randn(130, D, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16).float()
    want = O.delta_part(h.to(F64), {k: v.to(F64) for k, v in w.items()}, L["mixer"]["right"], 1e-5)
    for dtype, tol in ((torch.float32, 5e-5), (torch.bfloat16, 4e-2)):
        mix = ChannelDecayDeltaMixer({k: v.to(DEV) for k, v in w.items()}, H, G, dk, dv, taps, 1e-5, dtype)
        close(run_state_mixer(mix, h, sizes, dtype), want, tol, f"{dtype}")


def test_output_gate_on_the_tensor_cores_in_long_steps():
    D, H, G, dk, dv, T = 64, 2, 1, 16, 64, 300
    L = S.tavevik_delta_layer(1, 1, 8, 8, H, G, dk, dv, 4)
    w = {k[6:]: v for k, v in mixer_tensors(L, D, 2, (1, 8, 64)).items() if k.startswith("right.")}
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16).float()
    mix = ChannelDecayDeltaMixer({k: v.to(DEV) for k, v in w.items()}, H, G, dk, dv, 4, 1e-5, torch.bfloat16)
    want = O.delta_part(h.to(F64), {k: v.to(F64) for k, v in w.items()}, L["mixer"]["right"], 1e-5)
    close(run_state_mixer(mix, h, [T], torch.bfloat16), want, 4e-2, "one step")
    close(run_state_mixer(mix, h, [100], torch.bfloat16), want, 4e-2, "three steps")


@pytest.mark.parametrize("kind", ["shift", "delta"])
@pytest.mark.parametrize("ls,rs", [(0.8, 1.7), (1.0, 1.0), (0.0, 0.6), (-0.5, 0.9), (1.3, 0.0)])
def test_scaled_sum_of_two_mixers(kind, ls, rs):
    D, T, eps = 48, 150, 1e-5
    L = (S.tavevik_shift_layer(3, 1, 10, 14, 2, 12, 40, 3, 6, left_scale=ls, right_scale=rs) if kind == "shift" else
         S.tavevik_delta_layer(3, 1, 10, 14, 4, 2, 12, 9, 3, 40, 6, left_scale=ls, right_scale=rs))
    w = mixer_tensors(L, D, 5, (4, 5, 6))
    m = L["mixer"]
    sub = lambda side: {k[len(side):]: v for k, v in w.items() if k.startswith(side)}
    x = torch.randn(T, D, generator=torch.Generator().manual_seed(2)).to(torch.bfloat16).float()
    w64 = lambda side: {k: v.to(F64) for k, v in sub(side).items()}
    want = ls * O.attention_part(x.to(F64), w64("left."), m["left"], eps) + rs * O.RIGHT[L["type"]](x.to(F64), w64("right."), m["right"], eps)
    for dtype, tol in ((torch.float32, 5e-5), (torch.bfloat16, 4e-2)):
        g = {k: v.to(DEV) for k, v in sub("right.").items()}
        f = ParallelSumMixer.right_factor(ls, rs)
        right = TokenShiftLinearAttention(g, 2, 12, eps, dtype, norm_scale=f) if kind == "shift" else ChannelDecayDeltaMixer(g, 4, 2, 12, 9, 3, eps, dtype, norm_scale=f)
        mix = ParallelSumMixer(left_mixer(m["left"], sub("left."), dtype), right, ls)
        kv = tuple(torch.zeros(4, 64, 1, d, dtype=dtype, device=DEV) for d in (10, 14))
        st = tuple(torch.zeros((2,) + s, device=DEV) for s in mix.state_shapes())
        for sizes in ([T], [60, 1, 2, 1]):
            out = []
            for at, n in _portions(T, sizes):
                b = batch_of([dict(tokens=[0] * n, start=at, block_table=[2, 0, 1], state_slot=0, want=[])])
                xs = dev(x[at:at + n])
                y = mix.forward(xs, xs.to(dtype), b, kv, st) * mix.out_scale
                out.append(y if mix.out_bias is None else y + mix.out_bias)
            close(torch.cat(out), want, tol, f"{kind} {dtype} {sizes}")


# ----------------------------------------------------------------------------------------------------------------------
# whole models
# ----------------------------------------------------------------------------------------------------------------------
CONFIGS = {
    # both kinds with nothing equal to anything else, a layer without feed-forward
    "mix": S.tavevik_config(40, 211, [S.tavevik_shift_layer(6, 2, 14, 18, 3, 12, 37, 5, 10, 500.0, ff=56, limit=1.5), S.tavevik_delta_layer(4, 4, 10, 12, 4, 2, 20, 9, 3, 90, 6, 300.0, ff=72),
                                      S.tavevik_delta_layer(2, 1, 24, 10, 3, 3, 7, 16, 5, 20), S.tavevik_shift_layer(3, 3, 8, 30, 2, 24, 100, 70, 8, 900.0, left_scale=1.0,
                                                                                                                   right_scale=1.0, ff=30, limit=7.0)], eps=1e-5),
    # odd sizes, no window, no rotation, no cap, a one-tap convolution, one head, delta rule first
    "odd": S.tavevik_config(33, 57, [S.tavevik_delta_layer(3, 1, 9, 6, 1, 1, 7, 5, 1, rot_dims=4, base=90.0, ff=17), S.tavevik_shift_layer(5, 1, 9, 9, 1, 11, softcap=0.0),
                                     S.tavevik_shift_layer(1, 1, 7, 5, 3, 5, 11, 1, 2, 90.0, left_scale=0.4, right_scale=2.0, ff=11, limit=0.5)], eps=1e-4),
    # sizes of the tensor-core kernels
    "aligned": S.tavevik_config(128, 200, [S.tavevik_shift_layer(4, 1, 64, 128, 2, 64, 90, 9, 64, ff=256), S.tavevik_delta_layer(8, 2, 64, 64, 2, 1, 64, 64, 4, 70, 32, ff=256),
                                           S.tavevik_shift_layer(2, 2, 128, 128, 1, 128, 130, 66, 128, ff=128)]),
}
RANKS = {"mix": (7, 5, 11), "odd": (1, 3, 2), "aligned": (16, 24, 64)}
TOL = 2e-4
_CACHE = {}


def weights_of(name, seed=0):
    return S.tavevik_weights(CONFIGS[name], seed, RANKS[name])


def model_and_oracle(name, dtype, T):
    key = (name, T)
    if key not in _CACHE:
        cfg = CONFIGS[name]
        w = weights_of(name)
        toks = torch.randint(0, cfg["vocab"], (T,), generator=torch.Generator().manual_seed(1)).tolist()
        trace = []
        _CACHE[key] = (w, toks, O.forward(cfg, w, toks, trace), trace)
    w, toks, ref, trace = _CACHE[key]
    return TavevikModel(TavevikConfig.from_dict(CONFIGS[name]), w, dtype=dtype, block_size=64, max_pos=512, device=DEV), toks, ref, trace


def run_schedule(runner, seq_id, toks, sizes):
    runner.admit(seq_id)
    out = []
    for at, n in _portions(len(toks), sizes):
        out.append(runner.execute([dict(seq_id=seq_id, tokens=toks[at:at + n], want=list(range(n)))]))
    runner.release(seq_id)
    return torch.cat(out)


def row_errors(got, want):
    """per position: rms over the vocabulary of the centred difference, relative to the rms of the reference logits"""
    d = got.detach().cpu().to(F64) - want
    d = d - d.mean(-1, keepdim=True)
    return torch.sqrt((d * d).mean(-1)) / torch.sqrt((want * want).mean())


@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_matches_the_oracle(name):
    model, toks, ref, want_trace = model_and_oracle(name, torch.float32, 230)
    runner = ModelRunner(model, 8, 2, 64)
    trace = []
    runner.admit(0)
    got = runner.execute([dict(seq_id=0, tokens=toks, want=list(range(len(toks))))], hidden_trace=trace)
    close(got, ref, TOL, f"{name} logits")
    assert len(trace) == len(want_trace) == len(CONFIGS[name]["layers"])
    for i, (a, b) in enumerate(zip(trace, want_trace)):
        close(a, b, 1e-4, f"{name} stream after layer {i}")
    runner.admit(1)
    close(runner.execute([dict(seq_id=1, tokens=toks, want=[229, 3])]), ref[[229, 3]], TOL, f"{name} wanted rows alone")


@pytest.mark.parametrize("name", list(CONFIGS))
def test_bf16_stays_within_rounding(name):
    model, toks, ref, _ = model_and_oracle(name, torch.bfloat16, 230)
    runner = ModelRunner(model, 8, 2, 64)
    for sizes in ([230], [37, 2, 1, 1, 64], [100, 1, 1, 1, 1]):
        e = row_errors(run_schedule(runner, 0, toks, sizes), ref)
        assert float(e.median()) < 0.04 and float(e.max()) < 0.15, (sizes, float(e.median()), float(e.max()))


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("sizes", [[1], [2], [3, 2, 7], [64, 1, 1, 5], [39, 1, 41, 2, 63], [66, 70]])
def test_portions_and_decoding_match_the_whole_prompt(name, sizes):
    model, toks, ref, _ = model_and_oracle(name, torch.float32, 230)
    runner = ModelRunner(model, 4, 1, 64)
    close(run_schedule(runner, 5, toks, sizes), ref, TOL, f"{name} portions {sizes}")


@pytest.mark.parametrize("name,dtype", [("mix", torch.float32), ("odd", torch.float32), ("aligned", torch.float32), ("aligned", torch.bfloat16)])
def test_unequal_batches_match_each_request_alone(name, dtype):
    """Requests of different lengths advance together, portions of some beside single tokens of others, one left out now and then; the pools of pages and slots are
    smaller than the sum of all requests, so both go from finished requests to later ones."""
    cfg = CONFIGS[name]
    w = weights_of(name)
    model = TavevikModel(TavevikConfig.from_dict(cfg), w, dtype=dtype, block_size=64, max_pos=512, device=DEV)
    g = torch.Generator().manual_seed(9)
    lens = [130, 7, 64, 201, 65, 1, 90]
    seqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in lens]
    runner = ModelRunner(model, 9, 3, 64)
    plans = [[64, 1, 1, 30, 2, 1], [2, 1], [63, 1], [100, 3, 1, 1, 50, 2], [64, 1], [1], [1, 1, 1, 80, 2]]
    waiting, live, got = list(range(len(seqs))), {}, {i: [] for i in range(len(seqs))}
    step = 0
    while waiting or live:
        step += 1
        assert step < 500
        while waiting and runner.state.pool.num_free() > 0 and runner.can_admit(lens[waiting[0]], sum(-(-lens[i] // 64) - len(runner.blocks.tables.get(i, ())) for i in live)):
            i = waiting.pop(0)
            runner.admit(i)
            live[i] = [0, 0]
        entries = []
        for i, (fed, pi) in live.items():
            if i == 3 and step % 4 == 2 and len(live) > 1:
                continue                                              # sits this step out
            n = min(plans[i][pi % len(plans[i])] if pi < len(plans[i]) else 1, lens[i] - fed)
            entries.append(dict(seq_id=i, tokens=seqs[i][fed:fed + n], want=list(range(n))))
        out = runner.execute(entries)
        at = 0
        for e in entries:
            i, n = e["seq_id"], len(e["tokens"])
            got[i].append(out[at:at + n].clone()); at += n
            live[i][0] += n; live[i][1] += 1
        for i in [i for i, (fed, _) in live.items() if fed == lens[i]]:
            runner.release(i); del live[i]
    for i in range(len(seqs)):
        ref = O.forward(cfg, w, seqs[i])
        if dtype == torch.float32:
            close(torch.cat(got[i]), ref, TOL, f"{name} request {i} in a batch")
        else:
            assert float(row_errors(torch.cat(got[i]), ref).max()) < 0.15, i
    runner.blocks.check_invariants()
    assert runner.blocks.num_free_gpu_blocks() == 9 and runner.state.pool.num_free() == 3


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_long_decoding_across_pages_and_windows(dtype):
    model, toks, ref, _ = model_and_oracle("mix", dtype, 300)
    runner = ModelRunner(model, 5, 1, 64)
    runner.admit(0)
    got = [runner.execute([dict(seq_id=0, tokens=toks[:20], want=list(range(20)))])]
    for t in range(20, 300):
        got.append(runner.execute([dict(seq_id=0, tokens=[toks[t]], want=[0])]))
    if dtype == torch.float32:
        close(torch.cat(got), ref, TOL, "280 decoded tokens")
    else:
        assert float(row_errors(torch.cat(got), ref).max()) < 0.15


def test_first_tokens_and_single_token_requests():
    model, toks, ref, _ = model_and_oracle("odd", torch.float32, 230)
    runner = ModelRunner(model, 4, 2, 64)
    for n in (1, 2, 3):
        runner.admit(n)
        close(runner.execute([dict(seq_id=n, tokens=toks[:n], want=list(range(n)))]), ref[:n], TOL, f"first {n} tokens")
        runner.release(n)


@pytest.mark.parametrize("name,dtype", [("mix", torch.float32), ("aligned", torch.bfloat16)])
def test_graph_replay_of_decode_steps_matches_eager(name, dtype):
    cfg = CONFIGS[name]
    w = weights_of(name)
    model = TavevikModel(TavevikConfig.from_dict(cfg), w, dtype=dtype, block_size=64, max_pos=64, device=DEV)      # tables must grow
    g = torch.Generator().manual_seed(3)
    seqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (100, 140)]
    refs = [O.forward(cfg, w, s) for s in seqs]
    runner = ModelRunner(model, 6, 2, 64, decode_graphs=True)
    got = [[], []]
    runner.admit(0); runner.admit(1)
    out = runner.execute([dict(seq_id=0, tokens=seqs[0][:50], want=list(range(50))), dict(seq_id=1, tokens=seqs[1][:61], want=list(range(61)))])
    got[0].append(out[:50]); got[1].append(out[50:])
    fed = [50, 61]
    while fed[0] < 100 or fed[1] < 140:
        live = [i for i in (0, 1) if fed[i] < len(seqs[i])]
        out = runner.execute([dict(seq_id=i, tokens=[seqs[i][fed[i]]], want=[0]) for i in live]).clone()
        for r, i in enumerate(live):
            got[i].append(out[r:r + 1]); fed[i] += 1
    assert 1 in runner._graphs
    for i in (0, 1):
        if dtype == torch.float32:
            close(torch.cat(got[i]), refs[i], TOL, f"graph replay, request {i}")
        else:
            assert float(row_errors(torch.cat(got[i]), refs[i]).max()) < 0.15


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_greedy_generation_through_the_engine(dtype, tmp_path):
    """checkpoint on disk -> registry -> LLMEngine (scheduler, chunked prefill, sampler) against the oracle's greedy continuation"""
    from candle_vllm_b200.safetensors_io import save_file
    cfg = CONFIGS["mix"]
    w = weights_of("mix", 4)
    save_file(w, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    g = torch.Generator().manual_seed(2)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (70, 3, 33, 1, 129)]
    eng = LLMEngine.from_pretrained(str(tmp_path), dtype=dtype, num_blocks=7, max_num_seqs=2, prefill_chunk=48, max_batch_tokens=64, max_model_len=256)
    assert type(eng.model).__name__ == "TavevikModel"
    outs = eng.generate(prompts, pkg.SamplingParams(max_tokens=6))
    assert eng.runner.blocks.num_free_gpu_blocks() == 7 and eng.runner.state.pool.num_free() == 2
    for p, o in zip(prompts, outs):
        assert len(o) == 6
        if dtype == torch.float32:
            assert o == O.greedy(cfg, w, p, 6)
        else:
            assert all(0 <= t < cfg["vocab"] for t in o)


def test_command_line_and_trace_runner(tmp_path):
    """the two programs a user starts, as child processes on a checkpoint on disk"""
    from candle_vllm_b200.safetensors_io import save_file
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = CONFIGS["odd"]
    w = weights_of("odd", 1)
    save_file(w, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    env = dict(os.environ, PYTHONPATH=root)
    r = subprocess.run([sys.executable, "-m", "candle_vllm_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt-ids", "5,6,7,8", "--max-new-tokens", "5"],
                       capture_output=True, text=True, env=env, timeout=600)
    assert r.returncode == 0, r.stderr
    assert json.loads(r.stdout.strip().splitlines()[-1])["output"] == O.greedy(cfg, w, [5, 6, 7, 8], 5)
    a, b = list(range(3, 43)), [9, 8, 7]
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:30], want=[0, 29]), dict(id="b", tokens=b[:1], want=[0])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=a[30:], want=[9]), dict(id="b", tokens=b[1:2], want=[])], end=["a"]),
             dict(step=2, entries=[dict(id="b", tokens=b[2:], want=[0]), dict(id="c", tokens=a[:2], want=[1])], end=["b", "c"])]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, env=env, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(3)]
    ra, rb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    V = cfg["vocab"]
    read = lambda i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, V))
    close(read(0), torch.stack([ra[0], ra[29], rb[0]]), TOL, "step 0")
    close(read(1), ra[39:40], TOL, "step 1")
    close(read(2), torch.stack([rb[2], ra[1]]), TOL, "step 2")
