"""Sigalorn on the GPU against the plain float64 restatement in oracle/sigalorn.py: every mechanism alone, then whole models through the runner (portions down
to two tokens, decoding, unequal batches, pages and state slots handed from finished requests to new ones) and greedy generation through LLMEngine.
Configurations are small and made here; sizes that one model might happen to make equal or 1 (kv heads == heads, one kv head, value size == key size, rotation
over part of the head, tau 1, layers of different head counts, a layer without feed-forward or mask) differ between them.  Faults that random weights would
hide are made loud: a single key with a large score far back or at a chunk's edge, scores so low that the one in the softmax denominator carries the row."""
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
from candle_vllm_b200.mixers import ChannelDecayLinearAttention, TalkingAttentionMixer, UngatedMlp, yarn_rotary_tables
from candle_vllm_b200.sigalorn import SigalornConfig, SigalornModel
from oracle import sigalorn as O

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
@pytest.mark.parametrize("n", [5, 96, 321, 1032, 2048, 4100, 8200])
@pytest.mark.parametrize("biased", [False, True])
def test_norm_after_a_sublayer_sum_and_norm_before_the_next(n, biased):
    g = torch.Generator().manual_seed(n)
    T, eps = 7, 1e-3
    x, y = torch.randn(T, n, generator=g) * 3, torch.randn(T, n + 4, generator=g) * 0.2
    yb = torch.randn(n, generator=g) * 0.3 if biased else None
    wp, w = 1 + torch.randn(n, generator=g) * 0.3, 1 + torch.randn(n, generator=g) * 0.3
    tot = y[:, :n].to(F64) + (yb.to(F64) if biased else 0)
    new = x.to(F64) + O.rms(tot, eps) * wp.to(F64)
    bias = None if yb is None else dev(yb)
    for strided in (False, True):
        yd = dev(y)[:, :n] if strided else dev(y[:, :n])
        xd = dev(x)
        out = ops.post_norm_add_rms_norm(xd, yd, dev(wp), dev(w), eps, torch.float32, y_bias=bias)
        close(xd, new, 1e-6, "the stream")
        close(out, O.rms(new, eps) * w.to(F64), 2e-6, "the next sublayer's input")
        xd = dev(x)
        assert ops.post_norm_add_rms_norm(xd, yd, dev(wp), None, eps, y_bias=bias) is None
        close(xd, new, 1e-6, "the sum alone")
        xd, rows = dev(x), torch.tensor([6, 0, 3], dtype=torch.int32, device=DEV)
        out = ops.post_norm_add_rms_norm(xd, yd, dev(wp), dev(w), eps, torch.bfloat16, y_bias=bias, row_index=rows)
        close(xd, x, 1e-9, "selected rows leave the stream alone")
        close(out, (O.rms(new, eps) * w.to(F64))[[6, 0, 3]], 6e-3, "selected rows")


@pytest.mark.parametrize("ff", [3, 64, 1029])
def test_xielu_with_bias_and_two_numbers(ff):
    g = torch.Generator().manual_seed(ff)
    x = torch.randn(9, ff + 5, generator=g) * 3
    x[0, :3] = torch.tensor([0.0, -1e-4, 1e-4])
    x[1, :3] = torch.tensor([-40.0, 40.0, -1e-7])
    b = torch.randn(ff, generator=g)
    b[:3] = 0
    for p, q in ((0.4, -0.9), (-3.0, 2.0), (0.0, 0.0)):
        sp = lambda a: float(np.log1p(np.exp(a)))
        out = ops.xielu(dev(x)[:, :ff], dev(b), sp(p), 0.5 + sp(q), torch.float32)
        want = O.xielu(x[:, :ff].to(F64) + b.to(F64), p, q)
        z = x[:, :ff].to(F64) + b.to(F64)
        err = (out.cpu().to(F64) - want).abs() / (want.abs() + 0.5 * z.abs() + 1e-9)      # the negative branch crosses zero: relative to its terms
        assert float(err.max()) < 1e-5
        mlp = UngatedMlp({"up": dev(torch.randn(8, 6, generator=g)), "up.b": dev(b[:8].new_ones(8)), "down": dev(torch.randn(6, 8, generator=g)), "act": torch.tensor([p, q])},
                         torch.float32, act="xielu")
        h = torch.randn(4, 6, generator=g)
        wd = {"up": mlp.w_in.cpu().to(F64), "up.b": torch.ones(8, dtype=F64), "down": mlp.w_down.cpu().to(F64), "down.b": torch.zeros(6, dtype=F64),
              "act": torch.tensor([p, q], dtype=torch.float32).to(F64)}
        close(mlp.forward(dev(h)), O.dense_mlp(h.to(F64), wd), 1e-5, "feed-forward")
    same = ops.xielu(dev(x[:, :ff]), None, 0.5, 0.7, torch.bfloat16)
    assert same.dtype == torch.bfloat16 and same.shape == (9, ff)


@pytest.mark.parametrize("groups,glen", [(3, 5), (4, 64), (2, 300), (16, 128), (1, 1000), (2, 1030)])
def test_norm_per_group_times_a_silu_gate(groups, glen):
    g = torch.Generator().manual_seed(glen)
    n, T = groups * glen, 11
    o, z, w = torch.randn(T, n + 4, generator=g) * 2, torch.randn(T, n + 8, generator=g) * 3, 1 + torch.randn(n, generator=g) * 0.3
    x = o[:, :n].to(F64).view(T, groups, glen)
    want = (O.rms(x, 1e-3).reshape(T, n) * w.to(F64)) * O.silu(z[:, :n].to(F64))
    for od, zd in ((dev(o)[:, :n], dev(z)[:, :n]), (dev(o[:, :n]), dev(z[:, :n]))):
        close(ops.group_rms_norm_gate(od, dev(w), zd, groups, 1e-3, torch.float32, gate_act="silu"), want, 2e-6, "f32")
        close(ops.group_rms_norm_gate(od, dev(w), zd, groups, 1e-3, torch.bfloat16, gate_act="silu"), want, 6e-3, "bf16")
    close(ops.group_rms_norm_gate(dev(o[:, :n]), None, None, groups, 1e-3, torch.float32), O.rms(x, 1e-3).reshape(T, n), 2e-6, "norm alone")


def test_logit_cap():
    x = torch.randn(5, 77, generator=torch.Generator().manual_seed(0)) * 40
    close(ops.softcap(dev(x), 12.5), 12.5 * torch.tanh(x.to(F64) / 12.5), 1e-6, "cap")


# ----------------------------------------------------------------------------------------------------------------------
# linear attention with a decay per token and key row
# ----------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("N,R,tau", [(7, 1, 1.0), (64, 5, 16.0), (300, 16, 16.0), (513, 33, 0.5)])
def test_low_rank_decay(N, R, tau):
    g = torch.Generator().manual_seed(N)
    T = 19
    y, w, b = torch.randn(T, R + 3, generator=g), torch.randn(N, R, generator=g), torch.randn(N, generator=g) * 4
    b[0], b[1] = -60.0, 40.0                     # a decay that kills at once (tau 1), one that keeps everything
    got = ops.low_rank_decay(dev(y)[:, :R], dev(w), dev(b), tau).cpu().to(F64)
    want = O.decay_per_key(y[:, :R].to(F64) @ w.to(F64).T + b.to(F64), tau)
    assert float(((got - want).abs() / (want + 1e-30)).max()) < 5e-5 and float((got - want).abs().max()) < 1e-6
    close(ops.low_rank_decay(dev(y)[:1, :R], dev(w), None, tau), O.decay_per_key(y[:1, :R].to(F64) @ w.to(F64).T, tau), 1e-6, "one row, no bias")


def _decays(T, H, dk, g, kind):
    if kind == "mild":
        return torch.sigmoid(torch.randn(T, H, dk, generator=g) * 2 + 3) ** (1 / 16)
    if kind == "harsh":                          # down to e^-30 per token, exact zeros and exact ones among them
        a = torch.exp(-30 * torch.rand(T, H, dk, generator=g) ** 4)
        a[torch.rand(T, H, dk, generator=g) < 0.02] = 0.0
        a[torch.rand(T, H, dk, generator=g) < 0.05] = 1.0
        return a
    return torch.sigmoid(torch.randn(T, H, dk, generator=g) * 3)


GLA = [  # H, dk, dv
    (2, 16, 24, ), (3, 5, 7), (1, 40, 70), (4, 64, 64), (2, 130, 20), (1, 128, 128), (5, 33, 16)]


@pytest.mark.parametrize("H,dk,dv", GLA)
@pytest.mark.parametrize("kind", ["mild", "wide", "harsh"])
def test_recurrence_on_all_kernels_in_unequal_batches(H, dk, dv, kind):
    """Three sequences through two state slots that held something else before: whole on the token and chunked kernels, in portions (token and chunked), and token
    by token on the single-row kernel; every row and the final state against the recurrence run token by token in float64."""
    g = torch.Generator().manual_seed(H * 1000 + dk + dv)
    lens = [150, 3, 65]
    q_scale = 0.37
    data = []
    for T in lens:
        q, k, v = torch.randn(T, H, dk, generator=g), torch.randn(T, H, dk, generator=g), torch.randn(T, H, dv, generator=g)
        a = _decays(T, H, dk, g, kind)
        data.append((q, k, v, a, O.gated_linear_recurrence(q.to(F64) * q_scale, k.to(F64), v.to(F64), a.to(F64))))
    pad = 3
    off_k, off_v = H * dk + pad, 2 * H * dk + 2 * pad

    def step(entries, state, kernel):
        """entries: (sequence, first row, rows, slot)"""
        proj = torch.zeros(sum(n for _, _, n, _ in entries), off_v + H * dv + pad)
        alpha = torch.zeros(proj.shape[0], H * dk)
        at = 0
        for s, lo, n, _ in entries:
            q, k, v, a, _ = data[s]
            proj[at:at + n, :H * dk] = q[lo:lo + n].reshape(n, -1)
            proj[at:at + n, off_k:off_k + H * dk] = k[lo:lo + n].reshape(n, -1)
            proj[at:at + n, off_v:off_v + H * dv] = v[lo:lo + n].reshape(n, -1)
            alpha[at:at + n] = a[lo:lo + n].reshape(n, -1)
            at += n
        b = batch_of([dict(tokens=[0] * n, start=lo, block_table=list(range(8)), state_slot=slot, want=[]) for s, lo, n, slot in entries])
        out = ops.linear_attention_channel(dev(proj), 0, off_k, off_v, dev(alpha), state, b, H, dk, dv, q_scale=q_scale, kernel=kernel)
        return out.view(-1, H, dv).split([n for _, _, n, _ in entries])

    tol = 2e-5
    for kernel in ("token", "chunked"):
        state = torch.full((3, H, dv, dk), 9.0, device=DEV)
        outs = step([(0, 0, lens[0], 2), (1, 0, lens[1], 0), (2, 0, lens[2], 1)], state, kernel)
        for s in range(3):
            close(outs[s], data[s][4], tol, f"{kernel} sequence {s}")
        # a second pass of unequal portions over the same slots, in another order: what they hold is another sequence's
        got = {0: [], 2: []}
        outs = step([(2, 0, 2, 2), (0, 0, 70, 1)], state, kernel)
        got[2].append(outs[0]); got[0].append(outs[1])
        outs = step([(0, 70, 67, 1), (2, 2, 1, 2)], state, kernel)
        got[0].append(outs[0]); got[2].append(outs[1])
        outs = step([(2, 3, 62, 2), (0, 137, 13, 1)], state, "token" if kernel == "chunked" else "chunked")
        got[2].append(outs[0]); got[0].append(outs[1])
        for s in (0, 2):
            close(torch.cat(got[s]), data[s][4], tol, f"{kernel} portions of sequence {s}")
    state = torch.full((3, H, dv, dk), -5.0, device=DEV)
    got = [[], []]
    for t in range(lens[2]):
        live = [(2, t, 1, 1)] + ([(1, t, 1, 0)] if t < lens[1] else [])
        outs = step(live, state, "step")
        got[0].append(outs[0])
        if t < lens[1]:
            got[1].append(outs[1])
    close(torch.cat(got[0]), data[2][4], tol, "single rows")
    close(torch.cat(got[1]), data[1][4], tol, "single rows, short sequence")


@pytest.mark.parametrize("kernel", ["token", "chunked"])
def test_a_loud_key_far_back_survives_slow_decay_and_dies_with_a_fast_one(kernel):
    """One loud key at position 5 and queries at the end that ask for its direction alone: with decays of 0.9995 a third of it is left 2000 tokens later, in the
    other half of the key rows one small decay in between has removed it."""
    g = torch.Generator().manual_seed(7)
    T, H, dk, dv = 2050, 1, 32, 16
    q, k, v = torch.zeros(T, H, dk), torch.randn(T, H, dk, generator=g) * 1e-3, torch.randn(T, H, dv, generator=g)
    k[5] = 1.0
    q[-50:] = 1.0
    q[-50::2, :, 16:] = 0.0
    q[-49::2, :, :16] = 0.0
    a = torch.full((T, H, dk), 0.9995)
    a[1000, :, 16:] = 1e-6
    want = O.gated_linear_recurrence(q.to(F64), k.to(F64), v.to(F64), a.to(F64))
    proj = torch.cat([q.view(T, -1), k.view(T, -1), v.view(T, -1)], 1)
    b = batch_of([dict(tokens=[0] * T, start=0, block_table=list(range(33)), state_slot=0, want=[])])
    out = ops.linear_attention_channel(dev(proj), 0, H * dk, 2 * H * dk, dev(a.view(T, -1)), torch.zeros(1, H, dv, dk, device=DEV), b, H, dk, dv, kernel=kernel)
    got = out.view(T, H, dv)[-50:].cpu().to(F64)
    close(got[::2], want[-50:][::2], 1e-4, "still there")
    close(got[1::2], want[-50:][1::2], 1e-4, "gone")
    assert float(want[-50:][::2].abs().mean()) > 5 * float(want[-50:][1::2].abs().mean())


@pytest.mark.parametrize("H,dk,dv,tau,rank", [(3, 16, 24, 16.0, 16), (2, 20, 12, 1.0, 5), (4, 64, 64, 4.0, 32)])
@pytest.mark.parametrize("sizes", [[100], [2], [1], [70, 1, 3, 26]])
def test_gated_linear_attention_mixer(H, dk, dv, tau, rank, sizes):
    g = torch.Generator().manual_seed(dk)
    D, T = 48, 100
    cfg = S.sigalorn_config(D, 10, [S.sigalorn_gla_layer(H, dk, dv, tau=tau)])
    w = {k[7:]: v for k, v in S.sigalorn_weights(cfg, 3, rank=rank).items() if k.startswith("l0.mix.")}
    h = torch.randn(T, D, generator=g)
    want = O.gla_mixer(h.to(F64), {k: v.to(F64) for k, v in w.items()}, cfg["layers"][0]["mixer"], 1e-5)
    mix = ChannelDecayLinearAttention({k: v.to(DEV) for k, v in w.items()}, H, dk, dv, tau, 1e-5, torch.float32)
    state = tuple(torch.full((2,) + s, 3.0, device=DEV) for s in mix.state_shapes())
    out = [mix.forward(dev(h[at:at + n]), batch_of([dict(tokens=[0] * n, start=at, block_table=[0, 1], state_slot=1, want=[])]), state) for at, n in _portions(T, sizes)]
    close(torch.cat(out), want, 5e-5, f"portions {sizes}")


# ----------------------------------------------------------------------------------------------------------------------
# attention whose heads mix their scores
# ----------------------------------------------------------------------------------------------------------------------
def test_rotation_of_queries_keys_and_values():
    g = torch.Generator().manual_seed(1)
    T, start, base = 37, 130, 700.0
    for H, G, dk, dv, rot in ((4, 2, 12, 10, 8), (3, 3, 16, 6, 16), (2, 1, 10, 24, 4)):
        proj = torch.randn(T, (H + G) * dk + G * dv + 3, generator=g)
        tabs, vtabs = yarn_rotary_tables(rot, base, 256, None, DEV), yarn_rotary_tables(dv, base, 256, None, DEV)
        b = batch_of([dict(tokens=[0] * T, start=start, block_table=[2, 0, 1], state_slot=-1, want=[])])
        kc, vc = torch.zeros(3, 64, G, dk, device=DEV), torch.zeros(3, 64, G, dv, device=DEV)
        q = ops.qkv_rope_cache(dev(proj), tabs, vtabs, b, kc, vc, H, G, dk, dv, rot, torch.float32)
        pos = torch.arange(start, start + T)
        full = proj.to(F64)
        wq = O.rotate_halves(full[:, :H * dk].reshape(T, H, dk), pos, rot, base)
        wk = O.rotate_halves(full[:, H * dk:(H + G) * dk].reshape(T, G, dk), pos, rot, base)
        wv = O.rotate_halves(full[:, (H + G) * dk:(H + G) * dk + G * dv].reshape(T, G, dv), pos, dv, base)
        slots = [([2, 0, 1][p // 64], p % 64) for p in pos.tolist()]
        close(q.view(T, H, dk), wq, 3e-6, "queries")
        close(torch.stack([kc[a, o] for a, o in slots]), wk, 3e-6, "cached keys")
        close(torch.stack([vc[a, o] for a, o in slots]), wv, 3e-6, "cached values")
        kept = kc.clone()
        alone = ops.qkv_rope_cache(dev(proj[:, :H * dk]), tabs, vtabs, b, None, None, H, G, dk, dv, rot, torch.float32)
        close(alone, q.cpu(), 1e-9, "queries alone")
        assert torch.equal(kc, kept)


def run_attention(mix, h, sizes, table, dtype, cache=None, bs=64):
    """the rows of one sequence through a mixer in portions, over dirty pages in the order `table` gives"""
    g, dk, dv = mix.cache_shape()
    if cache is None:
        cache = (torch.full((max(table) + 1, bs, g, dk), 7.0, dtype=dtype, device=DEV), torch.full((max(table) + 1, bs, g, dv), -7.0, dtype=dtype, device=DEV))
    out = []
    for at, n in _portions(h.shape[0], sizes):
        b = batch_of([dict(tokens=[0] * n, start=at, block_table=table, state_slot=-1, want=[])], bs)
        out.append(mix.forward(dev(h[at:at + n], dtype), b, cache))
    return torch.cat(out), cache


def make_mixer(L, w, dtype, **kw):
    m = L["mixer"]
    return TalkingAttentionMixer({k: v.to(DEV) for k, v in w.items()}, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], dtype, rot=m["rot"], rotate_values=True,
                                 one_sink=True, chunk=(m.get("mask") or {}).get("size", 0), max_pos=600, **kw)


def mixer_case(H, G, dk, dv, chunk, rot, T, seed, D=48, scale=None):
    L = S.sigalorn_attention_layer(H, G, dk, dv, chunk=chunk, rot_dims=rot, base=300.0, scale=1.3 * dk ** -0.5 if scale is None else scale)
    w = {k[7:]: v for k, v in S.sigalorn_weights(S.sigalorn_config(D, 10, [L]), seed).items() if k.startswith("l0.mix.")}
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(seed)).to(torch.bfloat16).float()
    w64 = {k: v.to(F64) for k, v in w.items()}
    want = O.attention_mixer(h.to(F64), w64, L["mixer"], O.attention_keys_values(h.to(F64), w64, L["mixer"]))
    return L, w, h, want


ATT = [  # H, G, dk, dv, chunk, rot_dims: every head layout and odd sizes on the f32 kernel
    (4, 2, 12, 10, 9, 8), (3, 3, 16, 16, 70, 16), (6, 1, 10, 24, 0, 4), (2, 2, 20, 6, 1, 20), (8, 4, 8, 8, 130, 6), (1, 1, 7, 2, 64, 6), (12, 4, 36, 66, 50, 12),
    (16, 2, 24, 20, 77, 24), (40, 8, 16, 130, 33, 16), (5, 5, 9, 14, 128, 2)]
TABLE = [3, 1, 4, 0, 2, 6, 5]


@pytest.mark.parametrize("H,G,dk,dv,chunk,rot", ATT)
@pytest.mark.parametrize("sizes", [[260], [2], [61, 1, 1, 2, 70, 3]])
def test_talking_attention_f32(H, G, dk, dv, chunk, rot, sizes):
    T = 140 if sizes == [2] else 260
    L, w, h, want = mixer_case(H, G, dk, dv, chunk, rot, T, seed=dk + chunk)
    mix = make_mixer(L, w, torch.float32)
    got, _ = run_attention(mix, h, sizes, TABLE, torch.float32)
    close(got, want, 3e-5, f"portions {sizes}")
    for splits in (1, 3, 7):
        mix.splits = splits
        got, _ = run_attention(mix, h, sizes, TABLE, torch.float32)
        close(got, want, 3e-5, f"{splits} runs of keys, portions {sizes}")


WIDE = [  # H, G, dk, dv, chunk, rot_dims: sizes of the tensor-core kernel: one, two and four heads per warp, both tile widths, single and double buffers
    (4, 2, 64, 48, 100, 64), (8, 8, 32, 16, 0, 32), (16, 4, 128, 128, 130, 128), (12, 3, 80, 112, 64, 40), (32, 8, 64, 64, 90, 64), (20, 5, 40, 32, 33, 40),
    (5, 5, 88, 48, 200, 88), (16, 16, 128, 128, 100, 64), (32, 8, 128, 128, 150, 128), (1, 1, 8, 16, 7, 8), (6, 2, 72, 96, 1, 72), (24, 1, 128, 64, 0, 128), (16, 2, 64, 80, 70, 32), (18, 9, 24, 128, 90, 24)]


@pytest.mark.parametrize("H,G,dk,dv,chunk,rot", WIDE)
def test_talking_attention_on_the_tensor_core_kernel(H, G, dk, dv, chunk, rot):
    """bf16: whole prompts, portions that start inside pages, tiles and chunks, and single rows (the kernel of mixed queries in one and several runs of keys, and the
    f32-arithmetic kernel over the same 16-bit cache), against the oracle and against the f32 run"""
    T = 230
    L, w, h, want = mixer_case(H, G, dk, dv, chunk, rot, T, seed=H + dk)
    got32, _ = run_attention(make_mixer(L, w, torch.float32), h, [T], TABLE, torch.float32)
    close(got32, want, 3e-5, "f32")
    mix = make_mixer(L, w, torch.bfloat16)
    assert mix.prefill_kernel
    scale = float(want.abs().max())
    for sizes, splits, plain in (([T], None, False), ([100, 1, 37, 2, 64, 9], None, False), ([97, 1], None, False), ([130, 2, 1], 1, False), ([190, 1], 3, False), ([97, 1, 2], 2, True)):
        mix.splits, mix.plain = splits, plain
        got = run_attention(mix, h, sizes, TABLE, torch.bfloat16)[0].float().cpu().to(F64)
        err = (got - want).abs().max(-1).values / scale
        assert float(err.max()) < 5e-2 and float(err.median()) < 1.5e-2, (sizes, splits, plain, float(err.max()), float(err.median()), int(err.argmax()))


def test_entries_of_a_batch_do_not_see_each_other():
    """prompts, a portion that continues one and single rows side by side in one step, f32 and bf16 (tensor-core and row kernels)"""
    L, w, h, want = mixer_case(8, 4, 32, 32, 70, 32, 200, seed=5)
    for dtype, tol in ((torch.float32, 3e-5), (torch.bfloat16, 5e-2)):
        mix = make_mixer(L, w, dtype)
        g, dk, dv = mix.cache_shape()
        cache = (torch.full((12, 64, g, dk), 7.0, dtype=dtype, device=DEV), torch.full((12, 64, g, dv), -7.0, dtype=dtype, device=DEV))
        tables = [[0, 5, 2, 9], [1, 3, 8, 4], [10, 6, 7, 11]]
        fed = [0, 0, 0]
        got = [[], [], []]
        for plan in ([90, 3, 0], [1, 64, 30], [1, 1, 1], [13, 1, 9], [2, 2, 2]):
            entries = [(i, n) for i, n in enumerate(plan) if n]
            b = batch_of([dict(tokens=[0] * n, start=fed[i], block_table=tables[i], state_slot=-1, want=[]) for i, n in entries])
            x = torch.cat([h[fed[i]:fed[i] + n] for i, n in entries])
            for (i, n), o in zip(entries, mix.forward(dev(x, dtype), b, cache).split([n for _, n in entries])):
                got[i].append(o); fed[i] += n
        for i in range(3):
            close(torch.cat(got[i]), want[:fed[i]], tol, f"{dtype} entry {i}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_loud_key_at_page_and_chunk_edges(dtype):
    """Identity-like projections: head size 16, the key of one position points along the queries' direction and scores far above all others; its value is loud.
    Every query of the same chunk returns that value (turned by the distance), queries outside the chunk do not feel it."""
    H = G = 2
    dk = dv = 16
    D, chunk, T = 32, 100, 260
    eye = torch.eye(D)
    w = {"q": torch.cat([eye[:16], eye[:16]]), "k": torch.cat([eye[16:], eye[16:]]), "v": torch.cat([eye[16:], eye[16:]]) * 3, "o": torch.randn(24, 32, generator=torch.Generator().manual_seed(0)),
         "talk": torch.tensor([[1.0, 0.25], [-0.5, 0.75]])}
    L = dict(mixer=dict(heads=H, kv_heads=G, dim=dk, vdim=dv, scale=1.0, rot=dict(base=1e7, dims=2), mask=dict(size=chunk)))
    g = torch.Generator().manual_seed(2)
    for loud in (0, 63, 64, 99, 100, 127, 128, 199, 200):
        h = torch.randn(T, D, generator=g) * 0.02
        h[:, 2:8] = 1.0                                   # what every query asks for (entries 0 and 8 turn with the position, these do not)
        h[loud, 18:24] = 3.0
        h = h.to(torch.bfloat16).float()
        w64 = {k: v.to(F64) for k, v in w.items()}
        want = O.attention_mixer(h.to(F64), w64, L["mixer"], O.attention_keys_values(h.to(F64), w64, L["mixer"]))
        inside = [i for i in range(loud, T) if i // chunk == loud // chunk]
        outside = [i for i in range(loud + 1, T) if i // chunk != loud // chunk]
        assert float(want[inside].abs().mean()) > 10 * float(want[outside].abs().mean() if outside else 0.0)
        mix = make_mixer(L, w, dtype)
        for sizes in ([T], [1], [98, 2, 1, 1, 2, 96]):
            got, _ = run_attention(mix, h, sizes, TABLE, dtype)
            close(got, want, 3e-5 if dtype == torch.float32 else 3e-2, f"loud key {loud}, portions {sizes}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_one_in_the_denominator_carries_low_scores(dtype):
    """Scores of about -4: most of every row's weight is on the sink, so the outputs are far smaller than an ordinary softmax's; scores of +6: it hardly counts"""
    for shift in (-4.0, 6.0):
        H, G, dk, dv, D, T = 4, 2, 16, 16, 24, 70
        L, w, h, _ = mixer_case(H, G, dk, dv, 0, 2, T, seed=11, D=D, scale=0.25)
        h[:, 0] = 4.0
        w = {k: v.float().clone() for k, v in w.items()}
        w["q"] *= 0.1; w["k"] *= 0.1
        w["q"].view(H, dk, D)[:, 5, 0], w["k"].view(G, dk, D)[:, 5, 0] = 1.0, shift / 4.0
        w["talk"] = torch.eye(H) + 0.05
        w = {k: v.to(torch.bfloat16) for k, v in w.items()}
        h = h.to(torch.bfloat16).float()
        w64 = {k: v.to(F64) for k, v in w.items()}
        kv = O.attention_keys_values(h.to(F64), w64, L["mixer"])
        want = O.attention_mixer(h.to(F64), w64, L["mixer"], kv)
        mix = make_mixer(L, w, dtype)
        for sizes in ([T], [1]):
            got, _ = run_attention(mix, h, sizes, TABLE, dtype)
            close(got, want, 3e-5 if dtype == torch.float32 else 3e-2, f"shift {shift}, portions {sizes}")
        mix.one_sink = False
        plain, _ = run_attention(mix, h, [T], TABLE, dtype)
        moved = float((plain.float().cpu().to(F64) - want).abs().max() / want.abs().max())
        assert moved > 0.3 if shift < 0 else moved < 0.3, moved
        rows, _ = run_attention(mix, h, [1], TABLE, dtype)
        close(rows, plain.float().cpu(), 3e-5 if dtype == torch.float32 else 3e-2, "without the sink: row kernel against prompt kernel")


def test_a_layer_over_another_layers_keys_with_a_mask_of_its_own():
    H, G, dk, dv, D, T = 6, 2, 24, 32, 48, 180
    src, w_src, h, _ = mixer_case(H, G, dk, dv, 64, 12, T, seed=3)
    use = S.sigalorn_attention_layer(4, G, dk, dv, chunk=50, rot_dims=12, base=300.0, scale=0.3, kv_from=0)
    w_use = {k[7:]: v for k, v in S.sigalorn_weights(S.sigalorn_config(D, 10, [use]), 8).items() if k.startswith("l0.mix.")}
    assert "k" not in w_use and "v" not in w_use
    h2 = torch.randn(T, D, generator=torch.Generator().manual_seed(4)).to(torch.bfloat16).float()
    kv = O.attention_keys_values(h.to(F64), {k: v.to(F64) for k, v in w_src.items()}, src["mixer"])
    want = O.attention_mixer(h2.to(F64), {k: v.to(F64) for k, v in w_use.items()}, use["mixer"], kv)
    for dtype, tol in ((torch.float32, 3e-5), (torch.bfloat16, 5e-2)):
        own, shared = make_mixer(src, w_src, dtype), make_mixer(use, w_use, dtype, shared=True)
        _, cache = run_attention(own, h, [T], TABLE, dtype)
        before = [c.clone() for c in cache]
        for sizes in ([T], [1], [50, 2, 7]):
            got, _ = run_attention(shared, h2, sizes, TABLE, dtype, cache)
            close(got, want, tol, f"{dtype} portions {sizes}")
        assert all(torch.equal(a, b) for a, b in zip(before, cache))


# ----------------------------------------------------------------------------------------------------------------------
# whole models
# ----------------------------------------------------------------------------------------------------------------------
CONFIGS = {
    # both mixers with nothing equal to anything else, a shared layer with a mask of its own, a layer without feed-forward
    "mix": S.sigalorn_config(40, 211, [S.sigalorn_gla_layer(3, 12, 20, tau=8.0, ff=56), S.sigalorn_attention_layer(6, 2, 14, 18, chunk=37, rot_dims=10, base=500.0, ff=72),
                                       S.sigalorn_gla_layer(2, 24, 10, tau=1.0), S.sigalorn_attention_layer(4, 2, 14, 18, chunk=90, rot_dims=10, base=500.0, kv_from=1, ff=30)],
                             eps=1e-5, embedding_scale=2.5, softcap=9.0),
    # attention first, one kv head, odd sizes, no mask, no cap, two layers over the first one's keys
    "odd": S.sigalorn_config(33, 57, [S.sigalorn_attention_layer(3, 1, 9, 6, rot_dims=4, base=90.0, ff=17), S.sigalorn_attention_layer(5, 1, 9, 6, chunk=64, rot_dims=4, base=90.0, kv_from=0),
                                      S.sigalorn_gla_layer(1, 7, 5, tau=3.0, ff=11), S.sigalorn_attention_layer(2, 1, 9, 6, chunk=11, rot_dims=4, base=90.0, kv_from=0, ff=9)],
                             softcap=0.0),
    # sizes of the tensor-core kernels, kv heads == heads, value size == key size
    "aligned": S.sigalorn_config(128, 200, [S.sigalorn_attention_layer(4, 4, 64, 64, chunk=128, base=1e4, ff=256), S.sigalorn_gla_layer(2, 64, 64, ff=256),
                                            S.sigalorn_attention_layer(4, 4, 64, 64, chunk=100, base=1e4, ff=128, kv_from=0)], embedding_scale=0.5, softcap=30.0),
}
TOL = 2e-4
_CACHE = {}


def model_and_oracle(name, dtype, T):
    key = (name, T)
    if key not in _CACHE:
        cfg = CONFIGS[name]
        w = S.sigalorn_weights(cfg, 0)
        toks = torch.randint(0, cfg["vocab"], (T,), generator=torch.Generator().manual_seed(1)).tolist()
        trace = []
        _CACHE[key] = (w, toks, O.forward(cfg, w, toks, trace), trace)
    w, toks, ref, trace = _CACHE[key]
    return SigalornModel(SigalornConfig.from_dict(CONFIGS[name]), w, dtype=dtype, block_size=64, max_pos=512, device=DEV), toks, ref, trace


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
    if CONFIGS[name].get("logit_softcap"):
        assert float(ref.abs().max()) > 0.6 * CONFIGS[name]["logit_softcap"]          # the cap shows


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
    w = S.sigalorn_weights(cfg, 0)
    model = SigalornModel(SigalornConfig.from_dict(cfg), w, dtype=dtype, block_size=64, max_pos=512, device=DEV)
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


def test_long_decoding_across_pages_and_chunks():
    model, toks, ref, _ = model_and_oracle("mix", torch.float32, 300)
    runner = ModelRunner(model, 5, 1, 64)
    runner.admit(0)
    got = [runner.execute([dict(seq_id=0, tokens=toks[:20], want=list(range(20)))])]
    for t in range(20, 300):
        got.append(runner.execute([dict(seq_id=0, tokens=[toks[t]], want=[0])]))
    close(torch.cat(got), ref, TOL, "280 decoded tokens")


def test_first_tokens_and_single_token_requests():
    model, toks, ref, _ = model_and_oracle("odd", torch.float32, 230)
    runner = ModelRunner(model, 4, 2, 64)
    for n in (1, 2, 3):
        runner.admit(n)
        close(runner.execute([dict(seq_id=n, tokens=toks[:n], want=list(range(n)))]), ref[:n], TOL, f"first {n} tokens")
        runner.release(n)


def test_graph_replay_of_decode_steps_matches_eager():
    cfg = CONFIGS["mix"]
    w = S.sigalorn_weights(cfg, 0)
    model = SigalornModel(SigalornConfig.from_dict(cfg), w, dtype=torch.float32, block_size=64, max_pos=64, device=DEV)      # tables must grow
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
        close(torch.cat(got[i]), refs[i], TOL, f"graph replay, request {i}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_greedy_generation_through_the_engine(dtype, tmp_path):
    """checkpoint on disk -> registry -> LLMEngine (scheduler, chunked prefill, sampler) against the oracle's greedy continuation"""
    from candle_vllm_b200.safetensors_io import save_file
    cfg = CONFIGS["mix"]
    w = S.sigalorn_weights(cfg, 4)
    save_file(w, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    g = torch.Generator().manual_seed(2)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (70, 3, 33, 1, 129)]
    eng = LLMEngine.from_pretrained(str(tmp_path), dtype=dtype, num_blocks=7, max_num_seqs=2, prefill_chunk=48, max_batch_tokens=64, max_model_len=256)
    assert type(eng.model).__name__ == "SigalornModel"
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
    w = S.sigalorn_weights(cfg, 1)
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
