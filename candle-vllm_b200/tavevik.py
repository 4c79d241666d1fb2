"""Tavevik: a decoder whose layers run windowed softmax attention and a recurrent mixer side by side on the stream itself, with norms on the sublayers' outputs only
(x <- x + norm1(mixer(x)), x <- x + norm2(ff(x))), a dense clamped feed-forward, and the embedding table as the output head.

  parallel    left: grouped-query attention, q and k normed head by head and then rotated, scores capped, a sliding window plus the first tokens of the sequence, one
              sigmoid gate per output entry; right: linear attention over shifted tokens with decays exp(-exp(.)) and a bonus for the current token;
  parallel_2  left: grouped-query attention with biases on all four projections, normed and rotated q and k, a sliding window, a learned sink per head; right: the gated
              delta rule with a decay per token and key row, short convolutions, a low-rank output gate.

A layer's mixer returns left_scale * left + right_scale * right.  Everything size- or constant-like comes from ``config.json``:

  architecture, vocab, width, norm.eps,
  layers[i] = {type: "parallel" | "parallel_2", mixer: {left, right, left_scale, right_scale}, mlp: null | {kind: "dense", ff, limit}}
    left         {heads, kv_heads, dim, vdim, scale, rot: {base, dims}, mask: {size, keep_first}, softcap}
    right        {heads, dim} | {heads, kv_heads, dim, vdim, conv}
  (rot, mask, keep_first and softcap may be absent: no rotation, every earlier token, no kept tokens, no cap.)

Tensor names: embed, l<i>.norm1 / norm2, l<i>.mix.left.{q, k, v (+ .b), q.norm, k.norm, g, sink, o (+ .b)},
l<i>.mix.right.{mu.{r, k, v, g, w}, r, k, v, g, w1, w2, w0, u, norm, o} | {q, k, v (+ .conv), b, A_log, a1, a2, dt_bias, g1, g2, norm, o},
l<i>.mlp.{gate, up, down}, final.norm.  Low ranks come from the tensors' shapes; an output gate, a sink or a bias is there when its tensor is.
The model object holds weights only; the paged cache and the state (every layer has both) are allocated by the engine from ``cache_plan()``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ._lib import BackendError, require_device
from . import seq_ops as ops
from .mixers import ChannelDecayDeltaMixer, GatedMlp, PagedAttentionMixer, ParallelSumMixer, TokenShiftLinearAttention
from .seq_ops import StepBatch

MIXERS = ("parallel", "parallel_2")


@dataclass
class TavevikConfig:
    vocab: int
    width: int
    eps: float
    layers: List[dict]
    raw: dict = field(default_factory=dict)

    @classmethod
    def from_dict(cls, d: dict) -> "TavevikConfig":
        try:
            cfg = cls(vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]), layers=list(d["layers"]), raw=d)
            for i, L in enumerate(cfg.layers):
                if L.get("type") not in MIXERS:
                    raise BackendError(f"layer {i}: unknown mixer type {L.get('type')!r}")
                m = L["mixer"]
                m["left_scale"], m["right_scale"]
                for key in ("heads", "kv_heads", "dim", "vdim", "scale"):
                    m["left"][key]
                if m["left"].get("rot"):
                    m["left"]["rot"]["base"], m["left"]["rot"]["dims"]
                mask = m["left"].get("mask") or {}
                if mask.get("keep_first") and not mask.get("size"):
                    raise BackendError(f"layer {i}: kept first tokens without a window")
                for key in ("heads", "dim") if L["type"] == "parallel" else ("heads", "kv_heads", "dim", "vdim", "conv"):
                    m["right"][key]
                mlp = L.get("mlp")
                if mlp:
                    if mlp.get("kind", "dense") != "dense":
                        raise BackendError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
                    mlp["ff"], mlp["limit"]
        except KeyError as e:
            raise BackendError(f"Tavevik config lacks {e}")
        return cfg

    @classmethod
    def from_json(cls, path: str) -> "TavevikConfig":
        with open(path) as f:
            return cls.from_dict(json.load(f))


class _Layer:
    def __init__(self, cfg: TavevikConfig, i: int, w: Dict[str, torch.Tensor], dtype: torch.dtype, block_size: int, max_pos: int):
        L, p = cfg.layers[i], f"l{i}."
        sub = lambda pre: {k[len(pre):]: v for k, v in w.items() if k.startswith(pre)}
        f32 = lambda name: w[p + name].float().flatten().contiguous()
        m = L["mixer"]
        lm, rm, mask = m["left"], m["right"], m["left"].get("mask") or {}
        lw, rw = sub(p + "mix.left."), sub(p + "mix.right.")
        factor = ParallelSumMixer.right_factor(float(m["left_scale"]), float(m["right_scale"]))
        left = PagedAttentionMixer(lw, int(lm["heads"]), int(lm["kv_heads"]), int(lm["dim"]), int(lm["vdim"]), float(lm["scale"]), cfg.eps, dtype, rot=lm.get("rot") or None,
                                   window=int(mask.get("size") or 0), keep_first=int(mask.get("keep_first") or 0), softcap=float(lm.get("softcap") or 0.0), gate="element",
                                   head_norm="before", block_size=block_size, max_pos=max_pos)
        if L["type"] == "parallel":
            right = TokenShiftLinearAttention(rw, int(rm["heads"]), int(rm["dim"]), cfg.eps, dtype, norm_scale=factor)
        else:
            right = ChannelDecayDeltaMixer(rw, int(rm["heads"]), int(rm["kv_heads"]), int(rm["dim"]), int(rm["vdim"]), int(rm["conv"]), cfg.eps, dtype, norm_scale=factor)
        self.mixer = ParallelSumMixer(left, right, float(m["left_scale"]))
        self.norm1 = f32("norm1")
        self.mlp = None
        if L.get("mlp"):
            self.norm2 = f32("norm2")
            self.mlp = GatedMlp(sub(p + "mlp."), dtype, act="clamped", limit=float(L["mlp"]["limit"]))
            if self.mlp.w_down.shape[1] != int(L["mlp"]["ff"]):
                raise BackendError(f"layer {i}: feed-forward tensors have ff {self.mlp.w_down.shape[1]}, the config says {L['mlp']['ff']}")


class TavevikModel:
    architecture = "Tavevik"

    def __init__(self, cfg: TavevikConfig, weights: Dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16, block_size: int = 64, max_pos: int = 4096,
                 device="cuda"):
        require_device()
        if dtype not in (torch.bfloat16, torch.float32):
            raise BackendError("Tavevik runs in bfloat16 or float32")
        self.cfg, self.dtype, self.block_size, self.device = cfg, dtype, block_size, torch.device(device)
        w = {k: v.to(self.device) for k, v in weights.items()}
        self.embed = w["embed"].to(dtype).contiguous()
        if self.embed.shape != (cfg.vocab, cfg.width):
            raise BackendError(f"embed {tuple(self.embed.shape)} against vocab {cfg.vocab}, width {cfg.width}")
        self.final_norm = w["final.norm"].float().contiguous()
        self.layers = [_Layer(cfg, i, w, dtype, block_size, max_pos) for i in range(len(cfg.layers))]
        self.vocab = cfg.vocab

    @classmethod
    def from_pretrained(cls, path: str, dtype: torch.dtype = torch.bfloat16, **kw) -> "TavevikModel":
        from .safetensors_io import load_file
        cfg = TavevikConfig.from_json(os.path.join(path, "config.json"))
        return cls(cfg, load_file(os.path.join(path, "model.safetensors")), dtype=dtype, **kw)

    def ensure_positions(self, max_pos: int) -> bool:
        """grow the rotary tables (outside any graph capture) to cover positions below ``max_pos``; True if a table moved"""
        moved = False
        for L in self.layers:
            left = L.mixer.left
            if left.cos is not None and left.cos.shape[0] < max_pos:
                left.ensure_positions(max(2 * left.cos.shape[0], max_pos))
                moved = True
        return moved

    def cache_plan(self) -> dict:
        """What the engine allocates, one entry per layer each: (kv heads, key size, value size) of the paged cache and the tuple of per-slot state shapes."""
        return dict(kv_layers=[L.mixer.cache_shape() for L in self.layers], state_layers=[L.mixer.state_shapes() for L in self.layers])

    def forward(self, batch: StepBatch, kv_cache, state_cache, hidden_trace: Optional[list] = None) -> Optional[torch.Tensor]:
        """Runs the step's rows through every layer, advancing caches and states; returns f32 logits [R, vocab] of the wanted rows (None when nothing is wanted)."""
        cfg, dt = self.cfg, self.dtype
        x = ops.embedding_scaled(self.embed, batch.tokens, 1.0)
        # what the sublayers read: the f32 stream itself, or its copy in the compute dtype that every closing norm leaves beside the sum
        h = x if dt == torch.float32 else ops.cast_rows(x)
        copy = None if dt == torch.float32 else h
        last = None                       # the last sublayer's closing norm: summed with the final norm, on the wanted rows only
        for li, L in enumerate(self.layers):
            final = li + 1 == len(self.layers) and hidden_trace is None
            y = L.mixer.forward(x, h, batch, kv_cache[li], state_cache[li])
            closing = dict(y=y, post_weight=L.norm1, y_scale=L.mixer.out_scale, y_bias=L.mixer.out_bias)
            if L.mlp is not None:
                ops.post_norm_add_rms_norm(x, weight=None, eps=cfg.eps, copy=copy, **closing)
                closing = dict(y=L.mlp.forward(h), post_weight=L.norm2)
            if final:
                last = closing
            else:
                ops.post_norm_add_rms_norm(x, weight=None, eps=cfg.eps, copy=copy, **closing)
            if hidden_trace is not None:
                hidden_trace.append(x.clone())
        if batch.num_want == 0:
            return None
        if last is not None:
            hn = ops.post_norm_add_rms_norm(x, weight=self.final_norm, eps=cfg.eps, out_dtype=dt, row_index=batch.want_rows, **last)
        else:
            hn = ops.rms_norm_ex(x, self.final_norm, cfg.eps, 0.0, dt, row_index=batch.want_rows)
        return ops.linear(hn, self.embed)
