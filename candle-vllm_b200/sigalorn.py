"""Sigalorn: a decoder whose layers mix the sequence either with gated linear attention (a decay per token and key row over an f32 matrix state) or with
chunk-masked softmax attention whose heads mix their scores before the softmax, each sublayer wrapped in an RMS norm before and after
(x <- x + norm1b(mixer(norm1 x)), x <- x + norm2b(ff(norm2 x))), a dense ungated feed-forward with xIELU and biases, scaled embeddings, an untied head and a
cap on the logits.

  gla        q, k, v plain (q times dim^-1/2), alpha = sigmoid(a2 (a1 h) + a2.b)^(1 / tau), S <- diag(alpha) S + k v^T, o = S^T q, each head normed, times silu(g h);
  attention  grouped-query attention: rotated q and k, values cached turned by their position and outputs turned back, scores mixed by talk [H, H], one added to
             the softmax denominator, a query sees the keys of its own chunk of mask.size positions; with kv_from the layer attends over the keys and values of
             an earlier layer, with its own queries, scores and mask.

Everything size- or constant-like comes from ``config.json``:

  architecture, vocab, width, embedding.scale, norm.eps, logit_softcap,
  layers[i] = {type: "gla" | "attention", mixer: {...}, mlp: null | {kind: "dense", ff}}
    gla        mixer = {heads, dim, vdim, tau}
    attention  mixer = {heads, kv_heads, dim, vdim, scale, mask: {size}, rot: {base, dims}, kv_from}
  (mask, rot, kv_from, mlp, logit_softcap and embedding.scale may be absent: no mask, no rotation, keys and values of its own, no feed-forward, no cap, scale 1.)

Tensor names: embed, l<i>.norm1 / norm1b / norm2 / norm2b, l<i>.mix.{q, k, v, g, a1, a2, a2.b, norm, o} | {q, k, v, talk, o},
l<i>.mlp.{up, up.b, down, down.b, act}, final.norm, head.
The model object holds weights only; the paged cache of the attention layers and the state of the recurrent ones are allocated by the engine from
``cache_plan()`` and handed to ``forward``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ._lib import BackendError, require_device
from . import seq_ops as ops
from .mixers import ChannelDecayLinearAttention, TalkingAttentionMixer, UngatedMlp
from .seq_ops import StepBatch

MIXERS = ("gla", "attention")


@dataclass
class SigalornConfig:
    vocab: int
    width: int
    embedding_scale: float
    eps: float
    softcap: float
    layers: List[dict]
    raw: dict = field(default_factory=dict)

    @classmethod
    def from_dict(cls, d: dict) -> "SigalornConfig":
        try:
            cfg = cls(vocab=int(d["vocab"]), width=int(d["width"]), embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)), eps=float(d["norm"]["eps"]),
                      softcap=float(d.get("logit_softcap") or 0.0), layers=list(d["layers"]), raw=d)
            for i, L in enumerate(cfg.layers):
                m = L["mixer"]
                if L.get("type") not in MIXERS:
                    raise BackendError(f"layer {i}: unknown mixer type {L.get('type')!r}")
                if L["type"] == "gla":
                    for key in ("heads", "dim", "vdim", "tau"):
                        m[key]
                    if not float(m["tau"]) > 0:
                        raise BackendError(f"layer {i}: tau {m['tau']} is not positive")
                else:
                    for key in ("heads", "kv_heads", "dim", "vdim", "scale"):
                        m[key]
                    if m.get("rot"):
                        m["rot"]["base"], m["rot"]["dims"]
                    src = m.get("kv_from")
                    if src is not None:
                        src = int(src)
                        if not 0 <= src < i or cfg.layers[src]["type"] != "attention" or cfg.layers[src]["mixer"].get("kv_from") is not None:
                            raise BackendError(f"layer {i}: kv_from {src} must name an earlier attention layer with keys and values of its own")
                        sm = cfg.layers[src]["mixer"]
                        if any(int(sm[k]) != int(m[k]) for k in ("kv_heads", "dim", "vdim")) or sm.get("rot") != m.get("rot"):
                            raise BackendError(f"layer {i}: kv heads, key and value sizes and rotation must equal those of layer {src}")
                mlp = L.get("mlp")
                if mlp:
                    if mlp.get("kind", "dense") != "dense":
                        raise BackendError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
                    mlp["ff"]
        except KeyError as e:
            raise BackendError(f"Sigalorn config lacks {e}")
        return cfg

    @classmethod
    def from_json(cls, path: str) -> "SigalornConfig":
        with open(path) as f:
            return cls.from_dict(json.load(f))


class _Layer:
    def __init__(self, cfg: SigalornConfig, i: int, w: Dict[str, torch.Tensor], dtype: torch.dtype, block_size: int, max_pos: int):
        L, p = cfg.layers[i], f"l{i}."
        sub = lambda pre: {k[len(pre):]: v for k, v in w.items() if k.startswith(pre)}
        f32 = lambda name: w[p + name].float().contiguous()
        m, mw = L["mixer"], sub(p + "mix.")
        self.type = L["type"]
        self.kv_from = None
        self.norm1, self.norm1b = f32("norm1"), f32("norm1b")
        if self.type == "gla":
            self.mixer = ChannelDecayLinearAttention(mw, int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]), cfg.eps, dtype)
        else:
            self.kv_from = None if m.get("kv_from") is None else int(m["kv_from"])
            self.mixer = TalkingAttentionMixer(mw, int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), dtype, rot=m.get("rot") or None,
                                               rotate_values=True, one_sink=True, shared=self.kv_from is not None, chunk=int((m.get("mask") or {}).get("size", 0)),
                                               block_size=block_size, max_pos=max_pos)
        self.mlp = None
        if L.get("mlp"):
            self.norm2, self.norm2b = f32("norm2"), f32("norm2b")
            self.mlp = UngatedMlp(sub(p + "mlp."), dtype, act="xielu")
            if self.mlp.ff != int(L["mlp"]["ff"]):
                raise BackendError(f"layer {i}: feed-forward tensors have ff {self.mlp.ff}, the config says {L['mlp']['ff']}")


class SigalornModel:
    architecture = "Sigalorn"

    def __init__(self, cfg: SigalornConfig, weights: Dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16, block_size: int = 64, max_pos: int = 4096,
                 device="cuda"):
        require_device()
        if dtype not in (torch.bfloat16, torch.float32):
            raise BackendError("Sigalorn runs in bfloat16 or float32")
        self.cfg, self.dtype, self.block_size, self.device = cfg, dtype, block_size, torch.device(device)
        w = {k: v.to(self.device) for k, v in weights.items()}
        self.embed = w["embed"].to(dtype).contiguous()
        self.head = w["head"].to(dtype).contiguous()
        if self.embed.shape != (cfg.vocab, cfg.width) or self.head.shape != (cfg.vocab, cfg.width):
            raise BackendError(f"embed {tuple(self.embed.shape)} / head {tuple(self.head.shape)} against vocab {cfg.vocab}, width {cfg.width}")
        self.final_norm = w["final.norm"].float().contiguous()
        self.layers = [_Layer(cfg, i, w, dtype, block_size, max_pos) for i in range(len(cfg.layers))]
        # cache index of every layer: attention layers with keys of their own and recurrent layers count separately; a sharing layer uses its source's
        self.layer_cache, nkv, nst = [], 0, 0
        for L in self.layers:
            if L.type == "gla":
                self.layer_cache.append(nst); nst += 1
            elif L.kv_from is None:
                self.layer_cache.append(nkv); nkv += 1
            else:
                self.layer_cache.append(self.layer_cache[L.kv_from])
        self.vocab = cfg.vocab

    @classmethod
    def from_pretrained(cls, path: str, dtype: torch.dtype = torch.bfloat16, **kw) -> "SigalornModel":
        from .safetensors_io import load_file
        cfg = SigalornConfig.from_json(os.path.join(path, "config.json"))
        return cls(cfg, load_file(os.path.join(path, "model.safetensors")), dtype=dtype, **kw)

    def ensure_positions(self, max_pos: int) -> bool:
        """grow the rotary tables (outside any graph capture) to cover positions below ``max_pos``; True if a table moved"""
        moved = False
        for L in self.layers:
            cos = getattr(L.mixer, "cos", None)
            if cos is not None and cos.shape[0] < max_pos:
                L.mixer.ensure_positions(max(2 * cos.shape[0], max_pos))
                moved = True
        return moved

    def cache_plan(self) -> dict:
        """What the engine allocates: one (kv heads, key size, value size) per attention layer with keys of its own, one tuple of per-slot state shapes per
        recurrent layer, both in layer order."""
        return dict(kv_layers=[L.mixer.cache_shape() for L in self.layers if L.type == "attention" and L.kv_from is None],
                    state_layers=[L.mixer.state_shapes() for L in self.layers if L.type == "gla"])

    def forward(self, batch: StepBatch, kv_cache, state_cache, hidden_trace: Optional[list] = None) -> Optional[torch.Tensor]:
        """Runs the step's rows through every layer, advancing cache and states; returns f32 logits [R, vocab] of the wanted rows (None when nothing is wanted)."""
        cfg, dt = self.cfg, self.dtype
        x = ops.embedding_scaled(self.embed, batch.tokens, cfg.embedding_scale)
        pending = None                    # a sublayer's output, its bias and its closing norm: the next opening norm's kernel adds it to the stream first

        def opening(weight, row_index=None):
            nonlocal pending
            if pending is None:
                return ops.rms_norm_ex(x, weight, cfg.eps, 0.0, dt, row_index=row_index)
            y, bias, post = pending
            pending = None
            return ops.post_norm_add_rms_norm(x, y, post, weight, cfg.eps, dt, y_bias=bias, row_index=row_index)

        for L, ci in zip(self.layers, self.layer_cache):
            h = opening(L.norm1)
            pending = (L.mixer.forward(h, batch, state_cache[ci] if L.type == "gla" else kv_cache[ci]), None, L.norm1b)
            if L.mlp is not None:
                h = opening(L.norm2)
                pending = (L.mlp.forward(h), L.mlp.down_bias, L.norm2b)
            if hidden_trace is not None:
                y, bias, post = pending
                ops.post_norm_add_rms_norm(x, y, post, None, cfg.eps, y_bias=bias)
                pending = None
                hidden_trace.append(x.clone())
        if batch.num_want == 0:
            return None
        logits = ops.linear(opening(self.final_norm, row_index=batch.want_rows), self.head)
        return ops.softcap(logits, cfg.softcap) if cfg.softcap else logits
