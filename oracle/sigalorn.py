"""Plain, slow restatement of the Sigalorn decoder (test infrastructure only; shares no code with the product path).

One function per mechanism, float64 torch on the CPU, whole sequences only: a sequence is processed from position 0 with empty state,
token by token where the mechanism is a recurrence and query by query in attention.  The product (paged cache, state slots, batched
steps, CUDA kernels) is compared against this.

Notation: T tokens, D model width, H query heads, G key / value heads, dk key size, dv value size; linear weights are [out, in].
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def xielu(z: torch.Tensor, p: float, q: float) -> torch.Tensor:
    """softplus(p) z^2 + z / 2 where z > 0, (1/2 + softplus(q)) (e^z - 1 - z) + z / 2 elsewhere."""
    sp = lambda a: math.log1p(math.exp(-abs(a))) + max(a, 0.0)
    return torch.where(z > 0, sp(p) * z * z + 0.5 * z, (0.5 + sp(q)) * (torch.expm1(z.clamp(max=0.0)) - z) + 0.5 * z)


def decay_per_key(z: torch.Tensor, tau: float) -> torch.Tensor:
    """sigmoid(z)^(1/tau), through the logarithm so that strongly negative z keep their relative accuracy."""
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def gated_linear_recurrence(q, k, v, alpha) -> torch.Tensor:
    """q, k, alpha [T, H, dk], v [T, H, dv].  Per head, S [dk, dv] from zero: S[r, :] <- alpha_t[r] S[r, :] + k_t[r] v_t, o_t = sum_r q_t[r] S[r, :]."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=F)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for t in range(T):
        S = S * alpha[t][:, :, None] + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (q[t][:, :, None] * S).sum(1)
    return out


def gla_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T * dk ** -0.5).view(T, H, dk)
    k = (h @ w["k"].T).view(T, H, dk)
    v = (h @ w["v"].T).view(T, H, dv)
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    o = gated_linear_recurrence(q, k, v, decay_per_key(z, m["tau"]).view(T, H, dk))
    o = rms(o, eps) * w["norm"]
    return (o.reshape(T, H * dv) * silu(h @ w["g"].T)) @ w["o"].T


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float, back: bool = False) -> torch.Tensor:
    """x [T, heads, n]: entries (i, i + dims/2) of every head, i < dims/2, turned by the angle position * base^(-2 i / dims) (minus that if
    ``back``); entries from ``dims`` on pass."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(F) * base ** (-2.0 * i / dims) * (-1.0 if back else 1.0)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + dims // 2]
        out[:, :, i] = u * c - v * s
        out[:, :, i + dims // 2] = v * c + u * s
    return out


def sees(i: int, j: int, chunk: int) -> bool:
    """may the query at position i look at the key at position j?  chunk 0: every earlier key"""
    return j <= i and (chunk <= 0 or i // chunk == j // chunk)


def softmax_with_one(s: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s_j)) over the last axis."""
    m = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def talking_attention(q, k, v, scale: float, talk: torch.Tensor, chunk: int) -> torch.Tensor:
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] (all rotated already) -> [T, H, dv]: every query's H rows of scores are mixed by talk [H, H] before
    the softmax."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for i in range(T):
        js = [j for j in range(i + 1) if sees(i, j, chunk)]
        raw = torch.stack([k[js, h // group] @ q[i, h] for h in range(H)]) * scale           # [H, keys]
        p = softmax_with_one(talk @ raw)
        for h in range(H):
            out[i, h] = p[h] @ v[js, h // group]
    return out


def attention_keys_values(h, w, m):
    """what a layer's cache holds: keys rotated on rot.dims entries, values rotated over all of theirs"""
    T, G, dk, dv = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    k, v = (h @ w["k"].T).view(T, G, dk), (h @ w["v"].T).view(T, G, dv)
    rot = m["rot"]
    return rotate_halves(k, pos, rot["dims"], rot["base"]), rotate_halves(v, pos, dv, rot["base"])


def attention_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, kv) -> torch.Tensor:
    """``kv``: the keys and values of this layer or of the layer it shares them with"""
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos, rot = torch.arange(T), m["rot"]
    q = rotate_halves((h @ w["q"].T).view(T, H, dk), pos, rot["dims"], rot["base"])
    o = talking_attention(q, kv[0], kv[1], m["scale"], w["talk"], (m.get("mask") or {}).get("size", 0))
    o = rotate_halves(o, pos, dv, rot["base"], back=True)
    return o.reshape(T, H * dv) @ w["o"].T


def dense_mlp(h, w):
    p, q = (float(a) for a in w["act"])
    return xielu(h @ w["up"].T + w["up.b"], p, q) @ w["down"].T + w["down.b"]


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens, trace: Optional[list] = None) -> torch.Tensor:
    """tokens: T ids of ONE sequence from position 0 -> logits [T, vocab] (float64).  `trace`, if a list, receives the residual stream
    after every layer."""
    W = {k: v.to(F) for k, v in weights.items() if v.is_floating_point()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    shared = {}
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        sub = lambda pre: {k[len(p + pre):]: v for k, v in W.items() if k.startswith(p + pre)}
        m, w = L["mixer"], sub("mix.")
        h = rms(x, eps) * W[p + "norm1"]
        if L["type"] == "gla":
            y = gla_mixer(h, w, m, eps)
        else:
            if m.get("kv_from") is None:
                shared[i] = attention_keys_values(h, w, m)
            y = attention_mixer(h, w, m, shared[i if m.get("kv_from") is None else m["kv_from"]])
        x = x + rms(y, eps) * W[p + "norm1b"]
        if L.get("mlp"):
            y = dense_mlp(rms(x, eps) * W[p + "norm2"], sub("mlp."))
            x = x + rms(y, eps) * W[p + "norm2b"]
        if trace is not None:
            trace.append(x.clone())
    logits = (rms(x, eps) * W["final.norm"]) @ W["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


def greedy(cfg, weights, prompt, steps: int) -> List[int]:
    """Greedy continuation by re-running the whole sequence (slow, on purpose)."""
    ids = list(prompt)
    for _ in range(steps):
        ids.append(int(forward(cfg, weights, ids)[-1].argmax()))
    return ids[len(prompt):]
