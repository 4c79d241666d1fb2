"""Plain, slow restatement of the Tavevik decoder (test infrastructure only; shares no code with the product path).

One function per mechanism, float64 torch on the CPU, whole sequences only: a sequence is processed from position 0 with empty state,
token by token where the mechanism is a recurrence and query by query in attention.  The product (paged cache, state slots, batched
steps, CUDA kernels) is compared against this.

Notation: T tokens, D model width, H query heads, G key / value heads, dk key size, dv value size; linear weights are [out, in].
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

F = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0.0)


def clamped_glu(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    """g sigmoid(1.702 g) (u + 1) with g = min(gate, limit) and u held between -limit and limit."""
    g, u = gate.clamp(max=limit), up.clamp(min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


# ---- attention -------------------------------------------------------------------------------------------------------------------------

def rotate_halves(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, n]: entries (i, i + dims/2) of every head, i < dims/2, turned by the angle position * base^(-2 i / dims); the rest pass."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(F) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + dims // 2]
        out[:, :, i] = u * c - v * s
        out[:, :, i + dims // 2] = v * c + u * s
    return out


def sees(i: int, j: int, window: int, keep_first: int) -> bool:
    """may the query at position i look at the key at position j?  window 0: every earlier key; the first ``keep_first`` positions never leave."""
    return j <= i and (window <= 0 or i - j < window or j < keep_first)


def cap_scores(s: torch.Tensor, cap: float) -> torch.Tensor:
    """cap tanh(s / cap); cap 0: the scores as they are."""
    return cap * torch.tanh(s / cap) if cap else s


def softmax_with_sink(s: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """exp(s_j) / (exp(sink) + sum exp(s_j)) over the last axis; without a sink the ordinary softmax."""
    m = s.max() if sink is None else torch.maximum(s.max(), sink)
    e = torch.exp(s - m)
    return e / (e.sum() + (0.0 if sink is None else torch.exp(sink - m)))


def windowed_attention(q, k, v, scale: float, window: int, keep_first: int, cap: float, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv], one query and head at a time."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for i in range(T):
        js = [j for j in range(i + 1) if sees(i, j, window, keep_first)]
        for h in range(H):
            s = cap_scores((k[js, h // group] @ q[i, h]) * scale, cap)
            out[i, h] = softmax_with_sink(s, None if sink is None else sink[h]) @ v[js, h // group]
    return out


def attention_part(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    """h [T, D] -> [T, D]: biases, sink and the element-wise output gate are there when their tensors are"""
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    lin = lambda n, x: x @ w[n].T + (w[n + ".b"] if n + ".b" in w else 0.0)
    q = rms(lin("q", h).view(T, H, dk), eps) * w["q.norm"]
    k = rms(lin("k", h).view(T, G, dk), eps) * w["k.norm"]
    v = lin("v", h).view(T, G, dv)
    rot = m.get("rot")
    if rot:
        q, k = rotate_halves(q, pos, rot["dims"], rot["base"]), rotate_halves(k, pos, rot["dims"], rot["base"])
    mask = m.get("mask") or {}
    o = windowed_attention(q, k, v, m["scale"], mask.get("size", 0), mask.get("keep_first", 0), m.get("softcap") or 0.0, w.get("sink")).reshape(T, H * dv)
    if "g" in w:
        o = o * torch.sigmoid(h @ w["g"].T)
    return lin("o", o)


# ---- time mixing -----------------------------------------------------------------------------------------------------------------------

def previous_rows(h: torch.Tensor) -> torch.Tensor:
    """row t of the result is row t - 1 of h, row 0 is zero."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)


def shift_mix(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    """every entry moved by mu of the way towards the previous token's"""
    return h + (previous_rows(h) - h) * mu


def double_exponential_decay(z: torch.Tensor) -> torch.Tensor:
    return torch.exp(-torch.exp(z))


def bonus_recurrence(r, k, v, w, u) -> torch.Tensor:
    """r, k, w [T, H, dk], v [T, H, dv], u [H, dk].  Per head, S [dk, dv] from zero: o_t = sum_c r_t[c] (S[c, :] + u[c] k_t[c] v_t), and only then
    S[c, :] <- w_t[c] S[c, :] + k_t[c] v_t."""
    T, H, dk = r.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=F)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = (r[t][:, :, None] * (S + u[:, :, None] * kv)).sum(1)
        S = w[t][:, :, None] * S + kv
    return out


def time_mix_part(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T, H, n = h.shape[0], m["heads"], m["dim"]
    mix = {a: shift_mix(h, w["mu." + a]) for a in "rkvgw"}
    r, k, v = ((mix[a] @ w[a].T).view(T, H, n) for a in "rkv")
    z = torch.tanh(mix["w"] @ w["w1"].T) @ w["w2"].T + w["w0"]
    o = bonus_recurrence(r, k, v, double_exponential_decay(z).view(T, H, n), w["u"].view(H, n))
    o = rms(o, eps).reshape(T, H * n) * w["norm"]
    return (o * silu(mix["g"] @ w["g"].T)) @ w["o"].T


# ---- gated delta rule with a decay per key channel ------------------------------------------------------------------------------------

def short_conv(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """causal, per channel; x [T, C], taps [C, K], the last column multiplies the current token; zeros before the start"""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            src = t - (K - 1 - j)
            if src >= 0:
                y[t] += taps[:, j] * x[src]
    return y


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, beta, g) -> torch.Tensor:
    """q, k, g [T, H, dk], v [T, H, dv], beta [T, H].  Per head, S [dk, dv] from zero: S[c, :] <- g_t[c] S[c, :]; u = beta_t (v_t - S^T k_t);
    S <- S + k_t u^T; o_t = S^T q_t."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=F)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for t in range(T):
        S = S * g[t][:, :, None]
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def delta_part(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = lambda n: silu(short_conv(h @ w[n].T, w[n + ".conv"]))
    rep = H // G
    q = (unit(conv("q").view(T, G, dk)) * dk ** -0.5).repeat_interleave(rep, 1)
    k = unit(conv("k").view(T, G, dk)).repeat_interleave(rep, 1)
    v = conv("v").view(T, H, dv)
    beta = torch.sigmoid(h @ w["b"].T)
    z = ((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"].view(-1)).view(T, H, dk)
    g = torch.exp(-torch.exp(w["A_log"].view(H, 1)) * softplus(z))
    o = rms(delta_recurrence(q, k, v, beta, g), eps) * w["norm"]
    return (o.reshape(T, H * dv) * torch.sigmoid((h @ w["g1"].T) @ w["g2"].T)) @ w["o"].T


# ---- the decoder -----------------------------------------------------------------------------------------------------------------------

RIGHT = {"parallel": time_mix_part, "parallel_2": delta_part}


def dense_mlp(h: torch.Tensor, w: Dict[str, torch.Tensor], limit: float) -> torch.Tensor:
    return clamped_glu(h @ w["gate"].T, h @ w["up"].T, limit) @ w["down"].T


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens, trace: Optional[list] = None) -> torch.Tensor:
    """tokens: T ids of ONE sequence from position 0 -> logits [T, vocab] (float64).  `trace`, if a list, receives the residual stream
    after every layer."""
    W = {k: v.to(F) for k, v in weights.items() if v.is_floating_point()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        sub = lambda pre: {k[len(p + pre):]: v for k, v in W.items() if k.startswith(p + pre)}
        m = L["mixer"]
        y = m["left_scale"] * attention_part(x, sub("mix.left."), m["left"], eps) + m["right_scale"] * RIGHT[L["type"]](x, sub("mix.right."), m["right"], eps)
        x = x + rms(y, eps) * W[p + "norm1"]
        if L.get("mlp"):
            x = x + rms(dense_mlp(x, sub("mlp."), L["mlp"]["limit"]), eps) * W[p + "norm2"]
        if trace is not None:
            trace.append(x.clone())
    return (rms(x, eps) * W["final.norm"]) @ W["embed"].T


def greedy(cfg, weights, prompt, steps: int) -> List[int]:
    """Greedy continuation by re-running the whole sequence (slow, on purpose)."""
    ids = list(prompt)
    for _ in range(steps):
        ids.append(int(forward(cfg, weights, ids)[-1].argmax()))
    return ids[len(prompt):]
