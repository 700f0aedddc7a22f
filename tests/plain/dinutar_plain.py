"""A plain, slow implementation of the Dinutar architecture on whole sequences: no cache, no state carried between
calls, one function per mechanism, float64 by default.  It shares no code with the package; it reads the raw
configuration dictionary and the tensors by their names in the checkpoint.

Notation: T tokens, W the model's width; x [T, W]; positions are 0 .. T-1.
"""
from __future__ import annotations

import math
from typing import Dict, Optional

import torch

DT = torch.float64


def rms_norm(x: torch.Tensor, weight: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps), times the weight where there is one."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def bigram_rows(tokens, bigram: dict):
    """Row of every token in the bigram table: a hash of (the token before, the token), or for a sequence's first token
    the row behind the hashed ones."""
    n = bigram["buckets"]
    rows = []
    for t, tok in enumerate(tokens):
        rows.append(n if t == 0 else (int(tokens[t - 1]) * bigram["mul_prev"] + int(tok) * bigram["mul_cur"]) % n)
    return rows


def embedding(cfg: dict, w: Dict[str, torch.Tensor], tokens) -> torch.Tensor:
    """norm(table[token] * scale + bigram[row])."""
    emb = cfg.get("embedding") or {}
    x = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)] * emb.get("scale", 1.0)
    if emb.get("bigram"):
        x = x + w["bigram"][torch.as_tensor(bigram_rows(tokens, emb["bigram"]), dtype=torch.long)]
    return rms_norm(x, w["embed.norm"], cfg["norm"]["eps"])


def frequencies(rot: dict) -> torch.Tensor:
    """base^(-2i/dims) for i < dims/2; with ``scaling`` every frequency is blended with itself / factor: the fast ones
    (many turns over ``original`` positions) stay, the slow ones are divided, a ramp over i lies between."""
    dims, base = rot["dims"], float(rot["base"])
    i = torch.arange(dims // 2, dtype=DT)
    f = torch.pow(torch.tensor(base, dtype=DT), -2.0 * i / dims)
    sc = rot.get("scaling")
    if sc:
        def place(turns: float) -> float:            # the (fractional) i whose wave makes that many turns
            return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
        lo = max(math.floor(place(sc["fast"])), 0)
        hi = min(math.ceil(place(sc["slow"])), dims - 1)
        ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        f = f / sc["factor"] * ramp + f * (1.0 - ramp)
    return f


def magnitude(rot: dict) -> float:
    """What cos and sin are multiplied by: 0.1 ln(factor) + 1 where the frequencies are scaled."""
    sc = rot.get("scaling")
    return 0.1 * math.log(sc["factor"]) + 1.0 if sc else 1.0


def rotate_half(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, d]: columns i and i + dims/2 (i < dims/2) are a pair turned by p * f_i (and multiplied by the
    magnitude); columns from dims on pass."""
    if not rot or not rot.get("dims"):
        return x
    T, dims = x.shape[0], rot["dims"]
    a = torch.arange(T, dtype=DT)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(a)[:, None, :] * magnitude(rot), torch.sin(a)[:, None, :] * magnitude(rot)
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def causal_softmax(s: torch.Tensor) -> torch.Tensor:
    """Rows of s [T, T]: softmax over the columns up to the row's own."""
    T = s.shape[0]
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def latent_rows(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float):
    """(latent [T, rank], turned key part [T, rot_dim]) of a layer with a down projection."""
    R, dr = m["kv_rank"], m["rot_dim"]
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :R], w[p + "dkv.norm"], eps)
    return c, rotate_half(down[:, R:].view(h.shape[0], 1, dr), m.get("rot"))[:, 0]


def latent_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, rows) -> torch.Tensor:
    """``rows``: the latents and turned key parts this layer attends to (its own or another layer's)."""
    T = h.shape[0]
    H, d, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, k_turn = rows
    q = (h @ w[p + "q"].T).view(T, H, d + dr)
    q_plain, q_turn = q[..., :d], rotate_half(q[..., d:], m.get("rot"))
    k_plain = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    out = []
    for i in range(H):
        s = (q_plain[:, i] @ k_plain[:, i].T + q_turn[:, i] @ k_turn.T) * m["scale"]
        out.append(causal_softmax(s) @ v[:, i])
    return torch.stack(out, dim=1).reshape(T, H * dv) @ w[p + "o"].T


def retention_recurrence(q, k, v, decay, state: Optional[torch.Tensor] = None):
    """q, k [T, H, d], v [T, H, dv], decay [H]: S <- decay S + k v^T; o = S^T q.  Returns (o [T, H, dv], S)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hcv,hc->hv", S, q[t])
    return out, S


def retention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = rotate_half((h @ w[p + "q"].T).view(T, H, d), m.get("rot"))
    k = rotate_half((h @ w[p + "k"].T).view(T, H, d), m.get("rot")) * d ** -0.5
    v = (h @ w[p + "v"].T).view(T, H, dv)
    o, _ = retention_recurrence(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    o = rms_norm(o, None, eps).reshape(T, H * dv)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def feed_forward(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (torch.relu(h @ w[p + "up"].T) ** 2) @ w[p + "down"].T


def joined(x: torch.Tensor, y: torch.Tensor, w: Dict[str, torch.Tensor], p: str, which: int, alpha: float, eps: float) -> torch.Tensor:
    """norm(alpha x + scale * y): a sublayer's output, scaled channel by channel, enters the sum that is normed."""
    return rms_norm(alpha * x + w[f"{p}ls{which}"] * y, w[f"{p}norm{which}"], eps)


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, taps: Optional[dict] = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence.  ``taps``: receives "streams" (x after every layer)."""
    w = {k: v.to(DT) if v.is_floating_point() else v for k, v in w.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = embedding(cfg, w, tokens)
    rows_of = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "retention":
            y = retention(x, w, p + "mix.", m, eps)
        elif layer["type"] == "latent_attention":
            if m.get("kv_from") is None:
                rows_of[i] = latent_rows(x, w, p + "mix.", m, eps)
                rows = rows_of[i]
            else:
                rows = rows_of[m["kv_from"]]
            y = latent_attention(x, w, p + "mix.", m, rows)
        else:
            raise ValueError(layer["type"])
        x = joined(x, y, w, p, 1, alpha, eps)
        if layer.get("mlp") is not None:
            x = joined(x, feed_forward(x, w, p + "mlp."), w, p, 2, alpha, eps)
        if taps is not None:
            taps.setdefault("streams", []).append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(cfg: dict, w: Dict[str, torch.Tensor], prompt, n_new: int):
    """(the n_new tokens greedy decoding appends, the gap between the two best logits at every choice)."""
    ids, out, gaps = list(prompt), [], []
    for _ in range(n_new):
        top = torch.topk(forward(cfg, w, ids)[-1], 2)
        out.append(int(top.indices[0]))
        gaps.append(float(top.values[0] - top.values[1]))
        ids.append(out[-1])
    return out, gaps
