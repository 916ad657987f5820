"""Plain CPU implementation of the Medirax language model, one function per mechanism.

TEST INFRASTRUCTURE ONLY: what the tests hold ``vui_b200``'s token-model path against.  It shares no code with the product,
keeps no cache (every call runs the whole sequence, the recurrence token by token) and computes in the dtype of the
weights it is given (float64 in the tests), so a difference from it is a difference of the product.

A Medirax block norms a residual row once and adds what both halves make of it: ``x' = x + M(n) + F(n)``, n = N(x), with M
windowed grouped-query attention or a gated delta rule and F an MLP with squared ReLU (F may be absent).  A run of layers
may be repeated; every repetition is a layer of its own that shares its weights with the others.
"""

from __future__ import annotations

import torch
from torch import Tensor

UNIT_EPS = 1e-6


def rms(x: Tensor, eps: float) -> Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x: Tensor, w: Tensor, eps: float) -> Tensor:
    """RMS norm whose gain is one plus the stored weight."""
    return rms(x, eps) * (1 + w)


def silu(x: Tensor) -> Tensor:
    return x / (1 + torch.exp(-x))


def softplus(x: Tensor) -> Tensor:
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def unit(x: Tensor) -> Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def causal_conv(x: Tensor, w: Tensor) -> Tensor:
    """x (T, C), w (C, taps): y[t, c] = sum_j w[c, taps - 1 - j] x[t - j, c], zeros before the start."""
    y = torch.zeros_like(x)
    taps = w.shape[1]
    for j in range(min(taps, x.shape[0])):
        y[j:] += x[: x.shape[0] - j] * w[:, taps - 1 - j]
    return y


def rotate_halves(x: Tensor, pos: Tensor, base: float, dims: int) -> Tensor:
    """x (..., T, D): component i is turned together with component i + dims/2 by pos * base**(-2i/dims), i < dims/2;
    components from dims on stay."""
    h = dims // 2
    f = base ** (-2.0 * torch.arange(h, dtype=torch.float64) / dims) if h else torch.zeros(0, dtype=torch.float64)
    a = pos.double()[:, None] * f
    c, s = a.cos().to(x.dtype), a.sin().to(x.dtype)
    u, v = x[..., :h], x[..., h:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def window_weights(scores: Tensor, window: int) -> Tensor:
    """scores (..., T, T) -> softmax over the keys j with 0 <= i - j < window."""
    T = scores.shape[-1]
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    s = scores.masked_fill((back < 0) | (back >= window), float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def cap(scores: Tensor, limit: float) -> Tensor:
    return limit * torch.tanh(scores / limit)


def split_heads(x: Tensor, n: int) -> Tensor:
    return x.reshape(x.shape[0], n, -1).transpose(0, 1)


def normed_query_keys(h: Tensor, W: dict, m: dict, eps: float, pos: Tensor) -> tuple[Tensor, Tensor]:
    """(heads, T, dim) and (kv_heads, T, dim): projected, rotated, then divided by their root mean square."""
    q = split_heads(h @ W["q"].T + W["q.b"], m["heads"])
    k = split_heads(h @ W["k"].T + W["k.b"], m["kv_heads"])
    r = m["rot"]
    return rms(rotate_halves(q, pos, r["base"], r["dims"]), eps), rms(rotate_halves(k, pos, r["base"], r["dims"]), eps)


def window_attention(h: Tensor, W: dict, m: dict, eps: float, pos: Tensor) -> Tensor:
    T, rep = h.shape[0], m["heads"] // m["kv_heads"]
    q, k = normed_query_keys(h, W, m, eps, pos)
    v = split_heads(h @ W["v"].T + W["v.b"], m["kv_heads"])
    k, v = k.repeat_interleave(rep, 0), v.repeat_interleave(rep, 0)
    p = window_weights(cap((q @ k.transpose(1, 2)) * m["scale"], m["softcap"]), m["mask"]["size"])
    return (p @ v).transpose(0, 1).reshape(T, -1) @ W["o"].T + W["o.b"]


def delta_rule(q: Tensor, k: Tensor, v: Tensor, decay: Tensor, beta: Tensor) -> Tensor:
    """q, k (H, T, D), v (H, T, V), decay and beta (H, T): the recurrence, one token after the other."""
    S = torch.zeros(q.shape[0], q.shape[2], v.shape[2], dtype=q.dtype)
    out = []
    for t in range(q.shape[1]):
        S = decay[:, t, None, None] * S
        kt = k[:, t, :, None]
        u = beta[:, t, None, None] * (v[:, t, None, :] - (S * kt).sum(1, keepdim=True))
        S = S + kt * u
        out.append((S * q[:, t, :, None]).sum(1))
    return torch.stack(out, dim=1)


def delta_gates(h: Tensor, W: dict) -> tuple[Tensor, Tensor]:
    """(decay, beta), each (heads, T)."""
    beta = 1 / (1 + torch.exp(-(h @ W["b"].T)))
    decay = torch.exp(-torch.exp(W["A_log"]) * softplus(h @ W["a"].T + W["dt_bias"]))
    return decay.T, beta.T


def delta_mixer(h: Tensor, W: dict, m: dict, eps: float) -> Tensor:
    T, H, rep = h.shape[0], m["heads"], m["heads"] // m["kv_heads"]
    q, k, v = (silu(causal_conv(h @ W[n].T, W[n + ".conv"])) for n in "qkv")
    q = unit(split_heads(q, m["kv_heads"])) * m["dim"] ** -0.5
    k = unit(split_heads(k, m["kv_heads"]))
    decay, beta = delta_gates(h, W)
    o = delta_rule(q.repeat_interleave(rep, 0), k.repeat_interleave(rep, 0), split_heads(v, H), decay, beta)
    o = rms(o, eps) * W["norm"] * split_heads(silu(h @ W["g"].T), H)
    return o.transpose(0, 1).reshape(T, -1) @ W["o"].T


def relu2_mlp(h: Tensor, W: dict) -> Tensor:
    return torch.clamp(h @ W["up"].T, min=0).square() @ W["down"].T


def block(x: Tensor, sd: dict, i: int, layer: dict, eps: float, pos: Tensor) -> Tensor:
    def part(prefix):
        return {k[len(prefix):]: t for k, t in sd.items() if k.startswith(prefix)}

    h = centred_norm(x, sd[f"l{i}.norm1"], eps)
    mix, m = part(f"l{i}.mix."), layer["mixer"]
    out = delta_mixer(h, mix, m, eps) if layer["type"] == "delta" else window_attention(h, mix, m, eps, pos)
    if layer["mlp"] is not None:
        out = out + relu2_mlp(h, part(f"l{i}.mlp."))
    return x + out


def runs(cfg: dict) -> list[int]:
    """Layer numbers in the order they are run."""
    n, lo = len(cfg["layers"]), cfg.get("loop")
    if not lo:
        return list(range(n))
    return [*range(lo["start"]), *list(range(lo["start"], lo["stop"])) * lo["times"], *range(lo["stop"], n)]


def forward(cfg: dict, sd: dict, tokens: Tensor, want=None, taps: list | None = None) -> Tensor:
    """Logits (len(want), vocab) of one whole sequence; ``taps`` collects the residual rows after every layer run."""
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(tokens))
    x = sd["embed"][tokens]
    for i in runs(cfg):
        x = block(x, sd, i, cfg["layers"][i], eps, pos)
        if taps is not None:
            taps.append(x)
    if want is not None:
        x = x[want]
    return centred_norm(x, sd["final.norm"], eps) @ sd["head"].T * cfg["logit_scale"]


def greedy(cfg: dict, sd: dict, prompt: list[int], n: int) -> list[int]:
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(forward(cfg, sd, torch.tensor(ids), want=[-1])[0].argmax()))
    return ids[len(prompt):]
