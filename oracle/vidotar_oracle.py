"""Plain CPU implementation of the Vidotar language model, one function per mechanism.

TEST INFRASTRUCTURE ONLY: what the tests hold ``vui_b200``'s token-model path against.  It shares no code with the product,
keeps no cache (every call attends over the whole sequence) and computes in the dtype of the weights it is given
(float64 in the tests), so a difference from it is a difference of the product.

A Vidotar block reads one residual row x twice and adds both results at once:
``x' = x + A(LN1(x)) + F(LN2(x))`` with A latent attention and F a clamped gated MLP (F may be absent).
"""

from __future__ import annotations

import torch
from torch import Tensor

SIGMOID_SLOPE = 1.702


def layer_norm(x: Tensor, w: Tensor, b: Tensor, eps: float) -> Tensor:
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def rms_norm(x: Tensor, w: Tensor, eps: float) -> Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotate_pairs(x: Tensor, pos: Tensor, base: float, dims: int) -> Tensor:
    """x (..., T, D): components (2i, 2i+1), i < dims/2, turned by pos * base**(-2i/dims); the rest unchanged."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    ang = pos.double()[:, None] * base ** (-2.0 * i / dims)
    cos, sin = ang.cos().to(x.dtype), ang.sin().to(x.dtype)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def causal_softmax(scores: Tensor) -> Tensor:
    """scores (..., T, T) -> weights over keys j <= i."""
    T = scores.shape[-1]
    keep = torch.ones(T, T, dtype=torch.bool).tril()
    s = scores.masked_fill(~keep, float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def latent_queries(h: Tensor, W: dict, m: dict, eps: float, pos: Tensor) -> tuple[Tensor, Tensor]:
    """(H, T, dim) plain and (H, T, rot_dim) rotated query parts."""
    T, H = h.shape[0], m["heads"]
    cq = rms_norm(h @ W["dq"].T, W["dq.norm"], eps)
    q = (cq @ W["uq"].T).reshape(T, H, m["dim"] + m["rot_dim"]).transpose(0, 1)
    return q[..., : m["dim"]], rotate_pairs(q[..., m["dim"]:], pos, m["rot"]["base"], m["rot"]["dims"])


def latent_keys(h: Tensor, W: dict, m: dict, eps: float, pos: Tensor) -> tuple[Tensor, Tensor]:
    """What a cache would hold per position: the normed latent (T, kv_rank) and the shared rotated key (T, rot_dim)."""
    a = h @ W["dkv"].T
    c = rms_norm(a[:, : m["kv_rank"]], W["dkv.norm"], eps)
    return c, rotate_pairs(a[:, m["kv_rank"]:], pos, m["rot"]["base"], m["rot"]["dims"])


def latent_attention(h: Tensor, W: dict, m: dict, eps: float, pos: Tensor) -> Tensor:
    T, H = h.shape[0], m["heads"]
    qn, qr = latent_queries(h, W, m, eps, pos)
    c, kr = latent_keys(h, W, m, eps, pos)
    kn = (c @ W["uk"].T).reshape(T, H, m["dim"]).transpose(0, 1)
    v = (c @ W["uv"].T).reshape(T, H, m["vdim"]).transpose(0, 1)
    p = causal_softmax((qn @ kn.transpose(1, 2) + qr @ kr.T) * m["scale"])
    o = (p @ v).transpose(0, 1).reshape(T, H * m["vdim"])
    return (o * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


def clamped_mlp(h: Tensor, W: dict, limit: float) -> Tensor:
    g = (h @ W["gate"].T).clamp(max=limit)
    u = (h @ W["up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(SIGMOID_SLOPE * g) * (u + 1)) @ W["down"].T


def parallel_block(x: Tensor, sd: dict, i: int, layer: dict, eps: float, pos: Tensor) -> Tensor:
    p = f"l{i}."
    mix = {k[len(p) + 4:]: t for k, t in sd.items() if k.startswith(p + "mix.")}
    out = latent_attention(layer_norm(x, sd[p + "norm1"], sd[p + "norm1.b"], eps), mix, layer["mixer"], eps, pos)
    if layer["mlp"] is not None:
        mlp = {k[len(p) + 4:]: t for k, t in sd.items() if k.startswith(p + "mlp.")}
        out = out + clamped_mlp(layer_norm(x, sd[p + "norm2"], sd[p + "norm2.b"], eps), mlp, layer["mlp"]["limit"])
    return x + out


def forward(cfg: dict, sd: dict, tokens: Tensor, want=None, taps: list | None = None) -> Tensor:
    """Logits (len(want), vocab) of one whole sequence; ``taps`` collects the residual rows after every layer."""
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(tokens))
    x = sd["embed"][tokens] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        x = parallel_block(x, sd, i, layer, eps, pos)
        if taps is not None:
            taps.append(x)
    if want is not None:
        x = x[want]
    return layer_norm(x, sd["final.norm"], sd["final.norm.b"], eps) @ sd["head"].T


def greedy(cfg: dict, sd: dict, prompt: list[int], n: int) -> list[int]:
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(forward(cfg, sd, torch.tensor(ids), want=[-1])[0].argmax()))
    return ids[len(prompt):]
