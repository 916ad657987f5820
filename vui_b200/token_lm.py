"""Token language models: configuration, weights, and how the weights are packed for the kernels.

A model is a list of layers, each a mixer and an MLP described by a small record of sizes and constants
(``LatentMixer``, ``ClampedGLU``); a design is a subclass of ``TokenLM`` that reads its configuration into these
records and names its tensors.  Packing depends on the records alone, so a design that combines the same mechanisms
with other names or in another order needs no packing of its own.
"""

from __future__ import annotations

import json
import os
from dataclasses import dataclass

import torch
from torch import Tensor

from . import _lib


@dataclass(frozen=True)
class LatentMixer:
    """Latent attention (VUIB_LM_MIX_LATENT): queries and keys/values through normed low-rank latents, ``rot_dims``
    of the ``rot_dim`` extra components of a head rotated by position, keys' rotated part shared by all heads."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int


@dataclass(frozen=True)
class ClampedGLU:
    """g = min(a, limit), u = clamp(b, +-limit): g * sigmoid(slope * g) * (u + shift) (VUIB_LM_MLP_CLAMPED_GLU)."""

    ff: int
    limit: float
    slope: float = 1.702
    shift: float = 1.0


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentMixer
    mlp: ClampedGLU | None


@dataclass(frozen=True)
class TokenLMConfig:
    vocab: int
    width: int
    norm_eps: float
    embed_scale: float
    layers: tuple[LayerSpec, ...]


def abi_layer(spec: LayerSpec) -> "_lib.VuibLmLayer":
    m, f = spec.mixer, spec.mlp
    return _lib.VuibLmLayer(
        _lib.LM_MIX_LATENT, _lib.LM_MLP_NONE if f is None else _lib.LM_MLP_CLAMPED_GLU, m.heads, m.dim, m.rot_dim,
        m.rot_dims, m.vdim, m.kv_rank, m.q_rank, f.ff if f else 0, m.scale, f.limit if f else 0.0,
        f.slope if f else 0.0, f.shift if f else 0.0)


def trig_table(base: float, dims: int, n: int) -> Tensor:
    """(n, dims / 2, 2) fp32 (cos, sin) of position * base**(-2i/dims), the angles in float64."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    ang = torch.arange(n, dtype=torch.float64)[:, None] * float(base) ** (-2.0 * i / dims)
    return torch.stack((ang.cos(), ang.sin()), dim=-1).float().contiguous()


def _place(shape, dtype, device, parts) -> Tensor:
    """Zeros of ``shape`` with blocks (row, column, row step, tensor) written in."""
    out = torch.zeros(shape, dtype=dtype, device=device)
    for r, c, step, t in parts:
        out[r:r + step * t.shape[0]:step, c:c + t.shape[1]] = t
    return out


def pack_layer(spec: LayerSpec, width: int, t: dict[str, Tensor], d: "_lib.VuibLmDims", dtype, device) -> dict[str, Tensor]:
    """The matrices of one layer as include/vuib200_lm.h describes them (VuibLmDims), from tensors by role: dq, uq, dkv,
    uk, uv, g, o, gate, up, down (matrices (out, in)) and the norms' vectors."""
    m, f = spec.mixer, spec.mlp
    H, hd = m.heads, m.dim + m.rot_dim
    t = {k: v.to(device) for k, v in t.items()}
    blocks = [(0, 0, 1, t["dq"]), (d.n_dq, 0, 1, t["dkv"][: m.kv_rank]), (d.n_dq + d.rp, 0, 1, t["dkv"][m.kv_rank:]),
              (d.n_kv, 0, 1, t["g"])]
    out_blocks = [(0, 0, 1, t["o"])]
    if f is not None:
        blocks += [(d.n_mlp, 0, 2, t["gate"]), (d.n_mlp + 1, 0, 2, t["up"])]
        out_blocks.append((0, d.off_y, 1, t["down"]))
    p = {"w_in": _place((d.n_in, d.k_in), dtype, device, blocks),
         "w_out": _place((d.n_out, d.k_out), dtype, device, out_blocks)}
    # absorbed queries: the key matrix of a head folded into its query rows, in float64
    uq = t["uq"].double().view(H, hd, m.q_rank)
    uk = t["uk"].double().view(H, m.dim, m.kv_rank)
    q = torch.zeros(H, d.dp, m.q_rank, dtype=torch.float64, device=device)
    q[:, : m.kv_rank] = uk.transpose(1, 2) @ uq[:, : m.dim]
    q[:, d.rp:d.rp + m.rot_dim] = uq[:, m.dim:]
    p["w_q"] = _place((d.n_q, d.k_q), dtype, device, [(0, 0, 1, q.view(H * d.dp, m.q_rank))])
    uv = torch.zeros(H, m.vdim, d.rp, dtype=dtype, device=device)
    uv[:, :, : m.kv_rank] = t["uv"].view(H, m.vdim, m.kv_rank)
    p["w_uv"] = uv
    if d.x_ok:
        hx = d.dimp + d.rotp
        xq = torch.zeros(H, hx, m.q_rank, dtype=dtype, device=device)
        xq[:, : m.dim] = uq[:, : m.dim]
        xq[:, d.dimp:d.dimp + m.rot_dim] = uq[:, m.dim:]
        p["w_xq"] = _place((d.n_xq, d.k_q), dtype, device, [(0, 0, 1, xq.view(H * hx, m.q_rank))])
        xk = torch.zeros(H, d.dimp, m.kv_rank, dtype=dtype, device=device)
        xk[:, : m.dim] = uk
        xv = torch.zeros(H, d.vdp, m.kv_rank, dtype=dtype, device=device)
        xv[:, : m.vdim] = t["uv"].view(H, m.vdim, m.kv_rank)
        p["w_xkv"] = _place((d.n_xkv, d.k_kv), dtype, device, [(0, 0, 1, xk.view(-1, m.kv_rank)),
                                                              (H * d.dimp, 0, 1, xv.view(-1, m.kv_rank))])
    for k in ("norm1_w", "norm1_b", "norm2_w", "norm2_b", "q_norm", "kv_norm"):
        if k in t:
            p[k] = t[k].float().contiguous()
    return p


class TokenLM:
    """Weights of a token model: tensors under the checkpoint's names, packed on the device for an engine on first use.
    ``dtype`` is bfloat16 (serving) or float32 (everything in 32 bits)."""

    architecture: str

    def __init__(self, config: TokenLMConfig, sd: dict[str, Tensor], device="cuda", dtype=torch.bfloat16):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype} is not supported: bfloat16 or float32")
        self.config, self.device, self.dtype = config, torch.device(device), dtype
        self.sd: dict[str, Tensor] = {}
        for name, shape in self.tensor_shapes(config).items():
            if name not in sd:
                raise KeyError(f"checkpoint lacks '{name}'")
            if tuple(sd[name].shape) != shape:
                raise ValueError(f"'{name}' has shape {tuple(sd[name].shape)}, expected {shape}")
            self.sd[name] = sd[name]
        self._packed: list[dict[str, Tensor]] | None = None
        self._head: dict[str, Tensor] | None = None

    # -- what a design provides -------------------------------------------------
    @classmethod
    def parse_config(cls, cfg: dict) -> TokenLMConfig:
        raise NotImplementedError

    @classmethod
    def tensor_shapes(cls, config: TokenLMConfig) -> dict[str, tuple[int, ...]]:
        raise NotImplementedError

    def layer_tensors(self, i: int) -> dict[str, Tensor]:
        """The layer's tensors by the roles ``pack_layer`` names."""
        raise NotImplementedError

    def head_tensors(self) -> dict[str, Tensor]:
        """embed, final_w, final_b, head."""
        raise NotImplementedError

    # -- constructors -------------------------------------------------------------
    @classmethod
    def from_checkpoint(cls, path: str, device="cuda", dtype=torch.bfloat16):
        """A folder with config.json and model.safetensors."""
        from safetensors.torch import load_file

        with open(os.path.join(path, "config.json")) as f:
            config = cls.parse_config(json.load(f))
        return cls(config, load_file(os.path.join(path, "model.safetensors")), device=device, dtype=dtype)

    @classmethod
    def random_init(cls, config: TokenLMConfig, seed: int = 0, device="cuda", dtype=torch.bfloat16, std: float = 0.02):
        """Seeded weights: matrices N(0, std), norm gains 1, biases 0, drawn in the order of ``tensor_shapes``."""
        dev = torch.device(device)
        g = torch.Generator(device=dev).manual_seed(seed)
        sd = {}
        for name, shape in cls.tensor_shapes(config).items():
            if len(shape) == 1:
                t = torch.zeros(shape, device=dev) if name.endswith(".b") else torch.ones(shape, device=dev)
            else:
                t = torch.empty(shape, device=dev).normal_(0.0, std, generator=g)
            sd[name] = t.to(torch.bfloat16)
        return cls(config, sd, device=device, dtype=dtype)

    # -- packed weights -------------------------------------------------------------
    def packed(self, dims: list) -> tuple[dict[str, Tensor], list[dict[str, Tensor]]]:
        """(head, layers) on the device; ``dims`` are the library's VuibLmDims, which depend on configuration and dtype
        alone, so the engines of a model share one packed copy."""
        if self._packed is None:
            c = self.config
            h = {k: v.to(self.device) for k, v in self.head_tensors().items()}
            rows, k = (c.vocab + 127) // 128 * 128, (c.width + 63) // 64 * 64
            self._head = {"embed": h["embed"].to(self.dtype).contiguous(),
                          "head": _place((rows, k), self.dtype, self.device, [(0, 0, 1, h["head"])]),
                          "final_w": h["final_w"].float().contiguous(), "final_b": h["final_b"].float().contiguous()}
            self._packed = [pack_layer(s, c.width, self.layer_tensors(i), dims[i], self.dtype, self.device)
                            for i, s in enumerate(c.layers)]
        return self._head, self._packed

    def weight_bytes_per_step(self) -> int:
        """Distinct weight bytes one decode step reads: every checkpoint matrix once, without the embedding table."""
        es = 2 if self.dtype == torch.bfloat16 else 4
        embed = self.head_tensors()["embed"]
        return sum(t.numel() * es for t in self.sd.values() if t.dim() == 2 and t is not embed)


class Vidotar(TokenLM):
    """Parallel blocks with two layer norms: latent attention with an output gate beside a clamped gated MLP.

    config.json: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` and ``layers``, each with ``type``, ``mixer``
    and ``mlp`` (or null)."""

    architecture = "Vidotar"

    @classmethod
    def parse_config(cls, cfg: dict) -> TokenLMConfig:
        layers = []
        for i, e in enumerate(cfg["layers"]):
            if e["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer '{e['type']}'")
            m, f = e["mixer"], e.get("mlp")
            if f is not None and f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward '{f['kind']}'")
            mixer = LatentMixer(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=m["q_rank"],
                                kv_rank=m["kv_rank"], scale=float(m["scale"]), rot_base=float(m["rot"]["base"]),
                                rot_dims=m["rot"]["dims"])
            layers.append(LayerSpec(mixer, None if f is None else ClampedGLU(ff=f["ff"], limit=float(f["limit"]))))
        return TokenLMConfig(vocab=cfg["vocab"], width=cfg["width"], norm_eps=float(cfg["norm"]["eps"]),
                             embed_scale=float(cfg["embedding"]["scale"]), layers=tuple(layers))

    @classmethod
    def tensor_shapes(cls, config: TokenLMConfig) -> dict[str, tuple[int, ...]]:
        w = config.width
        out: dict[str, tuple[int, ...]] = {"embed": (config.vocab, w)}
        for i, s in enumerate(config.layers):
            m, f, p = s.mixer, s.mlp, f"l{i}."
            for n in ("norm1", "norm2") if f is not None else ("norm1",):
                out[p + n] = out[p + n + ".b"] = (w,)
            x = p + "mix."
            out[x + "dq"] = (m.q_rank, w)
            out[x + "dq.norm"] = (m.q_rank,)
            out[x + "uq"] = (m.heads * (m.dim + m.rot_dim), m.q_rank)
            out[x + "dkv"] = (m.kv_rank + m.rot_dim, w)
            out[x + "dkv.norm"] = (m.kv_rank,)
            out[x + "uk"] = (m.heads * m.dim, m.kv_rank)
            out[x + "uv"] = (m.heads * m.vdim, m.kv_rank)
            out[x + "g"] = (m.heads * m.vdim, w)
            out[x + "o"] = (w, m.heads * m.vdim)
            if f is not None:
                out[p + "mlp.gate"] = out[p + "mlp.up"] = (f.ff, w)
                out[p + "mlp.down"] = (w, f.ff)
        out["final.norm"] = out["final.norm.b"] = (w,)
        out["head"] = (config.vocab, w)
        return out

    def layer_tensors(self, i: int) -> dict[str, Tensor]:
        p = f"l{i}."
        names = {"norm1_w": "norm1", "norm1_b": "norm1.b", "q_norm": "mix.dq.norm", "kv_norm": "mix.dkv.norm"}
        names.update({k: "mix." + k for k in ("dq", "uq", "dkv", "uk", "uv", "g", "o")})
        if self.config.layers[i].mlp is not None:
            names.update({"norm2_w": "norm2", "norm2_b": "norm2.b", "gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"})
        return {role: self.sd[p + n] for role, n in names.items()}

    def head_tensors(self) -> dict[str, Tensor]:
        return {"embed": self.sd["embed"], "final_w": self.sd["final.norm"], "final_b": self.sd["final.norm.b"],
                "head": self.sd["head"]}
