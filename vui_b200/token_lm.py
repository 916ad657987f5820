"""Token language models: configuration, weights, and how the weights are packed for the kernels.

A model is a list of layers, each a mixer and an MLP described by a small record of sizes and constants (``LatentMixer``,
``GroupedMixer``, ``DeltaMixer``; ``ClampedGLU``, ``SquaredReLU``), the form of its blocks, and the order in which the
layers run; a design is a subclass of ``TokenLM`` that reads its configuration into these records and names its tensors.
Packing depends on the records alone, so a design that combines the same mechanisms with other names or in another order
needs no packing of its own.
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
class GroupedMixer:
    """Grouped-query attention (VUIB_LM_MIX_GROUPED): heads / kv_heads query heads share a key/value head; the first
    ``rot_dims`` components are rotated, component i with i + rot_dims/2; ``qk_norm`` divides rotated queries and keys by
    their root mean square; scores are softcap * tanh(score / softcap) (0: as they are); ``window`` keys are seen, the
    query's own among them (0: all before it)."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int
    window: int = 0
    softcap: float = 0.0
    qk_norm: bool = True
    biases: bool = True       # on the query, key, value and output projections


@dataclass(frozen=True)
class DeltaMixer:
    """Gated delta rule (VUIB_LM_MIX_DELTA): causal convolutions of ``taps`` taps and silu on queries, keys and values,
    unit queries (times ``scale``) and keys, a state of (dim, vdim) per head with a decay and a step size per token, output
    norm and silu gate per head."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    scale: float
    unit_eps: float = 1e-6
    rot_dims = 0


@dataclass(frozen=True)
class ClampedGLU:
    """g = min(a, limit), u = clamp(b, +-limit): g * sigmoid(slope * g) * (u + shift) (VUIB_LM_MLP_CLAMPED_GLU)."""

    ff: int
    limit: float
    slope: float = 1.702
    shift: float = 1.0


@dataclass(frozen=True)
class SquaredReLU:
    """relu(a)**2 (VUIB_LM_MLP_RELU2)."""

    ff: int


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentMixer | GroupedMixer | DeltaMixer
    mlp: ClampedGLU | SquaredReLU | None


@dataclass(frozen=True)
class TokenLMConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[LayerSpec, ...]
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    block: str = "ln2"                        # "ln2": two layer norms per block, "rms": one RMS norm
    order: tuple[int, ...] | None = None      # layers as they are run, one may appear several times (None: each once)

    @property
    def runs(self) -> tuple[int, ...]:
        return tuple(range(len(self.layers))) if self.order is None else self.order

    @property
    def recurrent(self) -> bool:
        return any(isinstance(s.mixer, DeltaMixer) for s in self.layers)


def abi_config(c: TokenLMConfig, **sizes) -> "_lib.VuibLmConfig":
    """``sizes``: dtype, n_slots, max_seq, max_rows, max_prefill_rows."""
    return _lib.VuibLmConfig(vocab=c.vocab, width=c.width, n_layers=len(c.runs),
                             block={"ln2": _lib.LM_BLOCK_LN2, "rms": _lib.LM_BLOCK_RMS}[c.block], norm_eps=c.norm_eps,
                             embed_scale=c.embed_scale, logit_scale=c.logit_scale, **sizes)


def abi_layer(spec: LayerSpec) -> "_lib.VuibLmLayer":
    m, f = spec.mixer, spec.mlp
    out = _lib.VuibLmLayer(heads=m.heads, dim=m.dim, rot_dims=m.rot_dims, vdim=m.vdim, scale=m.scale)
    if isinstance(m, LatentMixer):
        out.mixer, out.rot_dim, out.kv_rank, out.q_rank = _lib.LM_MIX_LATENT, m.rot_dim, m.kv_rank, m.q_rank
    elif isinstance(m, GroupedMixer):
        out.mixer, out.kv_heads, out.window = _lib.LM_MIX_GROUPED, m.kv_heads, m.window
        out.softcap, out.qk_norm = m.softcap, int(m.qk_norm)
    else:
        out.mixer, out.kv_heads, out.taps, out.unit_eps = _lib.LM_MIX_DELTA, m.kv_heads, m.taps, m.unit_eps
    if isinstance(f, ClampedGLU):
        out.mlp, out.ff, out.mlp_limit, out.mlp_slope, out.mlp_shift = _lib.LM_MLP_CLAMPED_GLU, f.ff, f.limit, f.slope, f.shift
    elif isinstance(f, SquaredReLU):
        out.mlp, out.ff = _lib.LM_MLP_RELU2, f.ff
    return out


def abi_layers(c: TokenLMConfig):
    return (_lib.VuibLmLayer * len(c.runs))(*[abi_layer(c.layers[i]) for i in c.runs])


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
    """The tensors of one layer as include/vuib200_lm.h describes them (VuibLmDims), from tensors by role."""
    t = {k: v.to(device) for k, v in t.items()}
    pack = {LatentMixer: _pack_latent, GroupedMixer: _pack_grouped, DeltaMixer: _pack_delta}[type(spec.mixer)]
    p = pack(spec, t, d, dtype, device)
    for k in ("norm1_w", "norm1_b", "norm2_w", "norm2_b", "q_norm", "kv_norm"):
        if k in t:
            p[k] = t[k].float().contiguous()
    return p


def _head_blocks(w: Tensor, heads: int, row0: int, padded: int, perm=None):
    """Blocks for ``_place``: every head's rows (or, for a vector as one column, entries) at its padded place."""
    for h, x in enumerate(w.view(heads, -1, w.shape[1]).unbind(0)):
        yield row0 + h * padded, 0, 1, x if perm is None else x[perm]


def _pair_order(dim: int, rot_dims: int) -> list[int]:
    """Components of a head with the members of each rotated pair next to each other."""
    half = rot_dims // 2
    return [c for i in range(half) for c in (i, i + half)] + list(range(rot_dims, dim))


def _out_matrix(spec: LayerSpec, t: dict[str, Tensor], d: "_lib.VuibLmDims", dtype, device) -> Tensor:
    """w_out of a layer whose mixer leaves its heads at padded places."""
    m = spec.mixer
    blocks = [(0, h * d.vdp, 1, t["o"][:, h * m.vdim:(h + 1) * m.vdim]) for h in range(m.heads)]
    if spec.mlp is not None:
        blocks.append((0, d.off_y, 1, t["down"]))
    return _place((d.n_out, d.k_out), dtype, device, blocks)


def _pack_grouped(spec: LayerSpec, t: dict[str, Tensor], d: "_lib.VuibLmDims", dtype, device) -> dict[str, Tensor]:
    """Roles q, k, v, o, up, down and, with biases, q_b, k_b, v_b, o_b."""
    m = spec.mixer
    perm = _pair_order(m.dim, m.rot_dims)

    def rows(q, k, v):
        return [*_head_blocks(q, m.heads, 0, d.dimp, perm), *_head_blocks(k, m.kv_heads, d.n_key, d.dimp, perm),
                *_head_blocks(v, m.kv_heads, d.n_value, d.vdp)]

    blocks = rows(t["q"], t["k"], t["v"])
    if spec.mlp is not None:
        blocks.append((d.n_mlp, 0, 1, t["up"]))
    p = {"w_in": _place((d.n_in, d.k_in), dtype, device, blocks), "w_out": _out_matrix(spec, t, d, dtype, device)}
    if m.biases:
        p["b_in"] = _place((d.n_raw, 1), torch.float32, device, rows(*[t[k + "_b"][:, None].float() for k in "qkv"])).view(-1)
        p["b_out"] = _place((d.n_out, 1), torch.float32, device, [(0, 0, 1, t["o_b"][:, None].float())]).view(-1)
    return p


def _pack_delta(spec: LayerSpec, t: dict[str, Tensor], d: "_lib.VuibLmDims", dtype, device) -> dict[str, Tensor]:
    """Roles q, k, v, q_conv, k_conv, v_conv, b (step size), a (decay), A_log, dt_bias, g, head_norm, o, up, down."""
    m = spec.mixer

    def rows(q, k, v):
        return [*_head_blocks(q, m.kv_heads, 0, d.dimp), *_head_blocks(k, m.kv_heads, d.n_key, d.dimp),
                *_head_blocks(v, m.heads, d.n_value, d.vdp)]

    blocks = [*rows(t["q"], t["k"], t["v"]), (d.n_ab, 0, 1, t["b"]), (d.n_ab + m.heads, 0, 1, t["a"]),
              *_head_blocks(t["g"], m.heads, d.n_raw, d.vdp)]
    if spec.mlp is not None:
        blocks.append((d.n_mlp, 0, 1, t["up"]))
    conv = _place((d.n_ab, m.taps), torch.float32, device, rows(*[t[k + "_conv"].float() for k in "qkv"]))
    return {"w_in": _place((d.n_in, d.k_in), dtype, device, blocks), "w_out": _out_matrix(spec, t, d, dtype, device),
            "conv": conv.t().contiguous(), "neg_a": -torch.exp(t["A_log"].float()), "dt_bias": t["dt_bias"].float().contiguous(),
            "head_norm": _place((d.vdp, 1), torch.float32, device, [(0, 0, 1, t["head_norm"][:, None].float())]).view(-1)}


def _pack_latent(spec: LayerSpec, t: dict[str, Tensor], d: "_lib.VuibLmDims", dtype, device) -> dict[str, Tensor]:
    """Roles dq, uq, dkv, uk, uv, g, o, gate, up, down (matrices (out, in))."""
    m, f = spec.mixer, spec.mlp
    H, hd = m.heads, m.dim + m.rot_dim
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
        """embed, final_w, head and, in blocks of layer norms, final_b."""
        raise NotImplementedError

    @classmethod
    def random_vector(cls, name: str, shape: tuple[int, ...], generator) -> Tensor:
        """A vector of a randomly initialised model: norm gains 1, biases 0."""
        dev = generator.device
        return torch.zeros(shape, device=dev) if name.endswith(".b") else torch.ones(shape, device=dev)

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
        """Seeded weights: matrices N(0, std), vectors by ``random_vector``, drawn in the order of ``tensor_shapes``."""
        dev = torch.device(device)
        g = torch.Generator(device=dev).manual_seed(seed)
        sd = {}
        for name, shape in cls.tensor_shapes(config).items():
            if len(shape) == 1:
                t = cls.random_vector(name, shape, g)
            else:
                t = torch.empty(shape, device=dev).normal_(0.0, std, generator=g)
            sd[name] = t.to(torch.bfloat16)
        return cls(config, sd, device=device, dtype=dtype)

    # -- packed weights -------------------------------------------------------------
    def packed(self, dims: list) -> tuple[dict[str, Tensor], list[dict[str, Tensor]]]:
        """(head, layers) on the device; ``dims`` are the library's VuibLmDims of the layers (None: the layer does not run), of
        which what a matrix is packed by depends on configuration and dtype alone, so the engines of a model share one
        packed copy."""
        if self._packed is None:
            c = self.config
            h = {k: v.to(self.device) for k, v in self.head_tensors().items()}
            rows, k = (c.vocab + 127) // 128 * 128, (c.width + 63) // 64 * 64
            self._head = {"embed": h["embed"].to(self.dtype).contiguous(),
                          "head": _place((rows, k), self.dtype, self.device, [(0, 0, 1, h["head"])]),
                          **{k: h[k].float().contiguous() for k in ("final_w", "final_b") if k in h}}
            self._packed = [{} if dims[i] is None else pack_layer(s, c.width, self.layer_tensors(i), dims[i], self.dtype, self.device)
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


class Medirax(TokenLM):
    """Parallel blocks with one RMS norm: windowed grouped-query attention or a gated delta rule beside an MLP with squared
    ReLU; a stretch of layers may run several times with the same weights.

    config.json: ``vocab``, ``width``, ``norm.eps``, ``logit_scale``, ``loop`` (start, stop, times; may be absent) and
    ``layers``, each with ``type`` ("attention" or "delta"), ``mixer`` and ``mlp`` (or null)."""

    architecture = "Medirax"

    @classmethod
    def parse_config(cls, cfg: dict) -> TokenLMConfig:
        layers = []
        for i, e in enumerate(cfg["layers"]):
            m, f = e["mixer"], e.get("mlp")
            if f is not None and f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward '{f['kind']}'")
            if m["heads"] % m["kv_heads"]:
                raise ValueError(f"layer {i}: {m['heads']} heads do not share {m['kv_heads']} key heads evenly")
            sizes = {k: m[k] for k in ("heads", "kv_heads", "dim", "vdim")}
            if e["type"] == "attention":
                mixer = GroupedMixer(**sizes, scale=float(m["scale"]), rot_base=float(m["rot"]["base"]), rot_dims=m["rot"]["dims"],
                                     window=m["mask"]["size"], softcap=float(m["softcap"]))
            elif e["type"] == "delta":
                mixer = DeltaMixer(**sizes, taps=m["conv"], scale=m["dim"] ** -0.5)
            else:
                raise ValueError(f"layer {i}: unknown mixer '{e['type']}'")
            layers.append(LayerSpec(mixer, None if f is None else SquaredReLU(ff=f["ff"])))
        order = None
        if cfg.get("loop"):
            start, stop, times = (cfg["loop"][k] for k in ("start", "stop", "times"))
            if not 0 <= start <= stop <= len(layers) or times < 0:
                raise ValueError(f"loop {cfg['loop']} does not fit {len(layers)} layers")
            order = (*range(start), *(tuple(range(start, stop)) * times), *range(stop, len(layers)))
        return TokenLMConfig(vocab=cfg["vocab"], width=cfg["width"], norm_eps=float(cfg["norm"]["eps"]),
                             logit_scale=float(cfg["logit_scale"]), block="rms", layers=tuple(layers), order=order)

    @classmethod
    def tensor_shapes(cls, config: TokenLMConfig) -> dict[str, tuple[int, ...]]:
        w = config.width
        out: dict[str, tuple[int, ...]] = {"embed": (config.vocab, w)}
        for i, s in enumerate(config.layers):
            m, p = s.mixer, f"l{i}."
            x = p + "mix."
            out[p + "norm1"] = (w,)
            if isinstance(m, GroupedMixer):
                for n, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                    out[x + n], out[x + n + ".b"] = (rows, w), (rows,)
                out[x + "o"], out[x + "o.b"] = (w, m.heads * m.vdim), (w,)
            else:
                for n, rows in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim)):
                    out[x + n], out[x + n + ".conv"] = (rows, w), (rows, m.taps)
                out[x + "b"] = out[x + "a"] = (m.heads, w)
                out[x + "A_log"] = out[x + "dt_bias"] = (m.heads,)
                out[x + "norm"] = (m.vdim,)
                out[x + "g"] = (m.heads * m.vdim, w)
                out[x + "o"] = (w, m.heads * m.vdim)
            if s.mlp is not None:
                out[p + "mlp.up"], out[p + "mlp.down"] = (s.mlp.ff, w), (w, s.mlp.ff)
        out["final.norm"] = (w,)
        out["head"] = (config.vocab, w)
        return out

    @classmethod
    def random_vector(cls, name: str, shape: tuple[int, ...], generator) -> Tensor:
        """Gains are stored around zero, but for the delta rule's output norm; decays from slow to fast."""
        u = torch.rand(shape, device=generator.device, generator=generator)
        if name.endswith("A_log"):
            return u * 4 - 4
        if name.endswith("dt_bias"):
            return u * 2 - 3
        return torch.ones_like(u) if name.endswith("mix.norm") else torch.zeros_like(u)

    def layer_tensors(self, i: int) -> dict[str, Tensor]:
        p, s = f"l{i}.", self.config.layers[i]
        if isinstance(s.mixer, GroupedMixer):
            names = {k: "mix." + k for k in "qkvo"} | {k + "_b": f"mix.{k}.b" for k in "qkvo"}
        else:
            names = {k: "mix." + k for k in ("q", "k", "v", "o", "b", "a", "g", "A_log", "dt_bias")}
            names |= {k + "_conv": f"mix.{k}.conv" for k in "qkv"} | {"head_norm": "mix.norm"}
        if s.mlp is not None:
            names |= {"up": "mlp.up", "down": "mlp.down"}
        out = {role: self.sd[p + n] for role, n in names.items()}
        out["norm1_w"] = 1.0 + self.sd[p + "norm1"].float()
        return out

    def head_tensors(self) -> dict[str, Tensor]:
        return {"embed": self.sd["embed"], "final_w": 1.0 + self.sd["final.norm"].float(), "head": self.sd["head"]}
