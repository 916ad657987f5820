"""Small seeded Medirax models for its tests: sizes that are multiples of nothing in particular, layers that differ from
one another, weights scaled so that every branch carries signal."""
import torch

from oracle import medirax_oracle as oracle
from tests.token_models import doubles
from vui_b200 import Medirax


def delta(heads=4, kv_heads=2, dim=24, vdim=20, conv=3):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attention(heads=4, kv_heads=2, dim=20, vdim=28, size=37, dims=12, base=700.0, scale=0.4, softcap=4.0):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
                                           "rot": {"base": base, "dims": dims}, "scale": scale, "softcap": softcap}}


def config(layers, width=90, vocab=131, eps=1e-5, logit_scale=0.7, loop=None):
    """``layers``: (mixer entry, MLP size or None)."""
    return {"architecture": "Medirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "loop": loop or {"start": 0, "stop": 0, "times": 1},
            "layers": [{**m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for m, ff in layers]}


CONFIGS = {
    "plain": config([(delta(), 72), (attention(), 72), (delta(), 40)], loop={"start": 0, "stop": 2, "times": 2}),
    # no MLP, one head, odd sizes, one tap and many, a window of one and one wider than the sequence, no and full rotation
    "mixed": config([(attention(heads=1, kv_heads=1, dim=7, vdim=9, size=1, dims=6, base=30.0), None),
                     (delta(heads=3, kv_heads=3, dim=11, vdim=7, conv=1), 33),
                     (attention(heads=3, kv_heads=3, dim=34, vdim=12, size=1000, dims=0, scale=0.2, softcap=30.0), 101),
                     (delta(heads=6, kv_heads=1, dim=40, vdim=52, conv=7), None),
                     (attention(heads=6, kv_heads=2, dim=16, vdim=16, size=64, dims=16, base=1e5), 16)],
                    width=77, vocab=203, eps=3e-3, logit_scale=1.6, loop={"start": 1, "stop": 4, "times": 2}),
    # more heads in a group than one MMA tile takes, heads wider than the fast forms take, columns in several blocks
    "wide": config([(attention(heads=34, kv_heads=2, dim=144, vdim=160, size=130, dims=64, scale=0.1, softcap=9.0), 200),
                    (delta(heads=2, kv_heads=1, dim=144, vdim=136, conv=4), 130),
                    (delta(heads=4, kv_heads=2, dim=128, vdim=72, conv=2), 64)], width=192, vocab=160,
                   loop={"start": 1, "stop": 3, "times": 1}),
}


def weights(cfg, seed=0):
    """bf16-valued tensors: matrices N(0, 1/fan_in), block gains around 0, biases around 0, decays from slow to fast."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in Medirax.tensor_shapes(Medirax.parse_config(cfg)).items():
        t, u = torch.randn(shape, generator=g), torch.rand(shape, generator=g)
        if name.endswith(".conv"):
            t = t * 0.7
        elif len(shape) == 2:
            t = t * (1.0 if name == "embed" else shape[1] ** -0.5)
        elif name.endswith("A_log"):
            t = u * 4.5 - 4.0
        elif name.endswith("dt_bias"):
            t = u * 3.0 - 2.5
        else:
            t = (1.0 if name.endswith("mix.norm") else 0.0) + 0.3 * t
        sd[name] = t.to(torch.bfloat16)
    return sd


def reference(cfg, sd, ids, want=None, taps=None):
    return oracle.forward(cfg, doubles(sd), torch.tensor(ids), want, taps)


def _apart(cfg, sd, layer, token, others):
    """The part of a token's normed embedding that is orthogonal to those of other tokens, scaled so that its product with
    the token's own is 1 (float64)."""
    h = oracle.centred_norm(sd["embed"].double(), sd[f"l{layer}.norm1"].double(), cfg["norm"]["eps"])
    q, _ = torch.linalg.qr(h[others].T)
    n = h[token] - q @ (q.T @ h[token])
    return n / (n @ h[token])


def point_attention(cfg, sd, needle, query, fillers, strength=40.0):
    """Layer 0's weights rewritten so that in every head the score of ``query`` with ``needle`` stands far out of all
    others, whatever lies between them: both have their largest component where no rotation reaches."""
    m = cfg["layers"][0]["mixer"]
    assert m["rot"]["dims"] < m["dim"]
    sd = {k: v.clone().float() for k, v in sd.items()}
    n, q = (_apart(cfg, sd, 0, t, [x for x in (needle, query, *fillers) if x != t]).float() for t in (needle, query))
    last = m["dim"] - 1
    sd["l0.mix.k"][last::m["dim"]] = strength * n
    sd["l0.mix.q"][last::m["dim"]] = strength * q
    sd["l0.mix.k.b"][:] = 0
    sd["l0.mix.q.b"][:] = 0
    return {k: v.to(torch.bfloat16) for k, v in sd.items()}


def point_delta(cfg, sd, needle, query, fillers, strength=40.0):
    """Layer 0's weights rewritten so that ``needle`` writes under a key of its own, which nothing in between overwrites,
    and ``query`` reads it: the first component of keys and queries, with no decay to speak of and no convolution in it."""
    m = cfg["layers"][0]["mixer"]
    sd = {k: v.clone().float() for k, v in sd.items()}
    n, q = (_apart(cfg, sd, 0, t, [x for x in (needle, query, *fillers) if x != t]).float() for t in (needle, query))
    for name, w in (("k", n), ("q", q)):
        sd[f"l0.mix.{name}"][0::m["dim"]] = strength * w
        sd[f"l0.mix.{name}.conv"][0::m["dim"]] = 0
        sd[f"l0.mix.{name}.conv"][0::m["dim"], -1] = 1
    sd["l0.mix.A_log"][:] = -9.0
    return {k: v.to(torch.bfloat16) for k, v in sd.items()}
