"""Small seeded Vidotar models for the token-model tests: sizes that are multiples of nothing in particular, layers that
differ from one another, weights scaled so that every branch carries signal."""
import torch

from oracle import vidotar_oracle as oracle
from vui_b200 import Vidotar


def mixer(heads=3, dim=20, rot_dim=12, vdim=24, q_rank=40, kv_rank=26, scale=None, base=700.0, dims=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
            "scale": scale if scale is not None else (dim + rot_dim) ** -0.5,
            "rot": {"base": base, "dims": rot_dim if dims is None else dims}}


def config(layers, width=90, vocab=131, eps=1e-5, scale=1.7):
    return {"architecture": "Vidotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": [{"type": "latent_attention", "mixer": m,
                        "mlp": None if ff is None else {"kind": "dense", "ff": ff[0], "limit": ff[1]}} for m, ff in layers]}


CONFIGS = {
    "plain": config([(mixer(), (72, 1.5)), (mixer(), (72, 1.5))]),
    # no MLP, one head, odd sizes, other bases and scales from layer to layer
    "mixed": config([(mixer(heads=1, dim=7, rot_dim=4, vdim=9, q_rank=11, kv_rank=17, base=30.0), None),
                     (mixer(heads=5, dim=33, rot_dim=10, vdim=13, q_rank=65, kv_rank=40, base=1e5, scale=0.31), (101, 0.4)),
                     (mixer(heads=2, dim=16, rot_dim=16, vdim=16, q_rank=16, kv_rank=16), (16, 3.0))],
                    width=77, vocab=203, eps=3e-3, scale=0.6),
    # more heads than one MMA tile of them, latents wider than the models above, part of the extra dimensions rotated
    "wide": config([(mixer(heads=19, dim=24, rot_dim=20, vdim=40, q_rank=96, kv_rank=152, dims=8), (200, 2.0)),
                    (mixer(heads=18, dim=48, rot_dim=32, vdim=72, q_rank=130, kv_rank=272), (130, 1.0))], width=192, vocab=160),
}


def weights(cfg, seed=0):
    """bf16-valued tensors: matrices N(0, 1/fan_in) with a little more on the MLP's inputs (so that both clamps act),
    norm gains around 1, biases around 0."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in Vidotar.tensor_shapes(Vidotar.parse_config(cfg)).items():
        t = torch.randn(shape, generator=g)
        if len(shape) == 2:
            t = t * (1.0 if name == "embed" else shape[1] ** -0.5)
            if ".mlp.gate" in name or ".mlp.up" in name:
                t = t * 1.8
        else:
            t = 0.2 * t if name.endswith(".b") else 1.0 + 0.3 * t
        sd[name] = t.to(torch.bfloat16)
    return sd


def doubles(sd):
    return {k: v.double() for k, v in sd.items()}


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rel_err(got, want):
    """Per row: RMS of the difference of the logits, their means taken off, over the RMS of the wanted ones."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean()**0.5


def reference(cfg, sd, ids, want=None):
    return oracle.forward(cfg, doubles(sd), torch.tensor(ids), want)


def point_at(cfg, sd, layer, needle, query, strength=3.0):
    """Rewrite the layer's weights so that ``query``'s score with ``needle`` stands far out of all others: a direction
    of its own through each of the four matrices on the way from a token to its score."""
    m = cfg["layers"][layer]["mixer"]
    sd = {k: v.clone().float() for k, v in sd.items()}
    eps, p = cfg["norm"]["eps"], f"l{layer}."
    x = sd["embed"][[needle, query]] * cfg["embedding"]["scale"]
    h = oracle.layer_norm(x.double(), sd[p + "norm1"].double(), sd[p + "norm1.b"].double(), eps).float()
    n, q = h[0] - h[1] * (h[0] @ h[1]) / (h[1] @ h[1]), h[1] - h[0] * (h[0] @ h[1]) / (h[0] @ h[0])
    sd[p + "mix.dkv"][0] = 4 * m["kv_rank"] ** 0.5 * n / (n @ h[0])
    sd[p + "mix.dq"][0] = 4 * m["q_rank"] ** 0.5 * q / (q @ h[1])
    sd[p + "mix.dkv.norm"][0] = sd[p + "mix.dq.norm"][0] = 1.0
    hd = m["dim"] + m["rot_dim"]
    for i in range(m["heads"]):
        sd[p + "mix.uk"][i * m["dim"], 0] = strength
        sd[p + "mix.uq"][i * hd, 0] = strength
    return {k: v.to(torch.bfloat16) for k, v in sd.items()}
