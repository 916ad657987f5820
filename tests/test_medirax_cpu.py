"""The Medirax model without a GPU: its oracle on hand values, configuration and weights, packing against the oracle's
mechanisms, what a mistake in a mechanism does to the logits, and the library's host checks."""
import ctypes as C
import json
import os

import pytest
import torch

from oracle import medirax_oracle as oracle
from tests import medirax_models as mm
from tests import token_models as tm
from vui_b200 import Medirax, _lib, load_model, registry
from vui_b200.token_lm import DeltaMixer, GroupedMixer, abi_config, abi_layers, pack_layer

D = torch.float64


def _handle(cfg, dtype=_lib.LM_BF16, **kw):
    c = Medirax.parse_config(cfg)
    a = abi_config(c, **{**dict(dtype=dtype, n_slots=3, max_seq=256, max_rows=2, max_prefill_rows=64), **kw})
    h = C.c_void_p()
    return _lib.load_lm().vuib_lm_create(C.byref(a), abi_layers(c), C.byref(h)), h


def _dims(h, n):
    out = [_lib.VuibLmDims() for _ in range(n)]
    for i, d in enumerate(out):
        assert _lib.load_lm().vuib_lm_layer_dims(h, i, C.byref(d)) == 0
    return out


# ------------------------------------------------------------------------------------------------ the oracle itself
def test_oracle_mechanisms_on_hand_values():
    t = lambda *v: torch.tensor(v, dtype=D)  # noqa: E731
    assert torch.allclose(oracle.centred_norm(t(3.0, 4.0), t(0.0, 1.0), 0.5), t(3.0, 8.0) / 13 ** 0.5)
    assert torch.allclose(oracle.unit(t(3.0, 4.0)), t(0.6, 0.8), atol=1e-6)
    # the convolution's last tap multiplies the current row, the first the one two before it
    y = oracle.causal_conv(t(1.0, 10.0, 100.0)[:, None], t(2.0, 3.0, 5.0)[None])
    assert torch.allclose(y[:, 0], t(5.0, 53.0, 532.0))
    r = oracle.rotate_halves(t(1.0, 0.0, 0.0, 1.0, 7.0)[None], torch.tensor([3]), 100.0, 4)[0]
    a, b = t(3.0), t(0.3)     # pairs (0, 2) and (1, 3)
    assert torch.allclose(r, torch.stack([a.cos()[0], -b.sin()[0], a.sin()[0], b.cos()[0], t(7.0)[0]]))
    p = oracle.window_weights(torch.zeros(4, 4, dtype=D), 2)
    assert torch.allclose(p, torch.tensor([[1, 0, 0, 0], [.5, .5, 0, 0], [0, .5, .5, 0], [0, 0, .5, .5]], dtype=D))
    assert torch.allclose(oracle.cap(t(0.001, 100.0), 2.0), t(0.001, 2.0), atol=1e-6)
    # the write is seen by the same token's read; decay acts before the difference to the old value is taken
    q, k = t(1.0, 0.0)[None, None].expand(1, 2, 2), t(1.0, 0.0)[None, None].expand(1, 2, 2)
    o = oracle.delta_rule(q, k, torch.tensor([[[4.0], [8.0]]], dtype=D), t(1.0, 0.5)[None], t(0.5, 0.25)[None])
    assert torch.allclose(o[0, :, 0], t(2.0, 1.0 + 0.25 * 7.0))
    W = {"up": torch.eye(2, dtype=D), "down": torch.eye(2, dtype=D)}
    assert torch.allclose(oracle.relu2_mlp(t(3.0, -3.0), W), t(9.0, 0.0))
    g = oracle.delta_gates(torch.zeros(1, 2, dtype=D), {"a": torch.ones(1, 2, dtype=D), "b": torch.ones(1, 2, dtype=D), "A_log": t(0.0), "dt_bias": t(1.0)})
    assert torch.allclose(g[0], 1 / (1 + t(1.0).exp())) and torch.allclose(g[1], t(0.5))
    assert oracle.runs(mm.CONFIGS["mixed"]) == [0, 1, 2, 3, 1, 2, 3, 4] and oracle.runs({"layers": [0, 0]}) == [0, 1]


MISTAKES = {   # what a fault in a mechanism would look like, planted in the oracle
    "window": ("window_weights", lambda f: lambda s, w: f(s, w + 1)),
    "cap": ("cap", lambda f: lambda s, c: s),
    "pairing": ("rotate_halves", lambda f: lambda x, p, b, d: torch.cat(
        [f(torch.cat([x[..., 0:d:2], x[..., 1:d:2]], -1), p, b, d), x[..., d:]], -1) if d else x),
    "angle": ("rotate_halves", lambda f: lambda x, p, b, d: f(x, p + 1, b, d) if x.shape[0] == 4 else f(x, p, b, d)),
    "unit": ("unit", lambda f: lambda x: x),
    "taps": ("causal_conv", lambda f: lambda x, w: f(x, w.flip(1))),
    "state": ("delta_rule", lambda f: lambda q, k, v, g, b: torch.cat([f(q[:, :9], k[:, :9], v[:, :9], g[:, :9], b[:, :9]),
                                                                     f(q[:, 9:], k[:, 9:], v[:, 9:], g[:, 9:], b[:, 9:])], 1)),
    "decay": ("delta_rule", lambda f: lambda q, k, v, g, b: f(q, k, v, torch.ones_like(g), b)),
    "step size": ("delta_rule", lambda f: lambda q, k, v, g, b: f(q, k, v, g, torch.ones_like(b))),
    "gain": ("centred_norm", lambda f: lambda x, w, e: f(x, w - 1, e)),
    "square": ("relu2_mlp", lambda f: lambda h, W: torch.clamp(h @ W["up"].T, min=0) @ W["down"].T),
    "loop": ("runs", lambda f: lambda c: list(range(len(c["layers"])))),
}


@pytest.mark.parametrize("what", list(MISTAKES))
def test_mistakes_show_in_the_logits(what, monkeypatch):
    """The test models' weights let every mechanism move the logits by more than what the GPU tests allow in bf16; a window
    one key too wide by far more than they allow in 32 bits (a key made to stand out shows it in bf16)."""
    cfg = mm.CONFIGS["plain"]
    sd, ids = mm.weights(cfg), tm.tokens(cfg, 60)
    want = mm.reference(cfg, sd, ids)
    name, wrong = MISTAKES[what]
    monkeypatch.setattr(oracle, name, wrong(getattr(oracle, name)))
    assert tm.rel_err(mm.reference(cfg, sd, ids), want).max() > (0.02 if what == "window" else 0.06)


# ------------------------------------------------------------------------------------------------ configuration, weights
def test_config_and_shapes():
    c = Medirax.parse_config(mm.CONFIGS["mixed"])
    assert c.block == "rms" and c.logit_scale == 1.6 and c.runs == (0, 1, 2, 3, 1, 2, 3, 4) and c.recurrent
    assert isinstance(c.layers[0].mixer, GroupedMixer) and c.layers[0].mixer.window == 1 and c.layers[0].mlp is None
    assert isinstance(c.layers[3].mixer, DeltaMixer) and c.layers[3].mixer.taps == 7 and c.layers[1].mixer.scale == 11 ** -0.5
    s = Medirax.tensor_shapes(c)
    assert s["l4.mix.q"] == (96, 77) and s["l4.mix.k.b"] == (32,) and s["l4.mix.o"] == (77, 96) and s["l4.mix.o.b"] == (77,)
    assert s["l3.mix.v.conv"] == (312, 7) and s["l3.mix.a"] == (6, 77) and s["l3.mix.norm"] == (52,) and s["l3.mix.g"] == (312, 77)
    assert "l0.mlp.up" not in s and s["l1.mlp.down"] == (77, 33) and "l0.norm2" not in s and "final.norm.b" not in s
    plain = {k: v for k, v in mm.CONFIGS["plain"].items() if k != "loop"}
    assert Medirax.parse_config(plain).runs == (0, 1, 2)
    for bad in ({"type": "other"}, {"mlp": {"kind": "sparse", "ff": 4}}, {"mixer": {**mm.delta()["mixer"], "kv_heads": 3}}):
        cfg = json.loads(json.dumps(plain))
        cfg["layers"][0].update(bad)
        with pytest.raises(ValueError):
            Medirax.parse_config(cfg)
    with pytest.raises(ValueError):
        Medirax.parse_config({**plain, "loop": {"start": 1, "stop": 9, "times": 2}})


def test_checkpoint_registry_and_random_init(tmp_path):
    from safetensors.torch import save_file

    cfg = mm.CONFIGS["mixed"]
    sd = mm.weights(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(sd, str(tmp_path / "model.safetensors"))
    m = load_model(str(tmp_path), device="cpu")
    assert isinstance(m, Medirax) and all(torch.equal(m.sd[k], sd[k]) for k in sd) and "Medirax" in registry.architectures()
    with pytest.raises(KeyError):
        Medirax(Medirax.parse_config(cfg), {k: v for k, v in sd.items() if k != "l1.mix.A_log"}, device="cpu")
    r = Medirax.random_init(Medirax.parse_config(cfg), device="cpu")
    assert (r.sd["l0.norm1"] == 0).all() and (r.sd["l1.mix.norm"] == 1).all() and (r.sd["l1.mix.A_log"].float() <= 0).all()
    assert torch.allclose(r.layer_tensors(0)["norm1_w"], torch.ones(77)) and torch.allclose(r.head_tensors()["final_w"], torch.ones(77))


@pytest.mark.parametrize("name", list(mm.CONFIGS))
def test_packed_tensors_compute_the_mechanisms(name):
    """The packed matrices, multiplied plainly, give what the oracle's functions give, head by head at its padded place."""
    cfg = mm.CONFIGS[name]
    sd = tm.doubles(mm.weights(cfg))
    c = Medirax.parse_config(cfg)
    rc, h = _handle(cfg)
    assert rc == 0
    dims = _dims(h, len(c.runs))
    model = Medirax(c, mm.weights(cfg), device="cpu", dtype=torch.float32)
    for i, s in enumerate(c.layers):
        d, m, lay = dims[c.runs.index(i)], s.mixer, cfg["layers"][i]["mixer"]
        p = pack_layer(s, c.width, model.layer_tensors(i), d, D, "cpu")
        W = {k[len(f"l{i}.mix."):]: v for k, v in sd.items() if k.startswith(f"l{i}.mix.")}
        T = 5
        x = torch.randn(T, c.width, dtype=D)
        y = torch.nn.functional.pad(x, (0, d.k_in - c.width)) @ p["w_in"].T

        def heads(first, n, padded, size, t=y):
            blk = t[:, first:first + n * padded].reshape(T, n, padded)
            assert blk[..., size:].abs().sum() == 0
            return blk[..., :size].transpose(0, 1)

        if isinstance(m, GroupedMixer):
            y = y.clone()
            y[:, : d.n_raw] += p["b_in"].double()
            pos = torch.arange(T) + 4

            def turned(t):     # rotation of adjacent pairs, then the norm
                t, r = t.clone(), m.rot_dims // 2
                a = pos.double()[:, None] * m.rot_base ** (-2.0 * torch.arange(r, dtype=D) / max(m.rot_dims, 1))
                u, v = t[..., 0:2 * r:2].clone(), t[..., 1:2 * r:2].clone()
                t[..., 0:2 * r:2], t[..., 1:2 * r:2] = u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()
                return oracle.rms(t, cfg["norm"]["eps"])

            q, k = turned(heads(0, m.heads, d.dimp, m.dim, y)), turned(heads(d.n_key, m.kv_heads, d.dimp, m.dim, y))
            qo, ko = oracle.normed_query_keys(x, W, lay, cfg["norm"]["eps"], pos)
            rep = m.heads // m.kv_heads
            assert torch.allclose(q @ k.repeat_interleave(rep, 0).transpose(1, 2), qo @ ko.repeat_interleave(rep, 0).transpose(1, 2))
            assert torch.allclose(heads(d.n_value, m.kv_heads, d.vdp, m.vdim, y), oracle.split_heads(x @ W["v"].T + W["v.b"], m.kv_heads))
            assert torch.allclose(p["b_out"][: c.width].double(), W["o.b"])
            assert d.cap % 64 == 0 and d.cap >= min(256, m.window + 64)
        else:
            for w, n, first, padded, size in (("q", m.kv_heads, 0, d.dimp, m.dim), ("k", m.kv_heads, d.n_key, d.dimp, m.dim),
                                              ("v", m.heads, d.n_value, d.vdp, m.vdim)):
                assert torch.allclose(heads(first, n, padded, size), oracle.split_heads(x @ W[w].T, n))
                conv = p["conv"].double()[:, first:first + n * padded].reshape(m.taps, n, padded)[..., :size]
                assert torch.allclose(conv.permute(1, 2, 0).reshape(-1, m.taps), W[w + ".conv"])
            assert torch.allclose(y[:, d.n_ab:d.n_ab + m.heads], x @ W["b"].T)
            assert torch.allclose(y[:, d.n_ab + m.heads:d.n_ab + 2 * m.heads], x @ W["a"].T)
            assert torch.allclose(heads(d.n_raw, m.heads, d.vdp, m.vdim), oracle.split_heads(x @ W["g"].T, m.heads))
            assert torch.allclose(p["neg_a"].double(), -W["A_log"].exp()) and torch.allclose(p["head_norm"][: m.vdim].double(), W["norm"])
            assert d.slot_bytes == 4 * (m.heads * d.vdp * d.dimp + m.taps * d.n_ab)
        a, want = torch.zeros(T, d.k_out, dtype=D), 0
        o = torch.randn(T, m.heads, m.vdim, dtype=D)
        for j in range(m.heads):
            a[:, j * d.vdp:j * d.vdp + m.vdim] = o[:, j]
        want = o.reshape(T, -1) @ W["o"].T
        if s.mlp is not None:
            assert torch.allclose(y[:, d.n_mlp:d.n_mlp + s.mlp.ff], x @ sd[f"l{i}.mlp.up"].T)
            a[:, d.off_y:d.off_y + s.mlp.ff] = torch.randn(T, s.mlp.ff, dtype=D)
            want = want + a[:, d.off_y:d.off_y + s.mlp.ff] @ sd[f"l{i}.mlp.down"].T
        assert torch.allclose((a @ p["w_out"].T)[:, : c.width], want)
        assert torch.allclose(p["norm1_w"].double(), 1 + sd[f"l{i}.norm1"])
        for k in ("w_in", "w_out"):
            assert p[k].shape[0] % 128 == 0 and p[k].shape[1] % 64 == 0
    _lib.load_lm().vuib_lm_destroy(h)


def test_pointed_models_make_one_key_stand_out():
    cfg = mm.config([(mm.attention(scale=0.6, softcap=20.0, size=500), None)])
    ids = [3, 4, 7, 5, 3, 9]
    sd = tm.doubles(mm.point_attention(cfg, mm.weights(cfg), 7, 9, (3, 4, 5)))
    h = oracle.centred_norm(sd["embed"][ids], sd["l0.norm1"], 1e-5)
    W = {k[7:]: v for k, v in sd.items() if k.startswith("l0.mix.")}
    m = cfg["layers"][0]["mixer"]
    q, k = oracle.normed_query_keys(h, W, m, 1e-5, torch.arange(6))
    s = oracle.cap((q @ k.repeat_interleave(2, 0).transpose(1, 2)) * m["scale"], m["softcap"])
    assert (torch.softmax(s[:, 5], -1)[:, 2] > 0.9).all()


# ------------------------------------------------------------------------------------------------ library, host side
def test_create_validates_and_a_slot_comes_once():
    lib, plain = _lib.load_lm(), mm.CONFIGS["plain"]

    def broken(layer, **kw):
        c = json.loads(json.dumps(plain))
        c["layers"][layer]["mixer"].update(kw)
        return _handle(c)[0]

    assert broken(1, rot={"base": 10.0, "dims": 22}) == -2 and broken(1, rot={"base": 10.0, "dims": 3}) == -2
    assert broken(1, dim=300) == -2 and broken(0, dim=300) == -2 and broken(0, conv=0) == -2 and broken(1, softcap=-1.0) == -2
    rc, h = _handle(plain)
    n = C.c_size_t()
    assert rc == 0 and lib.vuib_lm_workspace_bytes(h, C.byref(n)) == 0 and n.value > 0
    one = (C.c_int32 * 1)(1)
    assert lib.vuib_lm_prefill(h, 1, one, one, one, None, 0, None, None, None) == -4
    assert lib.vuib_lm_destroy(h) == 0


def test_command_line_info(tmp_path, capsys):
    from safetensors.torch import save_file
    from vui_b200.__main__ import main

    cfg = mm.CONFIGS["plain"]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(mm.weights(cfg), os.path.join(tmp_path, "model.safetensors"))
    assert main(["info", "--model", str(tmp_path)]) == 0
    assert json.loads(capsys.readouterr().out)["architecture"] == "Medirax"
