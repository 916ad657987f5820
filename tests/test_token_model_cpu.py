"""Token models without a GPU: configuration and weights, packing against the oracle's mechanisms, registry, the slot
engine's host logic, the trace replay's bookkeeping, and the library's host checks."""
import ctypes as C
import io
import json
import os
import re

import pytest
import torch

from oracle import vidotar_oracle as oracle
from tests import token_models as tm
from vui_b200 import TokenLM, Vidotar, VuiB200, _lib, load_model
from vui_b200 import registry, trace
from vui_b200.slots import SlotEngine
from vui_b200.token_lm import abi_config, abi_layers, pack_layer, trig_table

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _save(folder, cfg, sd):
    from safetensors.torch import save_file

    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in sd.items()}, os.path.join(folder, "model.safetensors"))


def _handle(cfg, dtype=_lib.LM_BF16, **kw):
    c = Vidotar.parse_config(cfg)
    a = abi_config(c, **{**dict(dtype=dtype, n_slots=3, max_seq=256, max_rows=2, max_prefill_rows=64), **kw})
    h = C.c_void_p()
    return _lib.load_lm().vuib_lm_create(C.byref(a), abi_layers(c), C.byref(h)), h


def _dims(h, n):
    out = []
    for i in range(n):
        d = _lib.VuibLmDims()
        assert _lib.load_lm().vuib_lm_layer_dims(h, i, C.byref(d)) == 0
        out.append(d)
    return out


# ------------------------------------------------------------------------------------------------ the oracle itself
def test_oracle_mechanisms_on_hand_values():
    x = torch.tensor([[1.0, 2.0, 6.0]], dtype=torch.float64)
    assert torch.allclose(oracle.layer_norm(x, torch.ones(3), torch.zeros(3), 0.0), (x - 3) / (14 / 3) ** 0.5)
    assert torch.allclose(oracle.rms_norm(x, torch.ones(3), 0.0), x / (41 / 3) ** 0.5)
    r = oracle.rotate_pairs(torch.tensor([[1.0, 0.0, 0.0, 1.0, 5.0]], dtype=torch.float64), torch.tensor([2]), 100.0, 4)
    c, s = torch.tensor(2.0).double().cos(), torch.tensor(2.0).double().sin()
    c2, s2 = torch.tensor(0.2).double().cos(), torch.tensor(0.2).double().sin()
    assert torch.allclose(r, torch.stack([c, s, -s2, c2, torch.tensor(5.0).double()])[None])
    p = oracle.causal_softmax(torch.zeros(3, 3, dtype=torch.float64))
    assert torch.allclose(p, torch.tensor([[1, 0, 0], [.5, .5, 0], [1 / 3, 1 / 3, 1 / 3]], dtype=torch.float64))
    # above the limit the gate is cut, below it is not; the other factor is cut on both sides
    W = {"gate": torch.eye(2).double(), "up": torch.eye(2).double(), "down": torch.eye(2).double()}
    y = oracle.clamped_mlp(torch.tensor([[3.0, -3.0]]).double(), W, 1.0)
    g = torch.tensor([1.0, -3.0]).double()
    assert torch.allclose(y[0], g * torch.sigmoid(1.702 * g) * torch.tensor([2.0, 0.0]).double())


# ------------------------------------------------------------------------------------------------ configuration, weights
def test_config_and_shapes():
    c = Vidotar.parse_config(tm.CONFIGS["mixed"])
    assert [s.mixer.heads for s in c.layers] == [1, 5, 2] and c.layers[0].mlp is None
    assert c.layers[1].mlp.limit == 0.4 and c.layers[1].mixer.rot_base == 1e5 and c.embed_scale == 0.6
    shapes = Vidotar.tensor_shapes(c)
    assert shapes["l1.mix.uq"] == (5 * 43, 65) and shapes["l1.mix.dkv"] == (50, 77) and shapes["l2.mlp.down"] == (77, 16)
    assert "l0.norm2" not in shapes and "l0.mlp.gate" not in shapes and "l1.norm2.b" in shapes
    for bad in ({"type": "other"}, {"mlp": {"kind": "sparse", "ff": 4, "limit": 1.0}}):
        cfg = json.loads(json.dumps(tm.CONFIGS["plain"]))
        cfg["layers"][1].update(bad)
        with pytest.raises(ValueError):
            Vidotar.parse_config(cfg)


def test_checkpoint_roundtrip_and_registry(tmp_path):
    cfg = tm.CONFIGS["mixed"]
    sd = tm.weights(cfg)
    _save(tmp_path, cfg, sd)
    m = load_model(str(tmp_path), device="cpu")
    assert isinstance(m, Vidotar) and isinstance(m, TokenLM) and all(torch.equal(m.sd[k], sd[k]) for k in sd)
    assert registry.architecture_of(str(tmp_path)) == "Vidotar" and {"Vidotar", "Vui"} <= set(registry.architectures())
    assert registry._resolve(registry._REGISTRY["Vui"].model) is VuiB200
    with pytest.raises(KeyError):
        Vidotar(Vidotar.parse_config(cfg), {k: v for k, v in sd.items() if k != "l1.mix.g"}, device="cpu")
    with pytest.raises(ValueError):
        Vidotar(Vidotar.parse_config(cfg), {**sd, "head": sd["head"][:-1]}, device="cpu")
    with pytest.raises(ValueError):
        Vidotar(Vidotar.parse_config(cfg), sd, device="cpu", dtype=torch.float16)
    (tmp_path / "config.json").write_text(json.dumps({**cfg, "architecture": "Nothing"}))
    with pytest.raises(ValueError, match="Nothing"):
        load_model(str(tmp_path), device="cpu")


def test_trig_table():
    t = trig_table(50.0, 6, 40)
    assert t.shape == (40, 3, 2) and t.dtype == torch.float32
    assert abs(float(t[39, 2, 1]) - torch.sin(torch.tensor(39 * 50.0 ** (-4 / 6), dtype=torch.float64)).item()) < 1e-7


@pytest.mark.parametrize("name", list(tm.CONFIGS))
@pytest.mark.parametrize("dtype", [_lib.LM_BF16, _lib.LM_F32])
def test_packed_matrices_compute_the_mechanisms(name, dtype):
    """The packed matrices, multiplied plainly, give what the oracle's functions give: projections by region, absorbed
    queries and keys, expanded keys and values, the joint output matrix; the padding is zero."""
    cfg = tm.CONFIGS[name]
    sd = tm.doubles(tm.weights(cfg))
    c = Vidotar.parse_config(cfg)
    rc, h = _handle(cfg, dtype)
    assert rc == 0
    model = Vidotar(c, tm.weights(cfg), device="cpu", dtype=torch.float32)
    for i, (d, s) in enumerate(zip(_dims(h, len(c.layers)), c.layers)):
        assert d.x_ok == (dtype == _lib.LM_BF16)
        m, lay = s.mixer, cfg["layers"][i]
        p = pack_layer(s, c.width, model.layer_tensors(i), d, torch.float64, "cpu")
        W = {k[len(f"l{i}.mix."):]: v for k, v in sd.items() if k.startswith(f"l{i}.mix.")}
        T, H = 5, m.heads
        x = torch.randn(T, c.width, dtype=torch.float64)
        pos = torch.arange(T) + 3
        xin = torch.nn.functional.pad(x, (0, d.k_in - c.width))
        y = xin @ p["w_in"].T
        assert torch.allclose(y[:, : m.q_rank], x @ W["dq"].T) and y[:, m.q_rank:d.n_dq].abs().sum() == 0
        dkv = x @ W["dkv"].T
        assert torch.allclose(y[:, d.n_dq:d.n_dq + m.kv_rank], dkv[:, : m.kv_rank])
        assert torch.allclose(y[:, d.n_dq + d.rp:d.n_dq + d.rp + m.rot_dim], dkv[:, m.kv_rank:])
        assert torch.allclose(y[:, d.n_kv:d.n_kv + H * m.vdim], x @ W["g"].T)
        if s.mlp is not None:
            assert torch.allclose(y[:, d.n_mlp:d.n_mlp + 2 * s.mlp.ff:2], x @ sd[f"l{i}.mlp.gate"].T)
            assert torch.allclose(y[:, d.n_mlp + 1:d.n_mlp + 2 * s.mlp.ff:2], x @ sd[f"l{i}.mlp.up"].T)
        # scores: absorbed query . cached row = plain + rotated score
        qn, qr = oracle.latent_queries(x, W, lay["mixer"], cfg["norm"]["eps"], pos)
        ck, kr = oracle.latent_keys(x, W, lay["mixer"], cfg["norm"]["eps"], pos)
        kn = (ck @ W["uk"].T).reshape(T, H, m.dim).transpose(0, 1)
        cq = torch.nn.functional.pad(oracle.rms_norm(x @ W["dq"].T, W["dq.norm"], cfg["norm"]["eps"]), (0, d.k_q - m.q_rank))
        q = (cq @ p["w_q"].T)[:, : H * d.dp].reshape(T, H, d.dp)
        rows = torch.zeros(T, d.dp, dtype=torch.float64)
        rows[:, : m.kv_rank], rows[:, d.rp:d.rp + m.rot_dim] = ck, kr
        q = q.transpose(0, 1).clone()
        q[..., d.rp:d.rp + m.rot_dim] = oracle.rotate_pairs(q[..., d.rp:d.rp + m.rot_dim], pos, m.rot_base, m.rot_dims)
        assert torch.allclose(q @ rows.T, qn @ kn.transpose(1, 2) + qr @ kr.T)
        assert torch.allclose(ck @ p["w_uv"][..., : m.kv_rank].transpose(1, 2), (ck @ W["uv"].T).reshape(T, H, m.vdim).transpose(0, 1))
        if d.x_ok:
            xk = torch.nn.functional.pad(ck, (0, d.k_kv - m.kv_rank)) @ p["w_xkv"].T
            assert torch.allclose(xk[:, : H * d.dimp].reshape(T, H, d.dimp)[..., : m.dim].transpose(0, 1), kn)
            v = xk[:, H * d.dimp:H * (d.dimp + d.vdp)].reshape(T, H, d.vdp)[..., : m.vdim].reshape(T, -1)
            assert torch.allclose(v, ck @ W["uv"].T)
            xq = (cq @ p["w_xq"].T)[:, : H * (d.dimp + d.rotp)].reshape(T, H, -1)
            assert torch.allclose(xq[..., : m.dim].transpose(0, 1), qn)
        a = torch.zeros(T, d.k_out, dtype=torch.float64)
        a[:, : H * m.vdim] = torch.randn(T, H * m.vdim, dtype=torch.float64)
        want = a[:, : H * m.vdim] @ W["o"].T
        if s.mlp is not None:
            a[:, d.off_y:d.off_y + s.mlp.ff] = torch.randn(T, s.mlp.ff, dtype=torch.float64)
            want = want + a[:, d.off_y:d.off_y + s.mlp.ff] @ sd[f"l{i}.mlp.down"].T
        assert torch.allclose((a @ p["w_out"].T)[:, : c.width], want)
        for k in ("w_in", "w_q", "w_out"):
            assert p[k].shape[0] % 128 == 0 and p[k].shape[1] % 64 == 0
    _lib.load_lm().vuib_lm_destroy(h)


def test_point_at_makes_one_score_stand_out():
    cfg = tm.CONFIGS["plain"]
    sd = tm.doubles(tm.point_at(cfg, tm.weights(cfg), 0, needle=7, query=9))
    ids = torch.tensor([1, 2, 7, 4, 5, 9])
    x = oracle.layer_norm(sd["embed"][ids] * cfg["embedding"]["scale"], sd["l0.norm1"], sd["l0.norm1.b"], cfg["norm"]["eps"])
    W = {k[7:]: v for k, v in sd.items() if k.startswith("l0.mix.")}
    m = cfg["layers"][0]["mixer"]
    qn, qr = oracle.latent_queries(x, W, m, cfg["norm"]["eps"], torch.arange(6))
    c, kr = oracle.latent_keys(x, W, m, cfg["norm"]["eps"], torch.arange(6))
    s = (qn @ (c @ W["uk"].T).reshape(6, m["heads"], -1).transpose(0, 1).transpose(1, 2) + qr @ kr.T) * m["scale"]
    assert (torch.softmax(s[:, 5], -1)[:, 2] > 0.9).all()


# ------------------------------------------------------------------------------------------------ library, host side
def test_lm_symbols_match_the_header():
    with open(os.path.join(ROOT, "include", "vuib200_lm.h")) as f:
        src = re.sub(r"/\*.*?\*/", "", f.read(), flags=re.S)
    names = sorted(set(re.findall(r"\b(vuib_lm_[a-z0-9_]+)\s*\(", src)))
    lib = _lib.load_lm()
    assert names == sorted(_lib.LM_SYMBOLS) and all(hasattr(lib, n) for n in names)
    assert C.sizeof(_lib.VuibLmConfig) == 48 and C.sizeof(_lib.VuibLmLayer) == 80 and C.sizeof(_lib.VuibLmDims) == 120


def test_lm_create_validates_and_refuses_unbound_calls():
    lib, cfg = _lib.load_lm(), tm.CONFIGS["plain"]
    assert _handle(cfg, dtype=7)[0] == -2 and _handle(cfg, max_seq=0)[0] == -3 and _handle({**cfg, "vocab": 0})[0] == -2
    c = json.loads(json.dumps(cfg))
    c["layers"][0]["mixer"]["rot"]["dims"] = 14   # more than the head has
    assert _handle(c)[0] == -2
    rc, h = _handle(cfg)
    assert rc == 0
    n = C.c_size_t()
    assert lib.vuib_lm_workspace_bytes(h, C.byref(n)) == 0 and n.value > 0
    assert lib.vuib_lm_bind_workspace(h, C.c_void_p(0x1001), n.value) == -6
    one = (C.c_int32 * 1)(1)
    assert lib.vuib_lm_prefill(h, 1, one, one, one, None, 0, None, None, None) == -4
    assert lib.vuib_lm_decode(h, 1, None, None, None, None, None) == -4
    assert lib.vuib_lm_sample(h, 1, C.c_void_p(256), C.c_void_p(256), C.c_void_p(256), None) == -4
    assert lib.vuib_lm_set_wait_limit(h, 2) == -3 and lib.vuib_lm_launch_count(h) == 0
    with pytest.raises(_lib.VuibError):
        _lib.check(h, -3, lib.vuib_lm_last_error)
    assert lib.vuib_lm_destroy(h) == 0


# ------------------------------------------------------------------------------------------------ slot engine, trace
class _Row:
    def __init__(self, eng, idx):
        self._e, self.idx = eng, idx

    @property
    def offset(self):
        return int(self._e.seq_lens[self.idx])

    def close(self):
        self._e._release_row(self)


class _Slots(SlotEngine):
    _ROW = _Row

    def __init__(self, max_rows, max_seq=100, max_prefill_rows=8):
        self.max_seq, self.max_prefill_rows = max_seq, max_prefill_rows
        self.seq_lens = torch.zeros(max_rows + 1, dtype=torch.int32)
        self._handle = None
        self._init_slots(max_rows)


def test_pack_rows_cuts_and_keeps_positions():
    e = _Slots(3)
    r = [e.new_row() for _ in range(3)]
    e.seq_lens[1] = 4
    calls = []
    e._pack_rows([(r[0], torch.arange(5)), (r[1], torch.arange(10)), (r[0], torch.arange(2)), (r[2], torch.arange(1))],
                 lambda pend: calls.append([(s, o, t.tolist(), k) for s, o, t, k in pend]))
    assert all(sum(len(t) for _, _, t, _ in c) <= 8 for c in calls)
    assert calls == [[(0, 0, [0, 1, 2, 3, 4], 0), (1, 4, [0, 1, 2], 1)],
                     [(1, 7, [3, 4, 5, 6, 7, 8, 9], 1), (0, 5, [0], 2)], [(0, 6, [1], 2), (2, 0, [0], 3)]]
    with pytest.raises(RuntimeError, match="overflows"):
        e._pack_rows([(r[1], torch.arange(97))], calls.append)


def test_continuous_batching_refills_slots():
    e = _Slots(2)
    need = [3, 1, 0, 2, 1]          # steps each request takes after it is admitted (0: ends at once)
    left, seen, order = dict(enumerate(need)), [], []

    def admit(batch):
        order.extend(ri for ri, _ in batch)
        return {slot: ri for ri, slot in batch if need[ri]}

    def step(slots, states):
        seen.append(tuple(states))
        for ri in states:
            left[ri] -= 1
        return [s for s, ri in zip(slots, states) if left[ri] == 0]

    e._run_continuous(5, admit, step)
    assert order == [0, 1, 2, 3, 4] and all(v == 0 for v in left.values()) and max(len(s) for s in seen) == 2
    assert e._rows == {}


def test_rows_are_taken_and_given_back():
    e = _Slots(2)
    a, b = e.new_row(), e.new_row()
    with pytest.raises(RuntimeError):
        e.new_row()
    e.seq_lens[a.idx] = 9
    a.close()
    c = e.new_row()
    assert c.idx == a.idx and c.offset == 0 and b.idx == 1


def test_trace_replay_bookkeeping(tmp_path):
    class Fake(_Slots):
        def step(self, entries):
            self.log.append([(r.idx, list(ids), list(w)) for r, ids, w in entries])
            return torch.tensor([[float(ids[w])] * 3 for _, ids, ws in entries for w in ws]).reshape(-1, 3)

        def check_device(self):
            pass

    e = Fake(2)
    e.log, out = [], []
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": [4, 5], "want": [1, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [6], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [7], "want": [0]}], "end": ["b"]}]
    trace.run(e, io.StringIO("\n".join(json.dumps(x) for x in lines)), str(tmp_path), emit=lambda s, flush: out.append(s))
    assert out == ["done 0", "done 1", "done 2"] and [c[0][0] for c in e.log] == [0, 0, 0] and e._free == {0, 1}
    import numpy as np

    assert np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(2, 3)[:, 0].tolist() == [5.0, 4.0]
    assert not (tmp_path / "1.f32").exists() and (tmp_path / "2.f32").stat().st_size == 12


def test_command_line_info_and_errors(tmp_path, capsys):
    from vui_b200.__main__ import main

    cfg = tm.CONFIGS["plain"]
    _save(tmp_path, cfg, tm.weights(cfg))
    assert main(["info", "--model", str(tmp_path)]) == 0
    info = json.loads(capsys.readouterr().out)
    assert info["architecture"] == "Vidotar" and info["parameters"] > 0
    assert main(["generate", "--model", str(tmp_path)]) == 2    # no prompt
