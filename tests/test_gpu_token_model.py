"""The token model's CUDA path against the plain oracle (float64), through the engine and its scheduler."""
import json
import os
import subprocess
import sys

import pytest
import torch

from tests import token_models as tm
from vui_b200 import TokenEngine, TokenGenConfig, Vidotar, open_engine

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"fp32": torch.float32, "bf16": torch.bfloat16}
LIMIT = {torch.float32: 5e-5, torch.bfloat16: 3e-2}   # relative RMS error of a row of logits
NEVER = 1 << 30


def engine(cfg, sd, dtype, **kw):
    kw = {"max_rows": 4, "max_seq": 512, "max_prefill_rows": 256, **kw}
    return TokenEngine(model=Vidotar(Vidotar.parse_config(cfg), sd, dtype=dtype), **kw)


def expand(eng, rows):
    """Prefills of at least `rows` rows expand their keys (NEVER: all attend in the absorbed form)."""
    eng._ck(eng._lib.vuib_lm_set_expand_min(eng._handle, rows))


def check(got, want, dtype, factor=1.0):
    e = tm.rel_err(got, want)
    assert e.max() <= factor * LIMIT[dtype], (e.max().item(), int(e.argmax()))


def run(eng, ids, cuts):
    """Logits of every position, the prompt cut into portions of the sizes `cuts` (the last repeated)."""
    with eng.new_row() as row:
        out, at, k = [], 0, 0
        while at < len(ids):
            n = min(cuts[min(k, len(cuts) - 1)], len(ids) - at)
            out.append(eng.step([(row, ids[at:at + n], list(range(n)))]))
            at, k = at + n, k + 1
        assert row.offset == len(ids)
    eng.check_device()
    return torch.cat(out)


@pytest.mark.parametrize("dt", list(DTYPES))
@pytest.mark.parametrize("name", list(tm.CONFIGS))
def test_prompts_portions_and_decoding(name, dt):
    """Whole prompts, portions down to two tokens, decoding token by token: all against the oracle, positions around
    every key-tile and query-tile border among them; expanded and absorbed prefill."""
    cfg, dtype = tm.CONFIGS[name], DTYPES[dt]
    sd = tm.weights(cfg)
    ids = tm.tokens(cfg, 275)
    want = tm.reference(cfg, sd, ids)
    eng = engine(cfg, sd, dtype)
    for cuts, emin in (([275], 0), ([275], NEVER), ([64, 2, 37, 2, 2, 128], 9), ([5, 9, 2, 3], NEVER), ([70, 1], 0), ([1], 0)):
        expand(eng, emin)
        check(run(eng, ids, cuts), want, dtype)


@pytest.mark.parametrize("dt", list(DTYPES))
def test_layers_one_by_one(dt):
    """The residual rows after every layer, prompt and decode, against the oracle's."""
    import ctypes as C

    from oracle import vidotar_oracle as oracle

    cfg, dtype = tm.CONFIGS["mixed"], DTYPES[dt]
    sd = tm.weights(cfg, seed=5)
    ids, taps = tm.tokens(cfg, 40), []
    oracle.forward(cfg, tm.doubles(sd), torch.tensor(ids), taps=taps)
    eng = engine(cfg, sd, dtype, max_prefill_rows=64)
    buf = torch.zeros(3, 64, cfg["width"], device="cuda")
    eng._ck(eng._lib.vuib_lm_set_taps(eng._handle, C.c_void_p(buf.data_ptr())))
    with eng.new_row() as row:
        eng.step([(row, ids[:-1], [])])
        for i in range(3):
            check(buf[i, :39], taps[i][:39], dtype)
        eng.step([(row, ids[-1:], [])])
        for i in range(3):
            check(buf[i, :1], taps[i][39:], dtype)


@pytest.mark.parametrize("dt", list(DTYPES))
def test_each_mechanism_alone(dt):
    """Models in which one mechanism alone moves the logits: the embedding's scale, the MLP (its clamps reached), the
    attention without its gate's variation, the gate."""
    dtype = DTYPES[dt]
    cfg = tm.config([(tm.mixer(heads=2), (40, 0.5))], scale=2.5)
    base = tm.weights(cfg, seed=3)
    zero = lambda *names: {k: torch.zeros_like(v) if k in names else v for k, v in base.items()}  # noqa: E731
    ids = tm.tokens(cfg, 20)
    outs = {}
    for label, sd in {"embedding": zero("l0.mix.o", "l0.mlp.down"), "mlp": zero("l0.mix.o"),
                      "attention": zero("l0.mlp.down", "l0.mix.g"), "gate": zero("l0.mlp.down")}.items():
        want = tm.reference(cfg, sd, ids)
        for cuts in ([20], [1]):
            check(run(engine(cfg, sd, dtype), ids, cuts), want, dtype)
        outs[label] = want
    keys = list(outs)
    for i, a in enumerate(keys):      # and each of them does move them
        for b in keys[i + 1:]:
            assert tm.rel_err(outs[a], outs[b]).max() > 0.05, (a, b)


@pytest.mark.parametrize("dt", list(DTYPES))
@pytest.mark.parametrize("emin", [1, NEVER])
def test_one_far_key_carries_the_query(dt, emin):
    """A query whose score with one key stands out, the key at the first positions, around the borders of key units and
    tiles, and just before the query; in a prompt and decoded.  Without that key the oracle's logits are far away."""
    dtype, cfg = DTYPES[dt], tm.config([(tm.mixer(heads=3), None)], vocab=131)
    sd = tm.point_at(cfg, tm.weights(cfg, seed=8), 0, needle=7, query=9)
    sd["l0.mix.o"] = sd["l0.mix.o"] * 4      # the attention's part of the residual
    eng = engine(cfg, sd, dtype, max_rows=2)
    expand(eng, emin)
    L = 262
    plain = [t if t not in (7, 9) else 3 for t in tm.tokens(cfg, L)]
    for at in (0, 1, 15, 16, 17, 31, 32, 33, 63, 64, 65, 127, 128, 129, 191, 192, 255, 256, L - 2):
        ids = list(plain)
        ids[at], ids[-1] = 7, 9
        want = tm.reference(cfg, sd, ids, [L - 1])
        blind = list(ids)
        blind[at] = 3
        seen = tm.rel_err(tm.reference(cfg, sd, blind, [L - 1]), want).max()
        assert seen > 0.15
        for cut in (L, L - 1):
            with eng.new_row() as row:
                if cut < L:
                    eng.step([(row, ids[:cut], [])])
                    got = eng.step([(row, ids[cut:], [0])])
                else:
                    got = eng.step([(row, ids, [L - 1])])
            assert tm.rel_err(got, want).max() <= min(LIMIT[dtype], 0.2 * seen), (at, cut)
    eng.check_device()


@pytest.mark.parametrize("dt", list(DTYPES))
def test_batches_of_unequal_requests_and_reused_slots(dt):
    """Prefills and decode steps of many rows at once against each row alone (by the oracle), one, few and many rows;
    then slots freed and taken by other requests while the rest go on."""
    cfg, dtype = tm.CONFIGS["plain"], DTYPES[dt]
    sd = tm.weights(cfg, seed=2)
    eng = engine(cfg, sd, dtype, max_rows=21)
    for n in (1, 2, 3, 5, 8, 9, 21):
        lens = [1 + (i * 53) % 140 for i in range(n)]
        seqs = [tm.tokens(cfg, k + 3, seed=i) for i, k in enumerate(lens)]
        rows = [eng.new_row() for _ in range(n)]
        got = [[g] for g in eng.step([(r, s[:k], [k - 1]) for r, s, k in zip(rows, seqs, lens)])]
        for j in range(3):
            for g, x in zip(got, eng.step([(r, [s[k + j]], [0]) for r, s, k in zip(rows, seqs, lens)])):
                g.append(x)
        for s, k, g in zip(seqs, lens, got):
            check(torch.stack(g), tm.reference(cfg, sd, s, list(range(k - 1, k + 3))), dtype)
        for r in rows:
            r.close()
    # two go on, one slot changes hands twice; a step mixes portions with single tokens
    a, b = tm.tokens(cfg, 90, seed=40), tm.tokens(cfg, 60, seed=41)
    ra, rb = eng.new_row(), eng.new_row()
    eng.step([(ra, a[:50], []), (rb, b[:30], [])])
    at, bt = 50, 30
    for seed in (42, 43):
        c = tm.tokens(cfg, 20, seed=seed)
        rc = eng.new_row()
        assert rc.idx == 2
        got = eng.step([(ra, a[at:at + 1], [0]), (rc, c, [19]), (rb, b[bt:bt + 7], [6])])
        for g, s, p in zip(got, (a, c, b), (at, 19, bt + 6)):
            check(g[None], tm.reference(cfg, sd, s, [p]), dtype)
        at, bt = at + 1, bt + 7
        rc.close()
    eng.check_device()


def test_portions_longer_than_a_call_and_several_expansion_groups():
    """More rows than one prefill call takes, and histories that do not fit the expansion scratch together."""
    cfg = tm.CONFIGS["plain"]
    sd = tm.weights(cfg, seed=6)
    eng = engine(cfg, sd, torch.bfloat16, max_rows=6, max_seq=200, max_prefill_rows=48)
    expand(eng, 5)
    seqs = [tm.tokens(cfg, 190, seed=60 + i) for i in range(6)]
    rows = [eng.new_row() for _ in range(6)]
    got = eng.step([(r, s[:180], [0, 100, 179]) for r, s in zip(rows, seqs)])
    more = eng.step([(r, s[180:187], [2, 6]) for r, s in zip(rows, seqs)])     # 6 x 187 keys, 42 rows
    for i, s in enumerate(seqs):
        want = tm.reference(cfg, sd, s, [0, 100, 179, 182, 186])
        check(torch.cat([got[3 * i:3 * i + 3], more[2 * i:2 * i + 2]]), want, torch.bfloat16)


@pytest.mark.parametrize("dt", list(DTYPES))
def test_rewind_forgets(dt):
    cfg, dtype = tm.CONFIGS["plain"], DTYPES[dt]
    sd = tm.weights(cfg)
    eng = engine(cfg, sd, dtype)
    a, b = tm.tokens(cfg, 50, seed=7), tm.tokens(cfg, 30, seed=8)
    with eng.new_row() as row:
        eng.step([(row, a, [])])
        row.rewind(20)
        got = eng.step([(row, b, [29])])
        check(got, tm.reference(cfg, sd, a[:20] + b, [49]), dtype)
        with pytest.raises(ValueError):
            row.rewind(99)


def _greedy_ok(cfg, sd, prompt, new, dtype):
    """Every greedy token is the oracle's argmax, unless the oracle's two best are closer than the precision allows."""
    ids = prompt + new
    want = tm.reference(cfg, sd, ids, list(range(len(prompt) - 1, len(ids) - 1)))
    top = want.max(-1)
    chosen = want.gather(1, torch.tensor(new)[:, None])[:, 0]
    slack = 6 * LIMIT[dtype] * (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    assert ((top.values - chosen) <= slack).all()
    return int((top.indices == torch.tensor(new)).sum())


@pytest.mark.parametrize("dt", list(DTYPES))
def test_greedy_generation_through_the_scheduler(dt):
    """More prompts than slots, unequal lengths and stop ids, against the oracle and against each prompt alone."""
    cfg, dtype = tm.CONFIGS["plain"], DTYPES[dt]
    sd = tm.weights(cfg, seed=9)
    eng = engine(cfg, sd, dtype, max_rows=3)
    prompts = [tm.tokens(cfg, 1 + (i * 37) % 80, seed=100 + i) for i in range(8)]
    out = eng.generate(prompts, TokenGenConfig(max_new_tokens=20))
    agree = sum(_greedy_ok(cfg, sd, p, o, dtype) for p, o in zip(prompts, out))
    assert all(len(o) == 20 for o in out) and agree >= (160 if dtype == torch.float32 else 140)
    if dtype == torch.float32:
        assert [eng.generate([p], TokenGenConfig(max_new_tokens=20))[0] for p in prompts] == out
    stop = out[0][4]
    cut = eng.generate(prompts[:1], TokenGenConfig(max_new_tokens=20, stop_ids=(stop,)))[0]
    assert cut == out[0][: out[0].index(stop)]
    with eng.new_row() as row:
        assert list(row.stream(prompts[0], TokenGenConfig(max_new_tokens=6))) == out[0][:6]
    assert eng.generate([], TokenGenConfig()) == []
    eng.check_device()


def test_long_decoding():
    cfg = tm.CONFIGS["plain"]
    sd = tm.weights(cfg, seed=10)
    for dtype in DTYPES.values():
        eng = engine(cfg, sd, dtype, max_rows=1, max_seq=420)
        prompt = tm.tokens(cfg, 10, seed=11)
        new = eng.generate([prompt], TokenGenConfig(max_new_tokens=400))[0]
        assert len(new) == 400 and _greedy_ok(cfg, sd, prompt, new, dtype) >= 350
        # the cache is full after 420 tokens, not before
        assert len(eng.generate([prompt], TokenGenConfig(max_new_tokens=1000))[0]) == 411


def test_sampling():
    """Top-k support and frequencies, the whole distribution, the seed, and the repetition penalty."""
    cfg = tm.CONFIGS["plain"]
    eng = engine(cfg, tm.weights(cfg), torch.float32, max_rows=64, seed=3)
    V = cfg["vocab"]
    logits = (torch.randn(V, generator=torch.Generator().manual_seed(0)) * 1.5).cuda()
    slots = torch.arange(64, device="cuda", dtype=torch.int32)

    def draws(n, **kw):
        eng._apply_cfg(TokenGenConfig(**kw))
        eng._ck(eng._lib.vuib_lm_reset_slot(eng._handle, -1, eng._stream))
        return torch.cat([eng._sample(slots, logits.expand(64, V).contiguous()) for _ in range(n)]).cpu()

    for T, k in ((0.8, 5), (1.3, 0)):
        d = draws(100, temperature=T, top_k=k)
        p = torch.softmax(logits.cpu().double() / T, 0)
        if k:
            keep = p >= p.topk(k).values[-1]
            assert set(d.tolist()) <= set(torch.nonzero(keep)[:, 0].tolist())
            p = torch.where(keep, p, torch.zeros_like(p)) / p[keep].sum()
        f = torch.bincount(d, minlength=V).double() / len(d)
        assert (f - p).abs().max() < 5 * (0.25 / len(d)) ** 0.5
        assert torch.equal(d, draws(100, temperature=T, top_k=k))      # the same seed, the same draws
    assert (draws(1) == int(logits.argmax())).all()
    # a penalty this strong never draws a token twice while its window holds it; a window of 2 lets it come back
    d = draws(8, rep_penalty=1e6, top_k=1).view(8, 64)
    assert all(len(set(d[:, i].tolist())) == 8 for i in range(64))
    d = draws(9, rep_penalty=1e6, rep_window=2, top_k=1).view(9, 64)
    assert (d[3:] == d[:-3]).all() and (d[1:] != d[:-1]).all()


def test_bad_input_is_refused_on_the_host():
    cfg = tm.CONFIGS["plain"]
    eng = engine(cfg, tm.weights(cfg), torch.bfloat16, max_seq=32)
    row = eng.new_row()
    for entry, err in (((row, [1, cfg["vocab"]], []), ValueError), ((row, [], []), ValueError), ((row, [1], [1]), ValueError),
                       ((row, list(range(33)), []), RuntimeError)):
        with pytest.raises(err):
            eng.step([entry])
    with pytest.raises(ValueError, match="twice"):
        eng.step([(row, [1], []), (row, [2], [])])
    assert row.offset == 0


def test_a_key_tile_smaller_than_the_widest_rows_need():
    """Cached rows so wide that a key tile takes fewer keys, and a value matrix that does not fit beside them."""
    cfg = tm.config([(tm.mixer(heads=2, dim=64, rot_dim=64, vdim=160, q_rank=64, kv_rank=900), (64, 1.0))], width=128)
    sd = tm.weights(cfg, seed=12)
    ids = tm.tokens(cfg, 150)
    want = tm.reference(cfg, sd, ids)
    for dtype in DTYPES.values():
        eng = engine(cfg, sd, dtype, max_seq=160)
        for cuts in ([150], [100, 1], [3]):
            check(run(eng, ids, cuts), want, dtype)


def test_command_line_and_trace_replay(tmp_path):
    import numpy as np
    from safetensors.torch import save_file

    cfg = tm.CONFIGS["mixed"]
    sd = tm.weights(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(sd, str(tmp_path / "model.safetensors"))
    ids = tm.tokens(cfg, 30)
    want = tm.reference(cfg, sd, ids)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:20], "want": [3, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": ids[20:28], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": ids[28:29], "want": [0]}], "end": ["x"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "64"], input="\n".join(json.dumps(x) for x in lines), text=True,
                       capture_output=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    got = [torch.from_numpy(np.fromfile(tmp_path / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"])) for s in (0, 2)]
    check(torch.cat(got), want[[3, 19, 28]], torch.float32)
    p = subprocess.run([sys.executable, "-m", "vui_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt-ids",
                        ",".join(map(str, ids)), "--prompt-ids", "5 6 7", "--max-new-tokens", "5"], text=True, capture_output=True,
                       timeout=300, cwd=ROOT)
    assert p.returncode == 0, p.stderr
    out = [json.loads(x) for x in p.stdout.strip().split("\n")]
    assert len(out) == 2 and _greedy_ok(cfg, sd, ids, out[0], torch.float32) == 5
    eng = open_engine(str(tmp_path), dtype=torch.float32, max_seq=64)
    assert isinstance(eng, TokenEngine) and eng.generate([[5, 6, 7]], TokenGenConfig(max_new_tokens=5))[0] == out[1]
