"""The Medirax model's CUDA path against the plain oracle (float64), through the engine and its scheduler."""
import ctypes as C
import json
import os
import subprocess
import sys

import pytest
import torch

from tests import medirax_models as mm
from tests import token_models as tm
from vui_b200 import Medirax, TokenEngine, TokenGenConfig, open_engine

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"fp32": torch.float32, "bf16": torch.bfloat16}
LIMIT = {torch.float32: 5e-5, torch.bfloat16: 3e-2}   # relative RMS error of a row of logits
NEVER = 1 << 30


def engine(cfg, sd, dtype, **kw):
    kw = {"max_rows": 4, "max_seq": 512, "max_prefill_rows": 256, **kw}
    return TokenEngine(model=Medirax(Medirax.parse_config(cfg), sd, dtype=dtype), **kw)


def forms(eng, rows):
    """Portions of at least `rows` rows take the prefill forms (NEVER: attention row by row, recurrence token by token)."""
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
@pytest.mark.parametrize("name", list(mm.CONFIGS))
def test_prompts_portions_and_decoding(name, dt):
    """Whole prompts, portions down to two tokens, decoding token by token: all against the oracle, positions around every
    window, chunk and tile border among them; the prefill forms and the row-by-row ones."""
    cfg, dtype = mm.CONFIGS[name], DTYPES[dt]
    sd = mm.weights(cfg)
    ids = tm.tokens(cfg, 200)
    want = mm.reference(cfg, sd, ids)
    eng = engine(cfg, sd, dtype)
    for cuts, emin in (([200], 0), ([200], NEVER), ([64, 2, 37, 2, 2, 65], 9), ([5, 9, 2, 3], NEVER), ([70, 1], 0), ([1], 0)):
        forms(eng, emin)
        check(run(eng, ids, cuts), want, dtype)


@pytest.mark.parametrize("dt", list(DTYPES))
def test_layers_one_by_one(dt):
    """The residual rows after every run of a layer, prompt and decode, against the oracle's."""
    cfg, dtype = mm.CONFIGS["mixed"], DTYPES[dt]
    sd = mm.weights(cfg, seed=5)
    ids, taps = tm.tokens(cfg, 40), []
    mm.reference(cfg, sd, ids, taps=taps)
    eng = engine(cfg, sd, dtype, max_prefill_rows=64)
    buf = torch.zeros(len(taps), 64, cfg["width"], device="cuda")
    eng._ck(eng._lib.vuib_lm_set_taps(eng._handle, C.c_void_p(buf.data_ptr())))
    forms(eng, 9)
    with eng.new_row() as row:
        eng.step([(row, ids[:-1], [])])
        for i, t in enumerate(taps):
            check(buf[i, :39], t[:39], dtype)
        eng.step([(row, ids[-1:], [])])
        for i, t in enumerate(taps):
            check(buf[i, :1], t[39:], dtype)


@pytest.mark.parametrize("dt", list(DTYPES))
def test_each_mechanism_alone(dt):
    """Models in which one mechanism alone moves the logits: MLP, attention with and without its scores, the delta rule
    with and without its convolutions, its decay and its reads of older tokens."""
    dtype = DTYPES[dt]
    cfg = mm.config([(mm.delta(), 40), (mm.attention(), 40)], logit_scale=2.5)
    base = mm.weights(cfg, seed=3)
    downs, outs_ = ("l0.mlp.down", "l1.mlp.down"), ("l0.mix.o", "l1.mix.o", "l1.mix.o.b")

    def zero(*names):
        return {k: torch.zeros_like(v) if k in names else v.clone() for k, v in base.items()}

    cases = {"embedding": zero(*downs, *outs_), "mlp": zero(*outs_), "attention": zero(*downs, "l0.mix.o"),
             "values": zero(*downs, "l0.mix.o", "l1.mix.q", "l1.mix.q.b"), "delta": zero(*downs, "l1.mix.o", "l1.mix.o.b")}
    cases["no convolution"] = {k: v.clone() for k, v in cases["delta"].items()}
    for n in "qkv":
        cases["no convolution"][f"l0.mix.{n}.conv"][:, :-1] = 0
    cases["no decay"] = {**cases["delta"], "l0.mix.A_log": torch.full((4,), -30.0, dtype=torch.bfloat16)}
    cases["fast decay"] = {**cases["delta"], "l0.mix.A_log": torch.full((4,), 4.0, dtype=torch.bfloat16)}
    cases["small steps"] = {**cases["delta"], "l0.mix.b": cases["delta"]["l0.mix.b"] * 20}
    ids = tm.tokens(cfg, 70)
    outs = {}
    for label, sd in cases.items():
        outs[label] = want = mm.reference(cfg, sd, ids)
        eng = engine(cfg, sd, dtype)
        for cuts in ([70], [66, 1]):
            check(run(eng, ids, cuts), want, dtype)
    keys = list(outs)
    for i, a in enumerate(keys):      # and each of them does move them
        for b in keys[i + 1:]:
            assert tm.rel_err(outs[a], outs[b]).max() > 0.05, (a, b)


@pytest.mark.parametrize("dt", list(DTYPES))
@pytest.mark.parametrize("emin", [1, NEVER])
@pytest.mark.parametrize("size", [1, 2, 16, 33, 64, 100, 1 << 20])
def test_one_key_at_the_windows_edges(dt, emin, size):
    """A query whose score with one key stands out, the key just inside and just outside the window, at its far end and at
    the first positions, and around tile borders; in a prompt and decoded, over rings that have wrapped.  Inside, the logits
    without that key are far away; outside, those of a window one wider."""
    dtype, fillers = DTYPES[dt], (3, 4, 5, 6)
    cfg = mm.config([(mm.attention(scale=0.6, softcap=20.0, size=size), None)])
    sd = mm.point_attention(cfg, mm.weights(cfg, seed=8), 7, 9, fillers)
    sd["l0.mix.o"] = sd["l0.mix.o"] * 4      # the attention's part of the residual
    eng = engine(cfg, sd, dtype, max_rows=2, max_prefill_rows=70)
    forms(eng, emin)
    L = 262
    g = torch.Generator().manual_seed(1)
    plain = [fillers[i] for i in torch.randint(0, len(fillers), (L,), generator=g).tolist()]
    backs = {1, 2, 15, 16, 17, 63, 64, 65, L - 1, L - 2} | {b for b in (size - 2, size - 1, size, size + 1) if 0 < b < L}
    for back in sorted(backs):
        at = L - 1 - back
        ids = list(plain)
        ids[at], ids[-1] = 7, 9
        want = mm.reference(cfg, sd, ids, [L - 1])
        if back < size:
            other = mm.reference(cfg, sd, ids[:at] + [3] + ids[at + 1:], [L - 1])
        else:
            wider = json.loads(json.dumps(cfg))
            wider["layers"][0]["mixer"]["mask"]["size"] = back + 1
            other = mm.reference(wider, sd, ids, [L - 1])
        seen = tm.rel_err(other, want).max()
        assert seen > 0.15
        for cut in (L, L - 1):
            with eng.new_row() as row:
                if cut < L:
                    eng.step([(row, ids[:cut], [])])
                    got = eng.step([(row, ids[cut:], [0])])
                else:
                    got = eng.step([(row, ids, [L - 1])])
            assert tm.rel_err(got, want).max() <= min(LIMIT[dtype], 0.2 * seen), (back, cut)
    eng.check_device()


@pytest.mark.parametrize("dt", list(DTYPES))
@pytest.mark.parametrize("emin", [1, NEVER])
def test_the_state_remembers_a_far_token(dt, emin):
    """A token written under a key of its own and read once, near and far, around chunk borders and at the first positions;
    in a prompt, after portions, and decoded."""
    dtype, fillers = DTYPES[dt], (3, 4, 5, 6)
    cfg = mm.config([(mm.delta(), None)])
    sd = mm.point_delta(cfg, mm.weights(cfg, seed=8), 7, 9, fillers)
    sd["l0.mix.o"] = sd["l0.mix.o"] * 4
    eng = engine(cfg, sd, dtype, max_rows=2)
    forms(eng, emin)
    L = 262
    g = torch.Generator().manual_seed(2)
    plain = [fillers[i] for i in torch.randint(0, len(fillers), (L,), generator=g).tolist()]
    for back in (1, 2, 3, 5, 6, 63, 64, 65, 127, 128, 129, 197, 198, 199, L - 2, L - 1):
        ids = list(plain)
        ids[L - 1 - back], ids[-1] = 7, 9
        want = mm.reference(cfg, sd, ids, [L - 1])
        blind = list(ids)
        blind[L - 1 - back] = 3
        seen = tm.rel_err(mm.reference(cfg, sd, blind, [L - 1]), want).max()
        assert seen > 0.15
        for cuts in ([L], [L - 1, 1], [100, 2, 64, 95, 1]):
            assert tm.rel_err(run(eng, ids, cuts)[-1:], want).max() <= min(LIMIT[dtype], 0.2 * seen), (back, cuts)


def test_chunks_over_wide_and_narrow_blocks_of_columns():
    """Enough heads and portions that the chunked recurrence takes its value columns in blocks of 32 and of 64 (one portion,
    three portions), and few enough that it takes 16; the last block is not full."""
    for heads in (60, 12):
        cfg = mm.config([(mm.delta(heads=heads, kv_heads=4, dim=21, vdim=76, conv=3), 40)], width=70)
        sd = mm.weights(cfg, seed=14)
        eng = engine(cfg, sd, torch.bfloat16)
        seqs = [tm.tokens(cfg, n, seed=70 + n) for n in (140, 75, 64, 9)]
        for group in (seqs[:1], seqs):
            rows = [eng.new_row() for _ in group]
            got = eng.step([(r, s, list(range(len(s)))) for r, s in zip(rows, group)])
            check(got, torch.cat([mm.reference(cfg, sd, s) for s in group]), torch.bfloat16)
            for x, s, r in zip(eng.step([(r, [5], [0]) for r in rows]), group, rows):
                check(x[None], mm.reference(cfg, sd, s + [5], [len(s)]), torch.bfloat16)
                r.close()
    eng.check_device()


@pytest.mark.parametrize("dt", list(DTYPES))
def test_batches_of_unequal_requests_and_reused_slots(dt):
    """Prefills and decode steps of many rows at once against each row alone (by the oracle), one, few and many rows; then
    slots freed and taken by other requests while the rest go on: nothing of the old state is left."""
    cfg, dtype = mm.CONFIGS["plain"], DTYPES[dt]
    sd = mm.weights(cfg, seed=2)
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
            check(torch.stack(g), mm.reference(cfg, sd, s, list(range(k - 1, k + 3))), dtype)
        for r in rows:
            r.close()
    # two go on, one slot changes hands twice; a step mixes portions with single tokens
    a, b = tm.tokens(cfg, 90, seed=40), tm.tokens(cfg, 60, seed=41)
    ra, rb = eng.new_row(), eng.new_row()
    eng.step([(ra, a[:50], []), (rb, b[:30], [])])
    at, bt = 50, 30
    for seed, first in ((42, 20), (43, 1)):    # the second one's first token goes through the decode step
        c = tm.tokens(cfg, 20, seed=seed)
        rc = eng.new_row()
        assert rc.idx == 2
        got = eng.step([(ra, a[at:at + 1], [0]), (rc, c[:first], [first - 1]), (rb, b[bt:bt + 7], [6])])
        for g, s, p in zip(got, (a, c, b), (at, first - 1, bt + 6)):
            check(g[None], mm.reference(cfg, sd, s, [p]), dtype)
        at, bt = at + 1, bt + 7
        rc.close()
    eng.check_device()


@pytest.mark.parametrize("dt", list(DTYPES))
def test_portions_longer_than_a_call_over_small_rings(dt):
    """More rows than one prefill call takes, rings much shorter than the sequences."""
    cfg, dtype = mm.CONFIGS["plain"], DTYPES[dt]
    sd = mm.weights(cfg, seed=6)
    eng = engine(cfg, sd, dtype, max_rows=5, max_seq=300, max_prefill_rows=48)
    forms(eng, 5)
    seqs = [tm.tokens(cfg, 260, seed=60 + i) for i in range(5)]
    rows = [eng.new_row() for _ in range(5)]
    got = eng.step([(r, s[:230], [0, 100, 229]) for r, s in zip(rows, seqs)])
    more = eng.step([(r, s[230:239], [2, 8]) for r, s in zip(rows, seqs)])
    last = [eng.step([(r, [s[239 + j]], [0]) for r, s in zip(rows, seqs)]) for j in range(20)]
    for i, s in enumerate(seqs):
        want = mm.reference(cfg, sd, s, [0, 100, 229, 232, 238, 239, 258])
        check(torch.cat([got[3 * i:3 * i + 3], more[2 * i:2 * i + 2], last[0][i:i + 1], last[19][i:i + 1]]), want, dtype)
    assert eng._ring_spare is not None


def test_a_slot_comes_once_in_a_call():
    cfg = mm.CONFIGS["plain"]
    eng = engine(cfg, mm.weights(cfg), torch.bfloat16)
    two = (C.c_int32 * 2)
    tok = torch.zeros(4, dtype=torch.long, device="cuda")
    with pytest.raises(RuntimeError, match="twice"):
        eng._ck(eng._lib.vuib_lm_prefill(eng._handle, 2, two(1, 1), two(0, 2), two(2, 2), C.c_void_p(tok.data_ptr()), 0, None, None, eng._stream))


@pytest.mark.parametrize("dt", list(DTYPES))
def test_rewind(dt):
    """State cannot be taken back but to the start; keys can, as far as the ring still holds what the window needs."""
    dtype = DTYPES[dt]
    a, b = tm.tokens(mm.CONFIGS["plain"], 150, seed=7), tm.tokens(mm.CONFIGS["plain"], 30, seed=8)
    cfg = mm.CONFIGS["plain"]
    sd = mm.weights(cfg)
    eng = engine(cfg, sd, dtype)
    with eng.new_row() as row:
        eng.step([(row, a, [])])
        with pytest.raises(ValueError, match="state"):
            row.rewind(20)
        row.rewind(0)
        check(eng.step([(row, b, [29])]), mm.reference(cfg, sd, b, [29]), dtype)
    cfg = mm.config([(mm.attention(), 72), (mm.attention(size=20), 40)])
    sd = mm.weights(cfg)
    eng = engine(cfg, sd, dtype, max_prefill_rows=40)
    with eng.new_row() as row:
        eng.step([(row, a, [])])
        with pytest.raises(ValueError, match="held"):
            row.rewind(20)
        row.rewind(130)
        check(eng.step([(row, b, [0, 29])]), mm.reference(cfg, sd, a[:130] + b, [130, 159]), dtype)


def _greedy_ok(cfg, sd, prompt, new, dtype):
    """Every greedy token is the oracle's argmax, unless the oracle's two best are closer than the precision allows."""
    ids = prompt + new
    want = mm.reference(cfg, sd, ids, list(range(len(prompt) - 1, len(ids) - 1)))
    top = want.max(-1)
    chosen = want.gather(1, torch.tensor(new)[:, None])[:, 0]
    slack = 6 * LIMIT[dtype] * (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    assert ((top.values - chosen) <= slack).all()
    return int((top.indices == torch.tensor(new)).sum())


@pytest.mark.parametrize("dt", list(DTYPES))
def test_greedy_generation_through_the_scheduler(dt):
    """More prompts than slots, unequal lengths and stop ids, against the oracle and against each prompt alone."""
    cfg, dtype = mm.CONFIGS["plain"], DTYPES[dt]
    sd = mm.weights(cfg, seed=9)
    eng = engine(cfg, sd, dtype, max_rows=3)
    prompts = [tm.tokens(cfg, 1 + (i * 37) % 80, seed=100 + i) for i in range(8)]
    out = eng.generate(prompts, TokenGenConfig(max_new_tokens=20))
    agree = sum(_greedy_ok(cfg, sd, p, o, dtype) for p, o in zip(prompts, out))
    assert all(len(o) == 20 for o in out) and agree >= (160 if dtype == torch.float32 else 130)
    if dtype == torch.float32:
        assert [eng.generate([p], TokenGenConfig(max_new_tokens=20))[0] for p in prompts] == out
    stop = out[0][4]
    cut = eng.generate(prompts[:1], TokenGenConfig(max_new_tokens=20, stop_ids=(stop,)))[0]
    assert cut == out[0][: out[0].index(stop)]
    with eng.new_row() as row:       # two turns of one row
        assert list(row.stream(prompts[0], TokenGenConfig(max_new_tokens=6))) == out[0][:6]
        more = list(row.stream(out[0][5:6], TokenGenConfig(max_new_tokens=4)))
        _greedy_ok(cfg, sd, prompts[0] + out[0][:6], more, dtype)
    eng.check_device()


def test_long_decoding():
    """Decoding far past the window, over rings that wrap several times."""
    cfg = mm.CONFIGS["plain"]
    sd = mm.weights(cfg, seed=10)
    for dtype in DTYPES.values():
        eng = engine(cfg, sd, dtype, max_rows=1, max_seq=420, max_prefill_rows=32)
        prompt = tm.tokens(cfg, 10, seed=11)
        new = eng.generate([prompt], TokenGenConfig(max_new_tokens=400))[0]
        assert len(new) == 400 and _greedy_ok(cfg, sd, prompt, new, dtype) >= 320
        assert len(eng.generate([prompt], TokenGenConfig(max_new_tokens=1000))[0]) == 411


def test_command_line_and_trace_replay(tmp_path):
    import numpy as np
    from safetensors.torch import save_file

    cfg = mm.CONFIGS["mixed"]
    sd = mm.weights(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(sd, str(tmp_path / "model.safetensors"))
    ids = tm.tokens(cfg, 30)
    want = mm.reference(cfg, sd, ids)
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
