"""TokenEngine: serving of token language models on the slot engine.

Rows, buckets, prefill packing, graph capture and continuous batching are ``SlotEngine``'s; a decode step is one
captured graph of the library's kernels per batch bucket, the drawn tokens feeding the next replay on the device.
"""

from __future__ import annotations

import ctypes as C
from collections.abc import Iterator, Sequence
from dataclasses import dataclass

import torch
from torch import Tensor

from . import _lib
from .slots import SlotEngine, _get_bucket, _ptr
from .token_lm import GroupedMixer, TokenLM, abi_config, abi_layers, trig_table

DEFAULT_MAX_SEQ = 2048


@dataclass(frozen=True)
class TokenGenConfig:
    """Sampling and stopping.  ``top_k`` 1 is greedy (first index of the maximum), 0 the whole distribution;
    ``rep_penalty`` > 1 divides (or multiplies) the logits of tokens drawn before, within the last ``rep_window`` draws
    (0: since the start)."""

    max_new_tokens: int = 64
    temperature: float = 1.0
    top_k: int = 1
    rep_penalty: float = 1.0
    rep_window: int = 0
    stop_ids: tuple[int, ...] = ()


class TokenRow:
    """One sequence: an index into the slot cache.  ``offset`` is kept on the host, without a device read."""

    def __init__(self, engine: "TokenEngine", idx: int):
        self._engine, self._idx, self._closed = engine, idx, False

    @property
    def idx(self) -> int:
        return self._idx

    @property
    def offset(self) -> int:
        return self._engine._len[self._idx]

    def prefill(self, ids) -> Tensor:
        """Append tokens; logits (vocab,) after the last."""
        return self._engine.step([(self, ids, [len(ids) - 1])])[0]

    def stream(self, prompt, cfg: TokenGenConfig = TokenGenConfig(), cancel=None) -> Iterator[int]:
        yield from self._engine._stream_row(self, prompt, cfg, cancel)

    def rewind(self, offset: int = 0) -> int:
        if not 0 <= offset <= self.offset:
            raise ValueError(f"cannot rewind from {self.offset} to {offset}")
        return self._engine._rewind_row(self, offset)

    def close(self) -> None:
        if not self._closed:
            self._engine._release_row(self)
            self._closed = True

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        self.close()


class TokenEngine(SlotEngine):
    _ABI = "vuib_lm_"
    _ROW = TokenRow

    def __init__(self, name: str | None = None, *, model: TokenLM | None = None, max_rows: int = 1, max_seq: int | None = None,
                 max_prefill_rows: int = 1024, seed: int = 0):
        if not torch.cuda.is_available():
            raise RuntimeError("vui_b200.TokenEngine needs a CUDA device (sm_100a); there is no CPU path")
        if model is None:
            from .registry import load_model

            model = load_model(name)
        if not isinstance(model, TokenLM):
            raise ValueError("not a token model; open it with vui_b200.open_engine")
        self.model, self.device, self.seed = model, model.device, seed
        self.max_seq = max_seq or DEFAULT_MAX_SEQ
        self.max_prefill_rows = max_prefill_rows
        self.V = model.config.vocab
        self._init_slots(max_rows)
        self._len = [0] * (max_rows + 1)
        self._lib = _lib.load_lm()
        self._handle = C.c_void_p()
        self._graphs: dict[tuple[int, bool], torch.cuda.CUDAGraph] = {}
        self._sampling_key = None
        self._setup_native()

    def _setup_native(self) -> None:
        m, dev, c = self.model, self.device, self.model.config
        n_slots = self.max_rows + 1
        b16 = m.dtype == torch.bfloat16
        cfg = abi_config(c, dtype=_lib.LM_BF16 if b16 else _lib.LM_F32, n_slots=n_slots, max_seq=self.max_seq, max_rows=self.max_rows,
                         max_prefill_rows=self.max_prefill_rows)
        _lib.check(None, self._lib.vuib_lm_create(C.byref(cfg), abi_layers(c), C.byref(self._handle)))
        dims = []                       # per run of a layer
        for i in range(len(c.runs)):
            d = _lib.VuibLmDims()
            self._ck(self._lib.vuib_lm_layer_dims(self._handle, i, C.byref(d)))
            dims.append(d)
        nbytes = C.c_size_t()
        self._ck(self._lib.vuib_lm_workspace_bytes(self._handle, C.byref(nbytes)))
        self._ws = torch.zeros(nbytes.value + 256, device=dev, dtype=torch.uint8)
        ws_ptr = (self._ws.data_ptr() + 255) & ~255
        self._ck(self._lib.vuib_lm_bind_workspace(self._handle, C.c_void_p(ws_ptr), nbytes.value))
        # what a slot holds per run of a layer: cached rows, key/value rings, or recurrent state
        self.cache = [torch.zeros(n_slots, d.slot_bytes, device=dev, dtype=torch.uint8) for d in dims]
        # positions a slot's shortest ring holds beyond its window (None: every position is kept)
        spare = [d.cap - s.window for d, s in zip(dims, (c.layers[i].mixer for i in c.runs))
                 if isinstance(s, GroupedMixer) and d.cap < self.max_seq]
        self._ring_spare = min(spare) if spare else None
        self._ring_top = [0] * n_slots   # the most positions a slot has held since it was taken
        self.seq_lens = torch.zeros(n_slots, device=dev, dtype=torch.int32)
        ptrs = (C.c_void_p * len(self.cache))(*[t.data_ptr() for t in self.cache])
        self._ck(self._lib.vuib_lm_bind_cache(self._handle, ptrs, C.c_void_p(self.seq_lens.data_ptr())))
        head, packed = m.packed([dims[c.runs.index(i)] if i in c.runs else None for i in range(len(c.layers))])
        self._trig: dict[tuple[float, int], Tensor] = {}
        lw = (_lib.VuibLmLayerWeights * len(c.runs))()
        for i, n in enumerate(c.runs):
            for k, t in packed[n].items():
                setattr(lw[i], k, t.data_ptr())
            mixer = c.layers[n].mixer
            if mixer.rot_dims:
                key = (mixer.rot_base, mixer.rot_dims)
                if key not in self._trig:
                    self._trig[key] = trig_table(*key, self.max_seq).to(dev)
                lw[i].trig = self._trig[key].data_ptr()
        hw = _lib.VuibLmHeadWeights(**{k: t.data_ptr() for k, t in head.items()})
        self._ck(self._lib.vuib_lm_bind_weights(self._handle, C.byref(hw), lw))
        # static I/O of the captured steps
        N = self.max_rows
        self._g_tokens = torch.zeros(N, device=dev, dtype=torch.long)
        self._g_logits = torch.zeros(N, self.V, device=dev, dtype=torch.float32)
        self._g_slot_idx = torch.arange(N, device=dev, dtype=torch.int32)
        self._g_seq_inc = torch.ones(N, device=dev, dtype=torch.int32)
        self._h_tokens = torch.zeros(N, dtype=torch.long).pin_memory()
        self._done = torch.cuda.Event()
        self._apply_cfg(TokenGenConfig())

    # ---------------------------------------------------------- row lifecycle
    def _set_len(self, slot: int, n: int) -> None:
        super()._set_len(slot, n)
        self._len[slot] = n
        if n == 0:
            self._ring_top[slot] = 0

    def _grow(self, slot: int, n: int) -> None:
        """The host's count of a slot's positions, after a call that appended to it."""
        self._len[slot] = n
        self._ring_top[slot] = max(self._ring_top[slot], n)

    def _rewind_row(self, row, offset: int) -> int:
        if 0 < offset < row.offset:
            if self.model.config.recurrent:
                raise ValueError("recurrent state cannot be taken back: rewind to 0")
            if self._ring_spare is not None and self._ring_top[row.idx] - offset >= self._ring_spare:
                raise ValueError(f"the keys that position {offset} sees are no longer held")
        return super()._rewind_row(row, offset)

    def reset(self) -> None:
        super().reset()
        self._len = [0] * (self.max_rows + 1)
        self._ring_top = [0] * (self.max_rows + 1)

    # --------------------------------------------------------------- sampling
    def _apply_cfg(self, cfg: TokenGenConfig) -> None:
        key = (float(cfg.temperature), int(cfg.top_k), float(cfg.rep_penalty), int(min(cfg.rep_window, 64)), int(self.seed))
        if key == self._sampling_key:
            return
        sp = _lib.VuibSampling(key[0], key[1], 0, key[2], key[3], 0, key[4])
        self._ck(self._lib.vuib_lm_set_sampling(self._handle, C.byref(sp), self._stream))
        self._sampling_key = key

    def _sample(self, slots: Tensor, logits: Tensor) -> Tensor:
        """One token per row of logits (B, vocab) fp32 (rewritten under a repetition penalty), on the device."""
        out = torch.empty(logits.shape[0], device=self.device, dtype=torch.long)
        self._ck(self._lib.vuib_lm_sample(self._handle, logits.shape[0], _ptr(slots), _ptr(logits), _ptr(out), self._stream))
        return out

    # ------------------------------------------------------------------ steps
    def _step_call(self, B: int, sample: bool) -> None:
        self._ck(self._lib.vuib_lm_decode(self._handle, B, _ptr(self._g_slot_idx), _ptr(self._g_seq_inc), _ptr(self._g_tokens),
                                          _ptr(self._g_logits), self._stream))
        if sample:
            self._ck(self._lib.vuib_lm_sample(self._handle, B, _ptr(self._g_slot_idx), _ptr(self._g_logits),
                                              _ptr(self._g_tokens), self._stream))

    def _step_graph(self, B: int, sample: bool) -> torch.cuda.CUDAGraph:
        g = self._graphs.get((B, sample))
        if g is None:
            g = self._capture_graph(lambda: self._step_call(B, sample), [self._g_tokens])
            self._graphs[(B, sample)] = g
        return g

    def _decode_replay(self, n: int, sample: bool) -> None:
        """One token for the first n rows of the static buffers."""
        g = self._step_graph(_get_bucket(n, self._buckets), sample)
        self._pad_to_bucket(n)
        g.replay()

    def _aim(self, slots: Sequence[int]) -> None:
        n = len(slots)
        self._g_slot_idx[:n] = torch.tensor(slots, device=self.device, dtype=torch.int32)
        self._g_seq_inc[:n].fill_(1)

    @torch.inference_mode()
    def step(self, entries) -> Tensor:
        """Run given tokens: entries of (row, ids, places whose logits are wanted).  Logits (wanted, vocab) fp32 in the
        order of the entries and places.  Single tokens go through the decode graph, portions through the prefill."""
        if len({row.idx for row, _, _ in entries}) != len(entries):
            raise ValueError("a row appears twice in one step")
        for row, ids, want in entries:
            if row.offset + len(ids) > self.max_seq:
                raise RuntimeError(f"{len(ids)} tokens overflow max_seq={self.max_seq}")
            if len(ids) < 1 or any(not 0 <= t < self.V for t in ids):
                raise ValueError("an entry needs at least one token, each inside the vocabulary")
            if any(not 0 <= w < len(ids) for w in want):
                raise ValueError("a wanted place lies outside its entry")
        n_want = sum(len(w) for _, _, w in entries)
        out = torch.empty(n_want, self.V, device=self.device, dtype=torch.float32)
        at, single, portions = 0, [], []
        for row, ids, want in entries:
            (single if len(ids) == 1 else portions).append((row, ids, want, at))
            at += len(want)
        if single:
            n = len(single)
            self._aim([row.idx for row, _, _, _ in single])
            self._g_tokens[:n] = torch.tensor([ids[0] for _, ids, _, _ in single], device=self.device)
            self._decode_replay(n, False)
            for k, (row, _, want, a) in enumerate(single):
                self._grow(row.idx, row.offset + 1)
                if want:
                    out[a:a + len(want)] = self._g_logits[k]
        if portions:
            self._prefill(portions, out)
        return out

    def _prefill(self, portions, out: Tensor) -> None:
        """(row, ids, wanted places, first row of ``out``) through the packed prefill."""
        seen = [0] * len(portions)   # tokens of each portion that earlier calls ran

        def run(pend):
            n = len(pend)
            slot, pos, ln = ((C.c_int32 * n)(*v) for v in zip(*[(s, p, t.shape[0]) for s, p, t, _ in pend]))
            want, dst, r0 = [], [], 0
            for _, _, t, k in pend:
                _, _, w, a = portions[k]
                lo = seen[k]
                for j, place in enumerate(w):
                    if lo <= place < lo + t.shape[0]:
                        want.append(r0 + place - lo)
                        dst.append(a + j)
                seen[k] += t.shape[0]
                r0 += t.shape[0]
            tokens = torch.cat([t for _, _, t, _ in pend]).to(self.device)
            rows = torch.tensor(want, dtype=torch.int32).to(self.device) if want else None
            logits = torch.empty(len(want), self.V, device=self.device, dtype=torch.float32) if want else None
            self._ck(self._lib.vuib_lm_prefill(self._handle, n, slot, pos, ln, _ptr(tokens), len(want), _ptr(rows), _ptr(logits),
                                               self._stream))
            for s, p, t, _ in pend:
                self._grow(s, p + t.shape[0])
            if want:
                out[torch.tensor(dst, device=self.device)] = logits

        self._pack_rows([(row, torch.as_tensor(ids, dtype=torch.long)) for row, ids, _, _ in portions], run)

    # ------------------------------------------------------------- generation
    def _read_tokens(self, n: int) -> list[int]:
        """The step's one device->host read."""
        self._h_tokens[:n].copy_(self._g_tokens[:n], non_blocking=True)
        self._done.record()
        self._done.synchronize()
        return self._h_tokens[:n].tolist()

    def _first_tokens(self, rows: list[TokenRow], prompts) -> Tensor:
        for row in rows:
            self._ck(self._lib.vuib_lm_reset_slot(self._handle, row.idx, self._stream))
        logits = self.step([(row, p, [len(p) - 1]) for row, p in zip(rows, prompts)])
        slots = torch.tensor([row.idx for row in rows], device=self.device, dtype=torch.int32)
        return self._sample(slots, logits)

    @torch.inference_mode()
    def generate(self, prompts: Sequence[Sequence[int]], cfg: TokenGenConfig = TokenGenConfig()) -> list[list[int]]:
        """Continuous batching: any number of prompts of token ids over ``max_rows`` slots; new tokens in input order
        (a stop id ends a request and is not part of it)."""
        self._apply_cfg(cfg)
        out: list[list[int]] = [[] for _ in prompts]
        stop = set(cfg.stop_ids)
        last: dict[int, int] = {}

        def goes_on(row, ri: int, tok: int) -> bool:
            if tok in stop:
                return False
            out[ri].append(tok)
            last[row.idx] = tok
            return len(out[ri]) < cfg.max_new_tokens and row.offset < self.max_seq

        def admit(batch):
            if cfg.max_new_tokens < 1:
                return {}
            rows = []
            for _, slot in batch:
                self._set_len(slot, 0)
                self._rows[slot] = TokenRow(self, slot)
                rows.append(self._rows[slot])
            toks = self._first_tokens(rows, [prompts[ri] for ri, _ in batch]).tolist()
            return {row.idx: (row, ri) for row, (ri, _), tok in zip(rows, batch, toks) if goes_on(row, ri, tok)}

        placed: list[int] = []   # slots the static buffers are aimed at, their last tokens in place

        def step(slots, states):
            n = len(slots)
            if placed != slots:
                self._aim(slots)
                self._g_tokens[:n] = torch.tensor([last[s] for s in slots], device=self.device)
                placed[:] = slots
            self._decode_replay(n, True)
            done = []
            for s, (row, ri), tok in zip(slots, states, self._read_tokens(n)):
                self._grow(s, row.offset + 1)
                if not goes_on(row, ri, tok):
                    done.append(s)
            if done:
                placed.clear()
            return done

        if self._rows:
            raise RuntimeError("generate() needs every row: close the rows in use first")
        self._run_continuous(len(prompts), admit, step)
        return out

    @torch.inference_mode()
    def _stream_row(self, row: TokenRow, prompt, cfg: TokenGenConfig, cancel=None) -> Iterator[int]:
        """Tokens of one row as they are drawn; the row keeps its cache for another turn."""
        self._apply_cfg(cfg)
        tok = int(self._first_tokens([row], [prompt])[0]) if cfg.max_new_tokens > 0 else None
        n = 0
        while tok is not None and tok not in cfg.stop_ids:
            yield tok
            n += 1
            if n >= cfg.max_new_tokens or row.offset >= self.max_seq or (cancel is not None and cancel.is_set()):
                return
            self._apply_cfg(cfg)   # the consumer may have used the engine in between
            self._aim([row.idx])
            self._g_tokens[0] = tok
            self._decode_replay(1, True)
            tok = self._read_tokens(1)[0]
            self._grow(row.idx, row.offset + 1)
