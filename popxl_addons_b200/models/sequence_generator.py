"""Serving of models with per-sequence state (recurrent state, caches): portions of prompts, decoding, logits on request and
greedy generation for a batch of unequal prompts.

A model object (see `models/dunelix.py`) describes its weights, its state and the ops of one portion; everything else is here
and does not know the architecture:

* **slots**: the batch axis of all state tensors. A request takes a slot (`admit`), its tokens advance the slot's position,
  `release` gives it back. A slot needs no clearing: a sequence at position 0 starts from the empty state.
* **portions**: `step` runs the next tokens of any of the live requests, of unequal lengths, cut anywhere. Portion lengths are
  rounded up to a ladder of sizes; padded rows touch neither caches nor recurrent state. One `Program` per size, captured
  into a CUDA graph at its second use.
* **decoding**: tokens, positions and the output buffer stay on the device, so a decoding step is one graph replay.
"""
from typing import Dict, List, Mapping, Optional, Sequence

import numpy as np
import torch

from .. import xl
from ..xl import ops

__all__ = ["SequenceGenerator", "portion_size"]


def portion_size(n: int) -> int:
    """Smallest ladder size >= n: 1, 2, 4, 8, 16, then eight steps per power of two (at most an eighth of the rows are
    padding), never finer than 16."""
    if n <= 16:
        return 1 << (n - 1).bit_length()
    step = max(16, 1 << ((n - 1).bit_length() - 4))
    return (n + step - 1) // step * step


class SequenceGenerator:
    def __init__(self, model, batch: int = 1, max_seq: int = 2048, max_portion: int = 4096, max_new_tokens: int = 256,
                 device: str = "auto", cuda_graphs: bool = True, use_native: Optional[bool] = None):
        """`max_seq`: positions a slot can hold; `max_portion`: tokens per sequence of one step's graph (longer portions are
        run in several); `max_new_tokens`: rows of the device buffer that collects generated tokens."""
        if batch < 1 or max_seq < 1:
            raise ValueError("batch and max_seq must be positive")
        self.model, self.batch, self.max_seq = model, batch, max_seq
        self.max_portion = portion_size(min(max_portion, max_seq))
        self.max_new = max_new_tokens
        self.ir = xl.Ir()
        self.ir.options.cuda_graphs = self.ir.options.cuda_graphs and cuda_graphs
        self._vars: Dict[str, xl.Variable] = {}
        self._mutable = set()
        with self.ir.main_graph:
            for name, (shape, dt) in model.weights().items():
                self._vars[name] = xl.variable(xl.LazyInit(shape, np.float32, "zeros"), dt, name)
            for name, arr in model.tables(max_seq).items():
                self._vars[name] = xl.variable(arr, xl.float32, name)
            state = dict(model.state(batch, max_seq))
            state["stream"] = ((batch * self.max_portion, model.width), xl.float32)
            state.update(pos=((batch,), xl.int32), count=((batch,), xl.int32), current=((batch,), xl.int32),
                         step=((1,), xl.int32), generated=((max_new_tokens, batch), xl.int32))
            for name, (shape, dt) in state.items():
                self._vars[name] = xl.variable(xl.LazyInit(shape, np.float32, "zeros"), dt, name)
                self._mutable.add(name)
            self._ctrl_in = xl.h2d_stream((2, batch), xl.int32, "slot_positions")
            self._tokens_out = xl.d2h_stream((max_new_tokens, batch), xl.int32, "generated")
        self.session = xl.Session(self.ir, device, use_native=use_native)
        self._programs: Dict[tuple, dict] = {}
        self.lengths = [0] * batch          # positions held by every slot (host mirror of the device-side `pos`)
        self.slots: Dict[object, int] = {}  # live request -> slot
        self._free = list(range(batch))[::-1]

    # -- weights -------------------------------------------------------------------------------------------------------
    def load(self, tensors: Mapping[str, torch.Tensor]):
        """Copy program tensors (`model.convert(...)` or `model.random_weights(...)`) into the session's variables."""
        names = set(self.model.weights())
        if set(tensors) != names:
            raise ValueError(f"weights do not fit: missing {sorted(names - set(tensors))[:8]}, unexpected "
                             f"{sorted(set(tensors) - names)[:8]}")
        for name, value in tensors.items():
            dst = self.session._vars[self._vars[name]][0]
            if tuple(dst.shape) != tuple(value.shape):
                raise ValueError(f"weight {name!r} has shape {tuple(value.shape)}, expected {tuple(dst.shape)}")
            dst.copy_(value)
        return self

    def load_checkpoint(self, ckpt: Mapping[str, torch.Tensor]):
        return self.load(self.model.convert(ckpt, self.session.device))

    # -- slots ---------------------------------------------------------------------------------------------------------
    def admit(self, request) -> int:
        """Give a request a slot; its first token will be at position 0."""
        if request in self.slots:
            raise ValueError(f"request {request!r} already holds a slot")
        if not self._free:
            raise RuntimeError(f"all {self.batch} slots are in use")
        slot = self._free.pop()
        self.slots[request] = slot
        self.lengths[slot] = 0
        return slot

    def release(self, request) -> None:
        slot = self.slots.pop(request)
        self.lengths[slot] = 0
        self._free.append(slot)

    # -- programs --------------------------------------------------------------------------------------------------------
    def _program(self, key, build):
        entry = self._programs.get(key)
        if entry is None:
            entry = {"program": xl.Program(self.ir, "_".join(str(k) for k in key))}
            with entry["program"] as p:
                build(entry, lambda name: p.use(self._vars[name], by_ref=name in self._mutable))
            self._programs[key] = entry
        return entry

    def _sample(self, t, h):
        """Greedy choice for every slot: becomes the current token and a row of the output buffer."""
        _, tok = ops.argmax_rows(self.model.logits(t, h), self.model.vocab, 0)
        ops.var_updates.copy_var_update_(t("current"), tok)
        ops.store_row_(t("generated"), t("step"), tok)
        ops.advance_position_(t("step"))

    def _portion_program(self, T: int, sample: bool):
        def build(entry, t):
            entry["tokens"] = xl.h2d_stream((self.batch * T,), xl.int32, f"tokens_{T}")
            ctrl = ops.host_load(self._ctrl_in)
            tokens = ops.host_load(entry["tokens"])
            ops.var_updates.copy_var_update_(t("pos"), ctrl[0])
            ops.var_updates.copy_var_update_(t("count"), ctrl[1])
            self.model.portion(T, t, tokens, t("pos"), t("count"), final_norm=False)
            if sample:
                self._sample(t, self.model.select(t, t("count"), stride=T, offset=1))
            ops.advance_by_(t("pos"), t("count"))

        return self._program(("portion", T, "sample") if sample else ("portion", T), build)

    def _decode_program(self):
        def build(entry, t):
            h = self.model.portion(1, t, t("current"), t("pos"), t("count"), final_norm=True)
            self._sample(t, h)
            ops.advance_by_(t("pos"), t("count"))

        return self._program(("decode",), build)

    def _logits_program(self, n: int):
        def build(entry, t):
            entry["rows"] = xl.h2d_stream((n,), xl.int32, f"rows_{n}")
            entry["logits"] = xl.d2h_stream((n, self.model.vocab), xl.float32, f"logits_{n}")
            rows = ops.host_load(entry["rows"])
            ops.host_store(entry["logits"], self.model.logits(t, self.model.select(t, rows)))

        return self._program(("logits", n), build)

    # -- steps -----------------------------------------------------------------------------------------------------------
    def _run_portion(self, part: Mapping[int, Sequence[int]], sample: bool = False) -> int:
        """`part`: slot -> its next tokens (at most `max_portion`). Returns the rows per sequence of the program."""
        T = portion_size(max(len(v) for v in part.values()))
        entry = self._portion_program(T, sample)
        tokens = np.zeros((self.batch, T), np.int32)
        ctrl = np.zeros((2, self.batch), np.int32)
        ctrl[0] = self.lengths
        for slot, toks in part.items():
            tokens[slot, :len(toks)] = toks
            ctrl[1, slot] = len(toks)
        self.session.run_program(entry["program"], {self._ctrl_in: ctrl, entry["tokens"]: tokens.reshape(-1)}, fetch=False)
        for slot, toks in part.items():
            self.lengths[slot] += len(toks)
        return T

    def _read_logits(self, rows: Sequence[int]) -> np.ndarray:
        n = portion_size(len(rows))
        entry = self._logits_program(n)
        padded = np.zeros((n,), np.int32)
        padded[:len(rows)] = rows
        out = self.session.run_program(entry["program"], {entry["rows"]: padded})[entry["logits"]]
        return np.asarray(out).reshape(n, -1)[:len(rows)]

    def step(self, entries: Mapping[object, Sequence[int]], want: Optional[Mapping[object, Sequence[int]]] = None
             ) -> Dict[object, np.ndarray]:
        """Advance live requests by their next tokens. `want[request]`: places among these tokens whose logits are returned,
        `{request: (len(want), vocab) float32}` in the given order."""
        want = {r: list(w) for r, w in (want or {}).items() if len(w)}
        todo = {}
        for req, toks in entries.items():
            slot, n = self.slots[req], len(toks)
            if self.lengths[slot] + n > self.max_seq:
                raise ValueError(f"request {req!r} would hold {self.lengths[slot] + n} positions, a slot has {self.max_seq}")
            if n and not (0 <= min(toks) and max(toks) < self.model.vocab):
                raise ValueError(f"request {req!r} has a token outside the vocabulary of {self.model.vocab}")
            if any(not 0 <= w < n for w in want.get(req, ())):
                raise ValueError(f"request {req!r} asks for logits outside its {n} tokens")
            if n:
                todo[req] = list(toks)
        out = {r: np.empty((len(w), self.model.vocab), np.float32) for r, w in want.items()}
        done = 0
        while todo:
            part = {self.slots[r]: toks[done:done + self.max_portion] for r, toks in todo.items()}
            T = self._run_portion(part)
            picks = [(r, k, self.slots[r] * T + w - done) for r in todo for k, w in enumerate(want.get(r, ()))
                     if done <= w < done + self.max_portion]
            if picks:
                for (r, k, _), row in zip(picks, self._read_logits([row for _, _, row in picks])):
                    out[r][k] = row
            done += self.max_portion
            todo = {r: toks for r, toks in todo.items() if len(toks) > done}
        return out

    def generate(self, prompts: Sequence[Sequence[int]], max_new_tokens: int) -> List[np.ndarray]:
        """Greedy continuation of every prompt; prompts beyond the number of slots run in further batches."""
        if max_new_tokens < 1 or max_new_tokens > self.max_new:
            raise ValueError(f"max_new_tokens must be in [1, {self.max_new}]")
        if self.slots:
            raise RuntimeError("generate() needs all slots: release the live requests first")
        out: List[np.ndarray] = []
        for lo in range(0, len(prompts), self.batch):
            out += self._generate_batch(prompts[lo:lo + self.batch], max_new_tokens)
        return out

    def _generate_batch(self, prompts, n_new: int) -> List[np.ndarray]:
        if any(len(p) < 1 or len(p) + n_new - 1 > self.max_seq for p in prompts):
            raise ValueError(f"prompts must hold between 1 and {self.max_seq - n_new + 1} tokens")
        reqs = list(range(len(prompts)))
        slot = {r: self.admit(r) for r in reqs}
        try:
            # all but the last portion of every prompt, then the last ones together: they end in the first sampled token
            last = {r: prompts[r][(len(prompts[r]) - 1) // self.max_portion * self.max_portion:] for r in reqs}
            head = {r: prompts[r][:len(prompts[r]) - len(last[r])] for r in reqs}
            self.step({r: h for r, h in head.items() if len(h)})
            self._set_device("step", 0)
            self.session.record_timestamp("start")
            self._run_portion({slot[r]: last[r] for r in reqs}, sample=True)
            self.session.record_timestamp("prefill_done")
            self._set_device("count", [1 if s in slot.values() else 0 for s in range(self.batch)])
            decode = self._decode_program()["program"]
            for _ in range(n_new - 1):
                self.session.run_program(decode, fetch=False)
            self.session.record_timestamp("decode_done")
            got = self.session.get_tensor_data(self._vars["generated"])
            if self.session.use_native:
                from ..ops import native

                native.check_gemm_errors()
        finally:
            for r in reqs:
                self.release(r)
        return [np.array(got[:n_new, slot[r]], np.int32) for r in reqs]

    def _set_device(self, name: str, value):
        v = self.session._vars[self._vars[name]][0]
        v.copy_(torch.as_tensor(value, dtype=v.dtype).reshape(-1).expand_as(v))

    def decode_ms(self) -> float:
        return self.session.elapsed_ms("prefill_done", "decode_done")

    def prefill_ms(self) -> float:
        return self.session.elapsed_ms("start", "prefill_done")
