"""What every decoder of the package shares, whatever its layers are: the jit that captures a decode step into a CUDA
graph, `sample`, and the calls a driver makes (jsgrad/models/llama.ts:131-220) — `call`, `call_host`, `decode_loop`.  A
model class supplies `forward` (any number of positions), `_workspace` and `_step` (one token per row, reading tokens and
positions from device memory).
"""
from __future__ import annotations

import numpy as np

from .device import CUDA, CUDAGraph, Tensor

_alpha_counter: dict[tuple, Tensor] = {}  # the reference keeps one module-level counter (jsgrad/models/llama.ts:130)


def sample(logits: Tensor, temp: float, k: int, p: float, af: float, ap: float, u: Tensor | None = None,
           out: Tensor | None = None) -> Tensor:
    """`sample` (jsgrad/models/llama.ts:131-185) per row of fp16 or fp32 logits [rows, V]: argmax with the lowest index among
    equals when temp < 1e-6, else alpha penalties, softmax(logits / temp), top-k, approximate top-p and the multinomial
    draw in one kernel.  `u`: float32 [rows] uniform samples for the draw; by default they come from the restated
    Tensor.rand stream (denograd_b200.rand, seeded by rand.manual_seed)."""
    V = logits.shape[-1]
    rows = logits.numel() // V
    if p < 0 or p > 1:
        raise ValueError("p must be between 0 and 1")
    if k < 0 or k > V:
        raise ValueError("k must be between 0 and numel")
    out = out if out is not None else Tensor.empty((rows,), "int32", logits.dev)
    f32 = logits.dtype == "float32"
    if temp < 1e-6:
        if f32:
            raise ValueError("the greedy pick of fp32 logits is made by the output layer")
        logits.dev.call("jg_argmax", out.ptr, logits.ptr, rows, V)
        return out
    if u is None:
        from . import rand
        u = Tensor(rand.rand(rows, logits.dev.device), device=logits.dev)
    counter_ptr = 0
    if af or ap:
        key = (logits.dev.device, rows, V)
        if key not in _alpha_counter:
            _alpha_counter[key] = Tensor.zeros((rows, V), "int32", logits.dev)
        counter_ptr = _alpha_counter[key].ptr
    logits.dev.call("jg_sample_f32" if f32 else "jg_sample", out.ptr, logits.ptr, u.ptr, counter_ptr, rows, V, float(temp), int(k), float(p), float(af), float(ap))
    return out


class TinyJit:
    """Call 0 runs eagerly, call 1 runs while being captured, later calls replay the capture
    (jsgrad/engine/jit.ts:273-353).  The wrapped function must read its varying inputs from device memory."""

    def __init__(self, fxn, dev: CUDA):
        self.fxn, self.dev = fxn, dev
        self.cnt = 0
        self.graph: CUDAGraph | None = None

    def reset(self) -> None:
        self.cnt, self.graph = 0, None

    def call(self, *args):
        if self.cnt == 0:
            self.fxn(*args)
        elif self.cnt == 1:
            g = CUDAGraph(self.dev)
            with g:
                self.fxn(*args)
            self.graph = g
            g.launch()  # a captured launch list has not run yet
        else:
            self.graph.launch()
        self.cnt += 1

    __call__ = call


class Decoder:
    dev: CUDA
    max_context: int

    def _init_decoder(self, dev: CUDA, jit: bool) -> None:
        self._jit_enabled = jit
        self._forward_jit: dict[int, TinyJit] = {}
        self._loop_graph: dict[int, CUDAGraph] = {}

    # ---- hooks
    def _workspace(self, B: int):
        raise NotImplementedError

    def _step(self, ws, advance: bool = False) -> None:
        raise NotImplementedError

    def forward(self, tokens, start_pos: int, temperature: float = 0.0, top_k: int = 0, top_p: float = 0.8,
                alpha_f: float = 0.0, alpha_p: float = 0.0) -> Tensor:
        raise NotImplementedError

    def _loop_launch(self, ws, n_steps: int) -> Tensor | None:
        """A run of steps in one launch, for a model that has such a kernel: the picks [>= n_steps, B], or None."""
        return None

    def _advance(self, B: int, start_pos: int, n: int) -> None:
        """n tokens from start_pos on are about to be fed to rows 0 .. B - 1.  A K/V cache takes them at any position it has
        reached; a model with recurrent state objects here when its state is elsewhere."""

    def reusable_prefix(self, n: int) -> int:
        """How many of the first n tokens fed last (batch row 0) need not be fed again when a new prompt starts with them."""
        return n

    def _pick(self, ws: _Workspace, temperature: float, top_k: int, top_p: float, alpha_f: float, alpha_p: float) -> Tensor:
        """The token of the last step: the greedy pick the logits kernel already made, or — temperature >= 1e-6 —
        `sample` over the step's logits (jsgrad/models/llama.ts:212)."""
        if temperature < 1e-6:
            return ws.next_tokens
        if getattr(self, "_tp", None) is not None:
            raise NotImplementedError("stochastic sampling over a vocabulary-sharded output layer: gather the logits first")
        return sample(ws.logits, temperature, top_k, top_p, alpha_f, alpha_p, out=ws.next_tokens)

    def call(self, tokens, start_pos: int, temperature: float = 0.0, top_k: int = 0, top_p: float = 0.8,
             alpha_f: float = 0.0, alpha_p: float = 0.0) -> Tensor:
        """Transformer.call (jsgrad/models/llama.ts:214-220): single-token calls after position 0 go through the jit."""
        toks = tokens.numpy() if isinstance(tokens, Tensor) else np.asarray(tokens, dtype=np.int32)
        B, S = toks.shape
        if S == 1 and self._jit_enabled and start_pos != 0:
            if start_pos + 1 > self.max_context:
                raise ValueError(f"start_pos {start_pos} + 1 exceeds max_context {self.max_context}")
            self._advance(B, start_pos, 1)
            ws = self._workspace(B)
            ws.tokens.assign(toks[:, 0])
            ws.pos.assign(np.full((B,), start_pos, np.int32))
            if B not in self._forward_jit:
                self._forward_jit[B] = TinyJit(lambda: self._step(ws), self.dev)
            self._forward_jit[B].call()
            return self._pick(ws, temperature, top_k, top_p, alpha_f, alpha_p)
        return self.forward(toks, start_pos, temperature, top_k, top_p, alpha_f, alpha_p)

    __call__ = call

    def call_host(self, tokens: np.ndarray, start_pos: int) -> np.ndarray:
        """`call(...)` followed by reading the ids back (`.item()` in the reference's loop), for one new token per
        row after position 0, with the copies staged through page-locked memory: per step B*8 bytes go up (tokens and
        positions), the captured step runs, B*4 bytes come back.  tokens: int32 [B, 1] -> int32 [B]."""
        B = tokens.shape[0]
        if start_pos == 0 or not self._jit_enabled:
            return self.call(tokens, start_pos).numpy()
        if start_pos + 1 > self.max_context:
            raise ValueError(f"start_pos {start_pos} + 1 exceeds max_context {self.max_context}")
        self._advance(B, start_pos, 1)
        ws = self._workspace(B)
        ws.h_tokens[:] = tokens.reshape(B)
        ws.h_pos[:] = start_pos
        dev = self.dev
        dev.call("jg_copyin_async", ws.tokens.ptr, ws.h_tokens.ctypes.data, 4 * B)
        dev.call("jg_copyin_async", ws.pos.ptr, ws.h_pos.ctypes.data, 4 * B)
        if B not in self._forward_jit:
            self._forward_jit[B] = TinyJit(lambda: self._step(ws), self.dev)
        self._forward_jit[B].call()
        dev.call("jg_copyout_async", ws.h_next.ctypes.data, ws.next_tokens.ptr, 4 * B)
        dev.synchronize()
        return ws.h_next.copy()

    # ------------------------------------------------------------------------------------------ device-resident loop
    def decode_loop(self, first_tokens, start_pos: int, n_steps: int, collect: bool = True,
                    resume: bool = False) -> np.ndarray | None:
        """Greedy-decode `n_steps` tokens per row with no host round trip between steps: the captured step feeds its
        own output back on the device.  Returns the generated ids [B, n_steps] (read back after the last step), or
        None when `collect` is false.  With `resume` the tokens and positions already on the device (left by the
        previous loop) are continued and `first_tokens` only gives the batch size; nothing is copied or synchronised,
        so a caller can time a run of steps with events."""
        toks = np.asarray(first_tokens, dtype=np.int32).reshape(-1)
        B = toks.shape[0]
        if start_pos + n_steps > self.max_context:
            raise ValueError(f"start_pos {start_pos} + {n_steps} steps exceeds max_context {self.max_context}")
        ws = self._workspace(B)
        if not resume:
            ws.tokens.assign(toks)
            ws.pos.assign(np.full((B,), start_pos, np.int32))
        self._advance(B, start_pos, n_steps)
        hist = self._loop_launch(ws, n_steps)
        if hist is not None:
            if not collect:
                return None
            out = hist.numpy()[:n_steps].T.copy()
            self.dev.call("jg_copy", ws.next_tokens.ptr, hist.ptr + 4 * B * (n_steps - 1), 4 * B)
            return out
        hist = Tensor.empty((n_steps, B), "int32", self.dev) if collect else None

        def keep(i: int) -> None:
            if collect:
                self.dev.call("jg_copy", hist.ptr + 4 * B * i, ws.next_tokens.ptr, 4 * B)

        done = 0
        if B not in self._loop_graph:
            if resume:
                raise ValueError("nothing to resume: run decode_loop once without `resume` first")
            self._step(ws, advance=True)  # the first step runs eagerly (sizes smem attributes), then the step is captured
            keep(0)
            done = 1
            g = CUDAGraph(self.dev)
            with g:
                self._step(ws, advance=True)
            self._loop_graph[B] = g
        g = self._loop_graph[B]
        for i in range(done, n_steps):
            g.launch()
            keep(i)
        return hist.numpy().T.copy() if collect else None

    def last_logits(self, B: int) -> np.ndarray:
        """fp16 logits of the last step widened to fp32 (`.float()` at jsgrad/models/llama.ts:210), [B, vocab]."""
        return self._workspace(B).logits.numpy().astype(np.float32)

    # ---- replayed traces
    def feed(self, slot: int, tokens, start_pos: int, want=()) -> np.ndarray:
        """The next tokens of one request (positions start_pos ..) and the fp32 logits at places `want` among them,
        [len(want), vocab].  This form cuts the portion after every wanted place and serves one request at a time."""
        toks = np.asarray(tokens, np.int32).reshape(1, -1)
        order = sorted(set(int(w) for w in want))
        got, at = {}, 0
        for end in order + ([toks.shape[1] - 1] if not order or order[-1] != toks.shape[1] - 1 else []):
            self.call(toks[:, at:end + 1], start_pos + at)
            got[end], at = self.last_logits(1)[0], end + 1
        return np.stack([got[int(w)] for w in want]) if len(want) else np.zeros((0, self.vocab_size), np.float32)

    def acquire_slot(self) -> int:
        if getattr(self, "_slot_taken", False):
            raise ValueError("this model serves one request at a time outside a batch")
        self._slot_taken = True
        return 0

    def release_slot(self, slot: int) -> None:
        self._slot_taken = False
