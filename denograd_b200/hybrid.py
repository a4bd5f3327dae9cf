"""Decoders given as a list of layers, each with its own kind of mixer, an optional feed-forward and an optional token input.

  stream x (fp32) = embedding rows * scale
  per layer   x <- x + norm_b(mixer(norm(x)));  with a feed-forward: x <- x + norm_b(ff(norm(x)));  with a token input
              x <- x + norm_b(W_proj (gelu(W_gate x) * the layer's part of the token's row in a second table))
  logits      = head norm(x)

What differs between architectures beyond sizes is a `Design` (`DESIGNS`): whether sublayers read a normed stream or the stream
itself, whether norm weights are stored around zero, a head of its own or the embedding table, and which feed-forward a
"dense" one is.

Mixers (`MIXERS`): ``mingru`` (gated linear recurrence), ``latent_attention`` (low-rank keys and values, sliding window,
sinks, YaRN rotary), ``delta`` (gated delta rule with short convolutions), and mixers made of one or more `Branches` side by
side: ``window_attention`` (grouped heads, sliding window and kept first tokens), ``lightning`` (linear attention with a decay
per head), ``mlstm`` (exponentially gated matrix memory), ``parallel`` (the first two of these).  Norms divide groups of
channels by their own root mean square.  A model's configuration gives every size; `ARCHITECTURES` (registry.py) maps a
configuration to the model.

How a step runs: each layer contributes library calls to a *plan* — descriptors of device addresses, made once per
workspace — and a step walks the plan with the batch (sequences, tokens per sequence, positions, slots) as the only
argument that changes.  With 1-2 rows the plan has no calls for norms and residual sums: the projection that follows takes
the fp32 stream and does them in its prologue, the minGRU recurrence is the epilogue of its projections, and the norm and
output gate after a linear recurrence are the prologue of the output projection.  A decode step is captured into a CUDA graph.
"""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass

import numpy as np

from . import ffi
from .cache import SlotStates
from .decoder import Decoder, TinyJit
from .device import CUDA, Tensor
from .nn import _dev

DTYPES = {"float32": ffi.JG_F32, "bfloat16": ffi.JG_BF16}


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


# ------------------------------------------------------------------------------------------------ parameters
class Param:
    """Where one checkpoint tensor goes: `shape` values plus `offset`, rows of `cols` in device rows `ld` apart (zeros in
    between)."""

    def __init__(self, tensor: Tensor, shape: tuple, ld: int | None = None, offset: float = 0.0):
        self.tensor, self.shape, self.ld, self.offset = tensor, tuple(shape), ld, offset

    @property
    def ptr(self) -> int:
        return self.tensor.ptr

    def assign(self, arr: np.ndarray) -> None:
        arr = np.asarray(arr, np.float32) + np.float32(self.offset)
        if self.ld is not None and self.ld != self.shape[-1]:
            wide = np.zeros(self.shape[:-1] + (self.ld,), np.float32)
            wide[..., :self.shape[-1]] = arr
            arr = wide
        self.tensor.assign(arr)


class ColumnParam(Param):
    """Columns [at, at + shape[1]) of a matrix whose columns come from several checkpoint tensors (`Columns`)."""

    def __init__(self, owner: "Columns", shape: tuple, at: int):
        super().__init__(owner.weight, shape, owner.ld)
        self.owner, self.at = owner, at

    @property
    def ptr(self) -> int:
        return self.tensor.ptr + self.at * self.tensor.nbytes // self.tensor.numel()

    def assign(self, arr: np.ndarray) -> None:
        self.owner.put(self, np.asarray(arr, np.float32))


class Matrix:
    """Projection weights [N][ld] of the model's element type; `parts` names runs of rows after checkpoint tensors: (name,
    rows), or (name, rows, alignment of the first row) with rows of zeros in between."""

    def __init__(self, m: "HybridTransformer", params: dict, parts: list[tuple], K: int):
        self.K, self.ld, self.row0, r = K, round_up(K, 8), {}, 0
        for name, n, *align in parts:
            self.row0[name] = r = round_up(r, align[0] if align else 1)
            r += n
        self.N = r
        self.weight = Tensor.zeros((self.N, self.ld), m.dtype, m.dev)
        for name, n, *_ in parts:
            r = self.row0[name]
            params[name] = Param(self.weight.view_rows(r, r + n), (n, K), self.ld)

    @property
    def ptr(self) -> int:
        return self.weight.ptr

    def rows_ptr(self, name: str) -> int:
        return self.weight.ptr + self.row0[name] * self.ld * self.weight.nbytes // self.weight.numel()


class Columns:
    """Projection weights [N][ld] whose columns are those of several checkpoint tensors (name, columns), each from a multiple
    of 8 on, zeros in between: one projection of several inputs side by side.  `col0`: where each starts."""

    def __init__(self, m: "HybridTransformer", params: dict, parts: list[tuple[str, int]], N: int):
        self.N, self.col0, c = N, {}, 0
        for name, n in parts:
            self.col0[name] = c = round_up(c, 8)
            c += n
        self.K, self.ld = c, round_up(c, 8)
        self.weight = Tensor.zeros((N, self.ld), m.dtype, m.dev)
        self.params = [ColumnParam(self, (N, n), self.col0[name]) for name, n in parts]
        params.update({name: q for (name, _), q in zip(parts, self.params)})
        self._host: np.ndarray | None = None
        self._missing: set[int] = set()

    @property
    def ptr(self) -> int:
        return self.weight.ptr

    def put(self, param: ColumnParam, arr: np.ndarray) -> None:
        """The matrix goes to the device when the last of its tensors has come."""
        if self._host is None:
            self._host, self._missing = np.zeros((self.N, self.ld), np.float32), {q.at for q in self.params}
        self._host[:, param.at:param.at + param.shape[1]] = arr
        self._missing.discard(param.at)
        if not self._missing:
            self.weight.assign(self._host)
            self._host = None


def vector(m: "HybridTransformer", params: dict, parts: list[tuple[str, tuple]], pad: int = 0, offset: float = 0.0) -> Tensor:
    """fp32 parameters of consecutive checkpoint tensors (scalars per channel, taps, ...) plus `offset`, `pad` zeros behind."""
    width = parts[0][1][1:]
    n = sum(s[0] for _, s in parts)
    t = Tensor.zeros((n + pad,) + width, "float32", m.dev)
    r = 0
    for name, s in parts:
        params[name] = Param(t.view_rows(r, r + s[0]), s, offset=offset)
        r += s[0]
    return t


def row_vector(m: "HybridTransformer", params: dict, w: Matrix, parts: list[tuple[str, str, int]]) -> Tensor:
    """fp32, one value per row of `w`: (name, part of w it belongs to, rows); zeros elsewhere."""
    t = Tensor.zeros((w.N,), "float32", m.dev)
    for name, part, n in parts:
        params[name] = Param(t.view_rows(w.row0[part], w.row0[part] + n), (n,))
    return t


# ------------------------------------------------------------------------------------------------ plans
class Plan:
    """The calls of one step on one workspace, and where the residual stream stands while it is being written.

    A sublayer's output `y` is not added to the stream by the kernel that made it: the sum, the norm before it and the norm
    after it happen together in whatever reads the stream next (`into`)."""

    def __init__(self, model: "HybridTransformer", ws: "_Rows", fused: bool, single: bool):
        self.model, self.ws, self.fused, self.single = model, ws, fused, single
        self.calls: list[tuple] = []
        self.cur = 0          # stream buffer that holds x
        self.pending = None   # norm weight of a sum that is still to be made (ws.y)

    def call(self, name: str, *args) -> None:
        self.calls.append((name,) + args)

    def stream(self, w_norm: Tensor | None, rows: int = 0, keep: bool = True, plain: bool = False) -> ffi.StreamDesc:
        m, ws = self.model, self.ws
        out = 0
        src = ws.x[self.cur].ptr
        y, w_add = (ws.y.ptr, self.pending.ptr) if self.pending is not None else (0, 0)
        if self.pending is not None and keep:
            if self.fused:
                self.cur ^= 1
            out = ws.x[self.cur].ptr
            self.pending = None
        return ffi.StreamDesc(m.width, m.groups, m.eps, int(plain), src, y, w_add, out, w_norm.ptr if w_norm is not None else 0, rows)

    def dense(self, desc: ffi.DenseDesc, w_norm: Tensor | None) -> None:
        """A projection of the normed stream, or (w_norm None) of the stream itself."""
        if self.fused:
            desc.stream = self.stream(w_norm, plain=w_norm is None)
        else:
            self.call("jg_stream_norm", self.stream(w_norm, plain=w_norm is None), self.ws.h.ptr, self.model.ld_width, self.model.dt)
            desc.x, desc.ldx = self.ws.h.ptr, self.model.ld_width
        self.call("jg_dense", desc)

    def project(self, w: Matrix, w_norm: Tensor | None, bias: int = 0, **kw) -> int:
        """Normed stream -> ws.proj; returns the row stride.  kw: further fields of the descriptor."""
        ld = round_up(w.N, 8)
        desc = ffi.DenseDesc(self.model.dt, ffi.DENSE_STORE, w.N, w.K, 0, w.ld, ld, 0, 0.0, 0, 0, w.ptr, 0, 0, bias, 0, 0, self.ws.proj.ptr)
        for k, v in kw.items():
            setattr(desc, k, v)
        self.dense(desc, w_norm)
        return ld

    def output(self, w: "Matrix | Columns", x: int, ldx: int, w_add: Tensor, bias: int = 0, gated: ffi.GatedDesc | None = None, lead: int = 0) -> None:
        """The sublayer's last projection -> ws.y, to be normed with w_add and added to the stream.  `gated`: columns of x from
        `lead` on are still to be made from a linear recurrence's read-out."""
        m = self.model
        desc = ffi.DenseDesc(m.dt, ffi.DENSE_STORE, w.N, w.K, ldx, w.ld, m.width, 1, 0.0, 0, x, w.ptr, 0, 0, bias, 0, 0, self.ws.y.ptr)
        if gated is not None:
            desc.gated, desc.lead = gated, lead
        self.call("jg_dense", desc)
        self.pending = w_add

    def finish_layer(self) -> None:
        self.calls.append(None)  # a boundary for `HybridTransformer.layer_outputs`

    def run(self, batch: ffi.Batch) -> None:
        ref, h = C.byref(batch), self.model.dev.handle
        for c in self.calls:
            if c is not None:
                ffi.call(c[0], h, ref, *c[1:])


# ------------------------------------------------------------------------------------------------ mixers
class MinGRU:
    def __init__(self, m: "HybridTransformer", cfg: dict, name: str, params: dict):
        W = self.width = int(cfg["width"])
        self.w = Matrix(m, params, [(name + "z", W), (name + "x", W), (name + "g", W)], m.width)
        self.gate_ptrs = [self.w.rows_ptr(name + n) for n in "zxg"]
        self.bias = vector(m, params, [(name + "z.b", (W,)), (name + "x.b", (W,))], pad=W)  # the output gate has none
        self.o = Matrix(m, params, [(name + "o", m.width)], W)
        self.state = m.states.per_slot((W,), "float32")
        self.proj_ld, self.act_ld, self.scratch = round_up(3 * W, 8), round_up(W, 8), lambda B, Sc: 0

    def plan(self, p: Plan, w_norm: Tensor, w_add: Tensor) -> None:
        m, ws, W = p.model, p.ws, self.width
        if p.fused and p.single:
            b = self.bias.ptr
            p.dense(ffi.DenseDesc(m.dt, ffi.DENSE_MINGRU, W, m.width, 0, self.w.ld, self.act_ld, 0, 0.0, 0, 0, *self.gate_ptrs, b, b + 4 * W, 0,
                                  ws.act.ptr, 0, self.state.ptr), w_norm)
        else:
            ld = p.project(self.w, w_norm, self.bias.ptr)
            p.call("jg_mingru_scan", ffi.MinGruDesc(m.dt, W, ld, self.act_ld, ws.proj.ptr, self.state.ptr, ws.act.ptr))
        p.output(self.o, ws.act.ptr, self.act_ld, w_add)


class GatedDelta:
    def __init__(self, m: "HybridTransformer", cfg: dict, name: str, params: dict):
        H, G, d, v, taps = (int(cfg[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
        self.sizes = (H, G, d, v, taps)
        qkv = [(name + "q", G * d), (name + "k", G * d), (name + "v", H * v)]
        self.w = Matrix(m, params, qkv + [(name + "b", H), (name + "a", H), (name + "g", H * v)], m.width)
        self.conv = vector(m, params, [(n + ".conv", (c, taps)) for n, c in qkv])
        self.a_log, self.dt_bias = vector(m, params, [(name + "A_log", (H,))]), vector(m, params, [(name + "dt_bias", (H,))])
        self.norm = vector(m, params, [(name + "norm", (v,))])
        self.o = Matrix(m, params, [(name + "o", m.width)], H * v)
        self.state = m.states.per_slot((H, v, round_up(d, 4)), "float32")
        self.tail = m.states.per_slot((taps, 2 * G * d + H * v), m.dtype)
        self.proj_ld, self.act_ld = round_up(self.w.N, 8), round_up(H * v, 8)

    def desc(self, m: "HybridTransformer") -> ffi.DeltaDesc:
        return ffi.DeltaDesc(m.dt, *self.sizes, self.proj_ld, self.act_ld, m.eps, 0, 0, self.conv.ptr, self.a_log.ptr, self.dt_bias.ptr,
                             self.norm.ptr, self.state.ptr, self.tail.ptr)

    def scratch(self, B: int, Sc: int) -> int:
        H, G, d, v, taps = self.sizes
        n = C.c_uint64(0)
        ffi.call("jg_delta_scratch_floats", C.byref(ffi.DeltaDesc(0, H, G, d, v, taps)), B * Sc, C.byref(n))
        return 4 * n.value

    def plan(self, p: Plan, w_norm: Tensor, w_add: Tensor) -> None:
        p.project(self.w, w_norm)
        d = self.desc(p.model)
        d.proj, d.scratch, d.out = p.ws.proj.ptr, p.ws.scratch.ptr, p.ws.act.ptr
        p.call("jg_delta_rule", d)
        p.output(self.o, p.ws.act.ptr, self.act_ld, w_add)


def yarn_table(dims: int, base: float, scaling: dict | None, positions: int) -> np.ndarray:
    """fp32 [positions][dims / 2][2]: cos and sin of position * frequency, both times YaRN's attention factor.  The
    frequencies base^(-2i / dims) are divided by `factor` where their wavelength exceeds the original context, left alone where
    it is short, and blended linearly in between (`slow` and `fast` are rotations over the original context)."""
    i = np.arange(dims // 2, dtype=np.float64)
    f = float(base) ** (-2.0 * i / dims)
    gain = 1.0
    if scaling:
        def pair_of(turns: float) -> float:  # the pair that turns that often over the original context
            return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

        lo, hi = max(math.floor(pair_of(scaling["fast"])), 0), min(math.ceil(pair_of(scaling["slow"])), dims - 1)
        blend = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        f = f / scaling["factor"] * blend + f * (1.0 - blend)
        gain = 0.1 * math.log(scaling["factor"]) + 1.0
    a = np.arange(positions, dtype=np.float64)[:, None] * f
    return (np.stack([np.cos(a), np.sin(a)], axis=-1) * gain).astype(np.float32)


class LatentAttention:
    def __init__(self, m: "HybridTransformer", cfg: dict, name: str, params: dict):
        H, d, rd, v, rank = (int(cfg[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        self.H, self.dim, self.rd, self.vd, self.rank = H, d, rd, v, rank
        self.scale = float(cfg["scale"])
        self.window = int((cfg.get("mask") or {}).get("size") or 0)
        rot = cfg["rot"]
        self.pairs = int(rot["dims"]) // 2
        if 2 * self.pairs > rd:
            raise ValueError(f"rotary over {rot['dims']} of {rd} dimensions")
        self.rot = m.shared_table(("yarn", rot["dims"], rot["base"], tuple(sorted((rot.get("scaling") or {}).items()))),
                                  lambda: yarn_table(int(rot["dims"]), float(rot["base"]), rot.get("scaling"), m.max_context))
        self.w = Matrix(m, params, [(name + "q", H * (d + rd)), (name + "dkv", rank + rd)], m.width)
        self.norm = vector(m, params, [(name + "dkv.norm", (rank,))])
        self.ukv = Matrix(m, params, [(name + "uk", H * d), (name + "uv", H * v)], rank)
        self.sink = vector(m, params, [(name + "sink", (H,))])
        self.o = Matrix(m, params, [(name + "o", m.width)], H * v)
        self.ring = m.states.ring(round_up(rank + rd, 8), m.dtype, self.window)
        self.eps, self.max_context, self.dt = m.eps, m.max_context, m.dt
        self.proj_ld, self.act_ld = round_up(self.w.N, 8), round_up(H * v, 8)

    def desc(self) -> ffi.LatentDesc:
        r = self.ring
        return ffi.LatentDesc(self.dt, self.H, self.dim, self.rd, self.vd, self.rank, self.window, self.proj_ld, self.act_ld, r.row, self.ukv.ld,
                              r.page, r.pages_per_slot, r.table.shape[0], self.pairs, self.max_context, self.eps, self.scale, 0, r.pool.ptr,
                              r.table.ptr, self.rot.ptr, self.norm.ptr, self.sink.ptr, self.ukv.ptr)

    def scratch(self, B: int, Sc: int) -> int:
        n = C.c_uint64(0)
        ffi.call("jg_latent_scratch_bytes", C.byref(self.desc()), B, Sc, C.byref(n))
        return n.value

    def plan(self, p: Plan, w_norm: Tensor, w_add: Tensor) -> None:
        p.project(self.w, w_norm)
        d = self.desc()
        d.proj, d.scratch, d.scratch_bytes, d.out = p.ws.proj.ptr, p.ws.scratch.ptr, p.ws.scratch.nbytes, p.ws.act.ptr
        p.call("jg_latent_attn", d)
        p.output(self.o, p.ws.act.ptr, self.act_ld, w_add)


# ------------------------------------------------------------------------------------------------ branches
class WindowBranch:
    """Grouped-head attention over a sliding window and the first tokens; query and key norms over the whole projection."""

    def __init__(self, m: "HybridTransformer", cfg: dict, name: str):
        self.name, self.H, self.G, self.dim, self.vd = name, *(int(cfg[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        if self.H % self.G:
            raise ValueError(f"{self.H} heads do not divide among {self.G} key / value heads")
        mask, rot = cfg.get("mask") or {}, cfg["rot"]
        self.window, self.keep, self.scale = int(mask.get("size") or 0), int(mask.get("keep_first") or 0), float(cfg["scale"])
        self.pairs = int(rot["dims"]) // 2
        if 2 * self.pairs > self.dim:
            raise ValueError(f"rotary over {rot['dims']} of {self.dim} dimensions")
        self.rot = m.shared_table(("yarn", rot["dims"], rot["base"], ()), lambda: yarn_table(int(rot["dims"]), float(rot["base"]), None, m.max_context))
        self.ring = m.states.ring(self.G * (round_up(self.dim, 8) + round_up(self.vd, 8)), m.dtype, self.window, self.keep)
        self.eps, self.dt, self.max_context = m.eps, m.dt, m.max_context
        self.sizes = [("q", self.H * self.dim), ("k", self.G * self.dim), ("v", self.G * self.vd)]
        self.parts, self.width, self.fp32, self.silu = [(name + n, r, 8) for n, r in self.sizes], self.H * self.vd, 0, None

    def bind(self, m: "HybridTransformer", params: dict, w: Matrix) -> list[tuple[str, str, int]]:
        self.col = [w.row0[self.name + n] for n in "qkv"]
        self.qn, self.kn = (vector(m, params, [(self.name + n + ".norm", (r,))]) for n, r in self.sizes[:2])
        return [(self.name + n + ".b", self.name + n, r) for n, r in self.sizes]

    def desc(self) -> ffi.WindowDesc:
        r = self.ring
        return ffi.WindowDesc(self.dt, self.H, self.G, self.dim, self.vd, self.window, self.keep, 0, 0, r.page, r.pages_per_slot, r.pinned, self.pairs,
                              self.max_context, self.eps, self.scale, 1.0, 0, 0, 0, 0, self.qn.ptr, self.kn.ptr, self.rot.ptr, r.pool.ptr, r.table.ptr)

    def scratch(self, B: int, Sc: int) -> int:
        n = C.c_uint64(0)
        ffi.call("jg_window_scratch_bytes", C.byref(self.desc()), B, Sc, C.byref(n))
        return n.value

    def plan(self, p: Plan, proj, ld: int, scratch: int, nbytes: int, out: int, ldo: int, scale: float) -> None:
        d = self.desc()
        d.q, d.k, d.v = (proj(c) for c in self.col)
        d.ldp, d.ldo, d.out, d.out_scale, d.scratch, d.scratch_bytes = ld, ldo, out, scale, scratch, nbytes
        p.call("jg_window_attn", d)


class LinearBranch:
    """A linear recurrence with a matrix state per head, its norm and output gate.  `gated`: mLSTM (gates i and f, a norm per head);
    else a constant decay per head, silu on queries, keys and values, one norm over all heads."""

    def __init__(self, m: "HybridTransformer", cfg: dict, name: str, gated: bool):
        self.H, self.dim, self.vd = H, d, v = tuple(int(cfg[k]) for k in ("heads", "dim", "vdim"))
        self.name, self.gated, self.eps, self.dt = name, gated, m.eps, m.dt
        self.q_scale, self.cap = (d ** -0.5, float(cfg["gate_cap"])) if gated else (1.0, 0.0)
        self.state = m.states.per_slot((H, v + int(gated), round_up(d, 4)), "float32")
        self.m = m.states.per_slot((2, H), "float32") if gated else None
        self.decay = None
        if not gated:
            if len(cfg["decay"]) != H:
                raise ValueError(f"{len(cfg['decay'])} decays for {H} heads")
            self.decay = Tensor(np.asarray(cfg["decay"], np.float32), device=m.dev)
        self.parts = [(name + "q", H * d, 8), (name + "k", H * d, 8), (name + "v", H * v, 8), (name + "g", H * v, 8)]
        if gated:
            self.parts += [(name + "i", H, 8), (name + "f", H)]
        self.width, self.fp32, self.silu = H * v, 2 * H if gated else 0, None if gated else (name + "q", name + "g")

    def bind(self, m: "HybridTransformer", params: dict, w: Matrix) -> list[tuple[str, str, int]]:
        self.col = [w.row0[self.name + n] for n in "qkvg"]
        self.norm = vector(m, params, [(self.name + "norm", (self.width,))])
        return [(self.name + n + ".b", self.name + n, self.H) for n in "if"] if self.gated else []

    def _layout(self, rows: int) -> tuple[int, int, int]:
        """Where the divisors and the tokens' weights begin behind the read-outs, and the end."""
        n = C.c_uint64(0)
        ffi.call("jg_linear_scratch_bytes", C.byref(ffi.LinearDesc(self.dt, self.H, self.dim, self.vd)), rows, C.byref(n))
        den = round_up(4 * rows * self.width, 256)
        tok = den + round_up(4 * rows * self.H, 256)
        return den, tok, tok + n.value

    def scratch(self, B: int, Sc: int) -> int:
        return self._layout(B * Sc)[2]

    def plan(self, p: Plan, proj, ld: int, scratch: int, nbytes: int, out: int, ldo: int, scale: float) -> ffi.GatedDesc:
        den, tok, _ = self._layout(p.ws.cap)
        q, k, v, g = (proj(c) for c in self.col)
        d = ffi.LinearDesc(self.dt, self.H, self.dim, self.vd, ld, 0, self.q_scale, self.cap, q, k, v, 0, 0, self.state.ptr, 0, scratch + tok, scratch, 0)
        if self.gated:
            d.gates, d.m, d.den = p.ws.aux.ptr, self.m.ptr, scratch + den
        else:
            d.decay = self.decay.ptr
        p.call("jg_linear_state", d)
        return ffi.GatedDesc(self.dt, self.H, self.vd, self.H if self.gated else 1, ld, 0, self.eps, scale, scratch, d.den, g, self.norm.ptr)


class Branches:
    """A mixer of one or more branches that read the same input: one projection for all of them, one output projection over
    their results side by side.  branches: (branch, factor on its result, name of its output matrix)."""

    def __init__(self, m: "HybridTransformer", branches: list[tuple], params: dict):
        self.branches = [b for b, _, _ in branches]
        self.scales = [f for _, f, _ in branches]
        last = self.branches[-1]
        if any(b.fp32 for b in self.branches[:-1]):
            raise ValueError("a branch with gates in 32 bits comes last")
        parts = [q for b in self.branches for q in b.parts]
        self.w = Matrix(m, params, parts, m.width)
        bias = [q for b in self.branches for q in b.bind(m, params, self.w)]
        self.bias = row_vector(m, params, self.w, bias) if bias else None
        self.o = Columns(m, params, [(name, b.width) for b, _, name in branches], m.width)
        self.at = [self.o.col0[name] for _, _, name in branches]
        self.aux_ld, self.split = last.fp32, self.w.N - last.fp32 if last.fp32 else 0
        silu = [b.silu for b in self.branches if b.silu]
        if len(silu) > 1:
            raise ValueError("one branch of a mixer may have silu in its projection")
        self.silu = tuple(self.w.row0[n] for n in silu[0]) if silu else None
        self.proj_ld, self.act_ld = round_up(self.w.N, 8), round_up(self.o.K, 8)

    def _scratch(self, B: int, Sc: int) -> list[int]:
        return [round_up(b.scratch(B, Sc), 256) for b in self.branches]

    def scratch(self, B: int, Sc: int) -> int:
        return sum(self._scratch(B, Sc))

    def plan(self, p: Plan, w_norm: Tensor | None, w_add: Tensor) -> None:
        m, ws = p.model, p.ws
        size = ws.act.nbytes // ws.act.numel()
        kw = {}
        if self.silu:
            kw.update(act=ffi.ACT_SILU, act_lo=self.silu[0], act_hi=self.silu[1])
        if self.split:
            kw.update(split=self.split, y2=ws.aux.ptr, ld2=self.aux_ld)
        ld = p.project(self.w, w_norm, self.bias.ptr if self.bias is not None else 0, **kw)
        scratch, gated = ws.scratch.ptr, None
        for i, (b, f, at, n) in enumerate(zip(self.branches, self.scales, self.at, self._scratch(ws.B, max(1, ws.cap // ws.B)))):
            out = ws.act.ptr + at * size
            gated = b.plan(p, lambda c: ws.proj.ptr + c * size, ld, scratch, n, out, self.act_ld, f)
            scratch += n
            if gated is not None and not (p.fused and i == len(self.branches) - 1):
                p.call("jg_gated_norm", gated, out, self.act_ld)
                gated = None
        p.output(self.o, ws.act.ptr, self.act_ld, w_add, gated=gated, lead=self.at[-1])


def window_attention(m: "HybridTransformer", cfg: dict, name: str, params: dict) -> Branches:
    return Branches(m, [(WindowBranch(m, cfg, name), 1.0, name + "o")], params)


def lightning(m: "HybridTransformer", cfg: dict, name: str, params: dict) -> Branches:
    return Branches(m, [(LinearBranch(m, cfg, name, False), 1.0, name + "o")], params)


def mlstm(m: "HybridTransformer", cfg: dict, name: str, params: dict) -> Branches:
    return Branches(m, [(LinearBranch(m, cfg, name, True), 1.0, name + "o")], params)


def parallel(m: "HybridTransformer", cfg: dict, name: str, params: dict) -> Branches:
    return Branches(m, [(WindowBranch(m, cfg["left"], name + "left."), float(cfg["left_scale"]), name + "left.o"),
                        (LinearBranch(m, cfg["right"], name + "right.", False), float(cfg["right_scale"]), name + "right.o")], params)


# ------------------------------------------------------------------------------------------------ feed-forwards
class DenseGLU:
    def __init__(self, m: "HybridTransformer", cfg: dict, name: str, params: dict):
        f = int(cfg["ff"])
        self.limit = float(cfg["limit"])
        self.gate, self.up = Matrix(m, params, [(name + "gate", f)], m.width), Matrix(m, params, [(name + "up", f)], m.width)
        self.down = Matrix(m, params, [(name + "down", m.width)], f)
        self.gate_b, self.up_b = vector(m, params, [(name + "gate.b", (f,))]), vector(m, params, [(name + "up.b", (f,))])
        self.down_b = vector(m, params, [(name + "down.b", (m.width,))])
        self.ffn_ld = round_up(f, 8)

    def plan(self, p: Plan, w_norm: Tensor, w_add: Tensor) -> None:
        m, g = p.model, self.gate
        p.dense(ffi.DenseDesc(m.dt, ffi.DENSE_GLU, g.N, g.K, 0, g.ld, self.ffn_ld, 0, self.limit, 0, 0, g.ptr, self.up.ptr, 0, self.gate_b.ptr,
                              self.up_b.ptr, 0, p.ws.ffn.ptr), w_norm)
        p.output(self.down, p.ws.ffn.ptr, self.ffn_ld, w_add, self.down_b.ptr)


class SquaredReLU:
    """W_down max(W_up h, 0)^2."""

    def __init__(self, m: "HybridTransformer", cfg: dict, name: str, params: dict):
        f = int(cfg["ff"])
        self.up, self.down = Matrix(m, params, [(name + "up", f)], m.width), Matrix(m, params, [(name + "down", m.width)], f)
        self.ffn_ld = round_up(f, 8)

    def plan(self, p: Plan, w_norm: Tensor | None, w_add: Tensor) -> None:
        u = self.up
        d = ffi.DenseDesc(p.model.dt, ffi.DENSE_STORE, u.N, u.K, 0, u.ld, self.ffn_ld, 0, 0.0, 0, 0, u.ptr, 0, 0, 0, 0, 0, p.ws.ffn.ptr)
        d.act = ffi.ACT_RELU2
        p.dense(d, w_norm)
        p.output(self.down, p.ws.ffn.ptr, self.ffn_ld, w_add)


class TokenSide:
    """Per-layer token input: W_proj (gelu(W_gate x) * e), e the layer's part of the token's row in `table`."""

    def __init__(self, m: "HybridTransformer", table: Matrix, layer: int, dim: int, name: str, params: dict):
        self.table, self.at, self.vocab = table, layer * dim, m.vocab_size
        self.gate, self.proj = Matrix(m, params, [(name + "gate", dim)], m.width), Matrix(m, params, [(name + "proj", m.width)], dim)
        self.norm = vector(m, params, [(name + "norm", (m.width,))])
        self.ld = round_up(dim, 8)

    def plan(self, p: Plan) -> None:
        g, t, out = self.gate, self.table, p.ws.side.ptr
        d = ffi.DenseDesc(p.model.dt, ffi.DENSE_STORE, g.N, g.K, 0, g.ld, self.ld, 0, 0.0, 0, 0, g.ptr, 0, 0, 0, 0, 0, out)
        d.act, d.side, d.tokens, d.ld_side, d.col_side, d.vocab = ffi.ACT_GELU_SIDE, t.ptr, p.ws.tokens.ptr, t.ld, self.at, self.vocab
        p.dense(d, None)
        p.output(self.proj, out, self.ld, self.norm)


MIXERS = {"mingru": MinGRU, "latent_attention": LatentAttention, "delta": GatedDelta, "window_attention": window_attention, "lightning": lightning,
          "mlstm": mlstm, "parallel": parallel}


@dataclass(frozen=True)
class Design:
    """What an architecture fixes beyond the sizes and constants of its configuration."""
    norms: tuple = (("norm1", "norm1b"), ("norm2", "norm2b"))  # before (None: the sublayer reads the stream) and after mixer and feed-forward
    norm_offset: float = 0.0        # these norms' weights, and the final one's, are stored minus this
    tied_head: bool = False         # logits from the embedding table
    feed_forwards: tuple = (("dense", DenseGLU),)


DESIGNS = {"Matulorn": Design(),
           "Rigazen": Design(norms=((None, "norm1"), (None, "norm2")), norm_offset=1.0, tied_head=True, feed_forwards=(("dense", SquaredReLU),))}


class Layer:
    def __init__(self, m: "HybridTransformer", cfg: dict, index: int, params: dict):
        name, kinds = f"l{index}.", dict(m.design.feed_forwards)
        if cfg["type"] not in MIXERS:
            raise ValueError(f"unknown mixer {cfg['type']!r} (known: {', '.join(MIXERS)})")
        self.mixer = MIXERS[cfg["type"]](m, cfg["mixer"], name + "mix.", params)
        self.norm1 = self._norms(m, name, m.design.norms[0], params)
        self.mlp = self.side = None
        if cfg.get("mlp"):
            kind = cfg["mlp"].get("kind", "dense")
            if kind not in kinds:
                raise ValueError(f"unknown feed-forward {kind!r} (known: {', '.join(kinds)})")
            self.mlp = kinds[kind](m, cfg["mlp"], name + "mlp.", params)
            self.norm2 = self._norms(m, name, m.design.norms[1], params)
        if m.side is not None:
            self.side = TokenSide(m, m.side, index, m.side_dim, name + "side.", params)

    @staticmethod
    def _norms(m: "HybridTransformer", name: str, which: tuple, params: dict) -> list:
        return [vector(m, params, [(name + n, (m.width,))], offset=m.design.norm_offset) if n else None for n in which]

    def plan(self, p: Plan) -> None:
        self.mixer.plan(p, *self.norm1)
        if self.mlp is not None:
            self.mlp.plan(p, *self.norm2)
        if self.side is not None:
            self.side.plan(p)
        p.finish_layer()


# ------------------------------------------------------------------------------------------------ workspaces
class _Rows:
    """Activation buffers for up to `cap` rows of B sequences, and the plans that use them."""

    def __init__(self, m: "HybridTransformer", B: int, cap: int):
        dev, layers = m.dev, m.layers
        self.B, self.cap = B, cap
        self.tokens, self.next_tokens = Tensor.zeros((cap,), "int32", dev), Tensor.zeros((B,), "int32", dev)
        self.pos, self.seq = Tensor.zeros((B,), "int32", dev), Tensor.zeros((B,), "int32", dev)
        self.x = [Tensor.zeros((cap, m.width), "float32", dev) for _ in range(2 if cap <= 2 else 1)]
        self.y = Tensor.zeros((cap, m.width), "float32", dev)
        self.h = Tensor.zeros((cap, m.ld_width), m.dtype, dev)
        self.proj = Tensor.zeros((cap, max(l.mixer.proj_ld for l in layers)), m.dtype, dev)
        self.act = Tensor.zeros((cap, max(l.mixer.act_ld for l in layers)), m.dtype, dev)
        ffn = max((l.mlp.ffn_ld for l in layers if l.mlp is not None), default=0)
        self.ffn = Tensor.zeros((cap, ffn * (2 if m.dtype == "float32" else 1)), m.dtype, dev) if ffn else None
        aux = max(getattr(l.mixer, "aux_ld", 0) for l in layers)  # columns of the projection kept in 32 bits
        self.aux = Tensor.zeros((cap, aux), "float32", dev) if aux else None
        self.side = Tensor.zeros((cap, layers[0].side.ld), m.dtype, dev) if m.side is not None else None
        Sc = max(1, cap // B)
        self.scratch = Tensor.empty((max(max(l.mixer.scratch(B, s) for l in layers for s in {1, Sc}), 16),), "uint8", dev)
        self.batch = ffi.Batch(B, 1, self.pos.ptr, self.seq.ptr, -1, 0)
        self.plans: dict[tuple, Plan] = {}
        self.heads: dict[tuple, tuple] = {}
        self.logits = None


class _Step(_Rows):
    """A decode step's workspace: one row per sequence, logits and picks of each, page-locked staging (cf. call_host)."""

    def __init__(self, m: "HybridTransformer", B: int):
        super().__init__(m, B, B)
        self.logits = Tensor.zeros((B, m.vocab_size), "float32", m.dev)
        self.key = Tensor.zeros((B,), "uint64", m.dev)
        self._dev, self._pinned = m.dev, C.c_void_p()
        ffi.call("jg_host_alloc", 3 * 4 * B, C.byref(self._pinned))
        arr = np.ctypeslib.as_array((C.c_int32 * (3 * B)).from_address(self._pinned.value))
        self.h_tokens, self.h_pos, self.h_next = arr[:B], arr[B:2 * B], arr[2 * B:]

    def __del__(self):
        try:
            if self._pinned and self._dev.handle is not None:
                ffi.call("jg_host_free", self._pinned)
        except Exception:
            pass


class HybridTransformer(Decoder):
    """A decoder over `config` (`width`, `vocab`, `norm`, `layers`; optional: `embedding.scale`, `token_side.dim`) under the
    conventions of its `architecture` (DESIGNS).  dtype: 'bfloat16' or 'float32'."""

    def __init__(self, config: dict, dtype: str = "bfloat16", max_context: int = 8192, max_batch: int = 1, jit: bool = True, device=None,
                 page_size: int = 64, max_rows: int = 2048):
        if dtype not in DTYPES:
            raise ValueError(f"dtype {dtype!r}: expected one of {', '.join(DTYPES)}")
        dev = _dev(device)
        self.dev, self.dtype, self.dt = dev, dtype, DTYPES[dtype]
        self.width, self.vocab_size = int(config["width"]), int(config["vocab"])
        name = config.get("architecture", "Matulorn")
        if name not in DESIGNS:
            raise ValueError(f"unknown architecture {name!r} (known: {', '.join(DESIGNS)})")
        self.design = DESIGNS[name]
        self.groups, self.eps = int(config["norm"].get("groups", 1)), float(config["norm"]["eps"])
        if self.width % self.groups:
            raise ValueError(f"width {self.width} does not divide into {self.groups} norm groups")
        self.ld_width = round_up(self.width, 8)
        self.max_context, self.max_batch, self.max_rows = max_context, max_batch, max(1, min(max_rows, max_context * max_batch))
        self.states = SlotStates(dev, max_batch, max_context, self.max_rows, page_size)
        self._tables: dict = {}
        self.params: dict[str, Param] = {}
        self.embed = Matrix(self, self.params, [("embed", self.vocab_size)], self.width)
        self.embed_scale = float((config.get("embedding") or {}).get("scale", 1.0))
        self.side, self.side_dim = None, int((config.get("token_side") or {}).get("dim", 0))
        if self.side_dim:
            self.side = Matrix(self, self.params, [("side.embed", self.vocab_size)], self.side_dim * len(config["layers"]))
        self.layers = [Layer(self, c, i, self.params) for i, c in enumerate(config["layers"])]
        self.norm = vector(self, self.params, [("final.norm", (self.width,))], offset=self.design.norm_offset)
        self.head = self.embed if self.design.tied_head else Matrix(self, self.params, [("head", self.vocab_size)], self.width)
        self._steps: dict[int, _Step] = {}
        self._chunks: dict[tuple[int, int], _Rows] = {}
        self._row_slots: list[int] = []
        self._slot_jit: TinyJit | None = None
        self._slot_ws: _Step | None = None
        self._out: dict[int, tuple[Tensor, Tensor, Tensor]] = {}
        self._init_decoder(dev, jit)

    def shared_table(self, key, make) -> Tensor:
        if key not in self._tables:
            self._tables[key] = Tensor(make(), device=self.dev)
        return self._tables[key]

    def load_state_dict(self, weights: dict[str, np.ndarray]) -> "HybridTransformer":
        """Copy host arrays (exact values of the checkpoint) into the model by name: every tensor, and no other."""
        missing, extra = sorted(set(self.params) - set(weights)), sorted(set(weights) - set(self.params))
        if missing or extra:
            raise KeyError(f"checkpoint does not fit the configuration: missing {missing[:4]}, unexpected {extra[:4]}")
        for name, p in self.params.items():
            if tuple(weights[name].shape) != p.shape:
                raise ValueError(f"Shape mismatch in {name}: Expected shape {p.shape}, but found {tuple(weights[name].shape)} in the checkpoint.")
            p.assign(weights[name])
        return self

    # ------------------------------------------------------------------------------------------ workspaces and plans
    def _workspace(self, B: int) -> _Step:
        if B > self.max_batch:
            raise ValueError(f"batch {B} exceeds max_batch {self.max_batch}")
        if B not in self._steps:
            self._steps[B] = _Step(self, B)
            self._steps[B].seq.assign(self._rows_of(B))
        return self._steps[B]

    def _rows_of(self, B: int) -> np.ndarray:
        """Slots of batch rows 0 .. B - 1: taken on first use and kept."""
        while len(self._row_slots) < B:
            self._row_slots.append(self.states.acquire())
        return np.array(self._row_slots[:B], np.int32)

    def _chunk(self, B: int, rows: int) -> _Rows:
        cap = 1
        while cap < rows:
            cap *= 2
        cap = min(max(cap, B), max(self.max_rows, B))
        cap = max(cap, rows)
        if (B, cap) not in self._chunks:
            self._chunks[(B, cap)] = _Rows(self, B, cap)
        return self._chunks[(B, cap)]

    def _plan(self, ws: _Rows, R: int, single: bool) -> Plan:
        fused = R <= 2
        key = (fused, single and fused)
        if key not in ws.plans:
            p = Plan(self, ws, *key)
            if fused and len(ws.x) < 2:
                ws.x.append(Tensor.zeros(ws.x[0].shape, "float32", self.dev))
            p.call("jg_stream_embed", ws.x[0].ptr, ws.tokens.ptr, self.embed.ptr, self.dt, self.width, self.embed.ld, self.vocab_size, self.embed_scale)
            for layer in self.layers:
                layer.plan(p)
            ws.plans[key] = p
        return ws.plans[key]

    def _run_layers(self, ws: _Rows, B: int, Sc: int, start: int = -1) -> Plan:
        """`start`: the position the rows begin at, or -1 when only the device knows it (a step that is captured)."""
        ws.batch.B, ws.batch.Sc, ws.batch.start = B, Sc, start
        p = self._plan(ws, B * Sc, Sc == 1)
        p.run(ws.batch)
        return p

    def _run_head(self, p: Plan, n: int, rows: int, logits: Tensor, key: Tensor, picks: int) -> None:
        """Final norm, logits and greedy picks of n rows of the stream: the first n, or those `rows` (device int32) names."""
        ws, w = p.ws, self.head
        hk = (n, rows, id(p))
        if hk not in ws.heads:
            st = p.stream(self.norm, rows, keep=False)
            d = ffi.DenseDesc(self.dt, ffi.DENSE_LOGITS, w.N, w.K, 0, w.ld, self.vocab_size, 1, 0.0, 0, 0, w.ptr, 0, 0, 0, 0, 0, logits.ptr, key.ptr)
            if n <= 2:
                d.stream = st
            else:
                d.ldx = self.ld_width
            ws.heads[hk] = (st, d, ffi.Batch(n, 1, ws.pos.ptr, ws.seq.ptr, -1, 0))
        st, d, batch = ws.heads[hk]
        d.y, d.key = logits.ptr, key.ptr
        if n > 2:
            h = self._head_rows(ws, n)
            d.x = h
            self.dev.call("jg_stream_norm", C.byref(batch), st, h, self.ld_width, self.dt)
        self.dev.call("jg_dense", C.byref(batch), d)
        self.dev.call("jg_argmax_finalize", picks, key.ptr, n)

    def _head_rows(self, ws: _Rows, n: int) -> int:
        if n <= ws.cap:
            return ws.h.ptr
        raise ValueError(f"{n} output rows from {ws.cap} rows")

    def _step(self, ws: _Step, advance: bool = False) -> None:
        """One token per row: reads ws.tokens / ws.pos / ws.seq, writes ws.logits and ws.next_tokens."""
        p = self._run_layers(ws, ws.B, 1)
        self._run_head(p, ws.B, 0, ws.logits, ws.key, ws.next_tokens.ptr)
        if advance:
            self.dev.call("jg_copy", ws.tokens.ptr, ws.next_tokens.ptr, 4 * ws.B)
            self.dev.call("jg_pos_advance", ws.pos.ptr, ws.B)

    # ------------------------------------------------------------------------------------------ decoder hooks
    def _advance(self, B: int, start_pos: int, n: int) -> None:
        for s in self._rows_of(B):
            self.states.advance(int(s), start_pos, n)

    def reusable_prefix(self, n: int) -> int:
        """State cannot be wound back: what was fed last is reusable only when it is exactly those n tokens."""
        return n if n and self._row_slots and self.states.length[self._row_slots[0]] == n else 0

    def _feed_rows(self, toks: np.ndarray, start_pos: int, slots: np.ndarray, want: np.ndarray | None) -> list[np.ndarray]:
        """Tokens [B, S] from start_pos on, in passes of up to max_rows rows.  `want` (B = 1): places whose logits are copied
        out, a list of [n, vocab] per pass.  Without it the rows of the last position leave logits and picks in the batch's
        step workspace."""
        B, S = toks.shape
        per = max(1, self.max_rows // B)
        got = []
        for s0 in range(0, S, per):
            part = toks[:, s0:s0 + per]
            Sc = part.shape[1]
            ws = self._chunk(B, B * Sc)
            buf = np.zeros((ws.cap,), np.int32)
            buf[:B * Sc] = part.T.reshape(-1)
            ws.tokens.assign(buf)
            ws.pos.assign(np.full((B,), start_pos + s0, np.int32))
            ws.seq.assign(slots)
            p = self._run_layers(ws, B, Sc, start_pos + s0)
            if want is None:
                if s0 + Sc >= S:
                    wsb = self._workspace(B)
                    rows = self._row_list(ws, np.arange((Sc - 1) * B, Sc * B))
                    self._run_head(p, B, rows, wsb.logits, wsb.key, wsb.next_tokens.ptr)
                continue
            places = want[(want >= s0) & (want < s0 + Sc)] - s0
            if len(places):
                n = len(places)
                logits, key, picks = self._outputs(n)
                self._run_head(p, n, self._row_list(ws, places), logits, key, picks.ptr)
                got.append(logits.numpy()[:n])
        return got

    def _row_list(self, ws: _Rows, rows: np.ndarray) -> int:
        if getattr(ws, "rows", None) is None:
            ws.rows = Tensor.zeros((ws.cap,), "int32", self.dev)
        buf = np.zeros((ws.cap,), np.int32)
        buf[:len(rows)] = rows
        ws.rows.assign(buf)
        return ws.rows.ptr

    def _outputs(self, n: int) -> tuple[Tensor, Tensor, Tensor]:
        cap = 1
        while cap < n:
            cap *= 2
        if cap not in self._out:
            self._out[cap] = (Tensor.zeros((cap, self.vocab_size), "float32", self.dev), Tensor.zeros((cap,), "uint64", self.dev),
                              Tensor.zeros((cap,), "int32", self.dev))
        return self._out[cap]

    def forward(self, tokens, start_pos: int, temperature: float = 0.0, top_k: int = 0, top_p: float = 0.8,
                alpha_f: float = 0.0, alpha_p: float = 0.0) -> Tensor:
        """Tokens int32 [B, S] at positions start_pos ..; the pick after the last one, int32 [B]."""
        toks = tokens.numpy() if isinstance(tokens, Tensor) else np.asarray(tokens, dtype=np.int32)
        B, S = toks.shape
        ws = self._workspace(B)
        self._advance(B, start_pos, S)
        self._feed_rows(toks, start_pos, self._rows_of(B), None)
        return self._pick(ws, temperature, top_k, top_p, alpha_f, alpha_p)

    # ------------------------------------------------------------------------------------------ requests with slots of their own
    def acquire_slot(self) -> int:
        return self.states.acquire()

    def release_slot(self, slot: int) -> None:
        self.states.release(slot)

    def feed(self, slot: int, tokens, start_pos: int, want=()) -> np.ndarray:
        toks = np.asarray(tokens, np.int32).reshape(1, -1)
        want = np.asarray(list(want), np.int64)
        S = toks.shape[1]
        if S == 0:
            return np.zeros((0, self.vocab_size), np.float32)
        if len(want) and (want.min() < 0 or want.max() >= S):
            raise ValueError(f"wanted places {want.tolist()} outside a portion of {S} tokens")
        self.states.advance(slot, start_pos, S)
        if S == 1 and self._jit_enabled:  # the captured decode step
            if self._slot_ws is None:
                self._slot_ws = _Step(self, 1)
                self._slot_jit = TinyJit(lambda: self._step(self._slot_ws), self.dev)
            ws = self._slot_ws
            ws.tokens.assign(toks[0])
            ws.pos.assign(np.array([start_pos], np.int32))
            ws.seq.assign(np.array([slot], np.int32))
            self._slot_jit.call()
            return np.repeat(ws.logits.numpy(), len(want), axis=0)
        uniq, back = np.unique(want, return_inverse=True)
        got = self._feed_rows(toks, start_pos, np.array([slot], np.int32), uniq)
        return np.concatenate(got)[back] if got else np.zeros((0, self.vocab_size), np.float32)

    def layer_outputs(self, slot: int, tokens, start_pos: int = 0) -> np.ndarray:
        """The residual stream after every layer, fp32 [layers, S, width] (inspection: one portion, up to max_rows tokens)."""
        toks = np.asarray(tokens, np.int32).reshape(-1)
        S = len(toks)
        self.states.advance(slot, start_pos, S)
        ws = self._chunk(1, S)
        buf = np.zeros((ws.cap,), np.int32)
        buf[:S] = toks
        ws.tokens.assign(buf)
        ws.pos.assign(np.array([start_pos], np.int32))
        ws.seq.assign(np.array([slot], np.int32))
        ws.batch.B, ws.batch.Sc, ws.batch.start = 1, S, start_pos
        out, peek = [], Plan(self, ws, S <= 2, S == 1)
        if S <= 2 and len(ws.x) < 2:
            ws.x.append(Tensor.zeros(ws.x[0].shape, "float32", self.dev))
        peek.call("jg_stream_embed", ws.x[0].ptr, ws.tokens.ptr, self.embed.ptr, self.dt, self.width, self.embed.ld, self.vocab_size, self.embed_scale)
        res = Tensor.zeros((ws.cap, self.width), "float32", self.dev)
        for layer in self.layers:
            layer.plan(peek)
            st = peek.stream(None, keep=False)
            st.x_out = res.ptr
            peek.call("jg_stream_norm", st, 0, self.ld_width, self.dt)
            peek.run(ws.batch)
            peek.calls.clear()
            out.append(res.numpy()[:S])
        return np.stack(out)

    def last_logits(self, B: int) -> np.ndarray:
        return self._workspace(B).logits.numpy()
