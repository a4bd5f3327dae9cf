"""Rigazen on the device against the plain restatement in oracle/rigazen.py: each mechanism alone and all together, in 32 bits
(tight) and as served (bf16), whole prompts, portions, decoding, reused slots and pages, keys at every kind of edge, and the
drivers on top."""
import ctypes as C
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import rigazen as O
from tests.util import ROOT, write_safetensors_bf16

pytestmark = pytest.mark.gpu

F32_TOL, BF16_TOL = 2e-4, 0.06


def window(**kw):
    c = {"dim": 24, "heads": 6, "kv_heads": 2, "mask": {"keep_first": 5, "size": 17}, "rot": {"base": 2000.0, "dims": 16}, "scale": 0.2, "vdim": 20}
    c.update(kw)
    return c


def light(decay=(0.5, 0.9, 0.99), **kw):
    c = {"decay": list(decay), "dim": 20, "heads": len(decay), "vdim": 28}
    c.update(kw)
    return c


def parallel(left=None, right=None, left_scale=0.7, right_scale=1.3):
    return {"type": "parallel", "mixer": {"left": left or window(), "right": right or light(), "left_scale": left_scale, "right_scale": right_scale}, "mlp": None}


def mlstm(**kw):
    c = {"dim": 20, "gate_cap": 9.0, "heads": 3, "vdim": 28}
    c.update(kw)
    return {"type": "mlstm", "mixer": c, "mlp": None}


def with_mlp(layer, ff=72):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def config(*layers, width=48, vocab=97, eps=1e-5, scale=7.0, side=12):
    return {"architecture": "Rigazen", "embedding": {"scale": scale}, "layers": list(layers), "norm": {"eps": eps}, "token_side": {"dim": side}, "vocab": vocab,
            "width": width}


MIXED = config(with_mlp(parallel()), mlstm(), with_mlp(mlstm(dim=36, vdim=12, heads=2, gate_cap=15.0)),
               with_mlp(parallel(window(heads=4, kv_heads=1, dim=32, vdim=48, mask={"keep_first": 3, "size": 30}, rot={"base": 100.0, "dims": 32}),
                                 light((0.3, 0.8, 1.0, 0.95), dim=16, vdim=16)), ff=40),
               parallel(window(heads=2, kv_heads=2, dim=8, vdim=16, mask={"keep_first": 21, "size": 9}, rot={"base": 40.0, "dims": 4}), light((0.97,), dim=40, vdim=24)))


def build(cfg, params, dtype="float32", max_context=256, max_batch=3, **kw):
    from denograd_b200.hybrid import HybridTransformer
    return HybridTransformer(cfg, dtype, max_context, max_batch, **kw).load_state_dict(params)


def error(got, want):
    """Worst row: rms of the difference (mean taken off) over the rms of the expected logits."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return float(np.max(np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())))


def check(got, want, dtype="float32", what=None):
    """32 bits: every row.  bf16: all rows together, and no row far off."""
    worst = error(got, want)
    if dtype == "float32":
        assert worst < F32_TOL, (what, worst)
        return
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    total = float(np.sqrt((d * d).mean() / (w * w).mean()))
    assert total < BF16_TOL and worst < 6 * BF16_TOL, (what, total, worst)


def run(model, toks, cuts, slot=None):
    """Logits of every position, the tokens fed in portions of the given sizes (the last size repeats)."""
    own = slot is None
    slot = model.acquire_slot() if own else slot
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(model.feed(slot, toks[at:at + n], at, range(n)))
        at, i = at + n, i + 1
    if own:
        model.release_slot(slot)
    return np.concatenate(out)


def tokens(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


# ------------------------------------------------------------------------------------------------ each mechanism
SINGLE = {
    "mlstm": config(mlstm()),
    "mlstm, sizes on the tensor-core grid": config(mlstm(dim=64, vdim=64, heads=2), width=96),
    "mlstm, 96 x 40": config(mlstm(dim=96, vdim=40, heads=3), width=64),
    "mlstm, wide heads": config(mlstm(dim=200, vdim=136, heads=2, gate_cap=4.0), width=64),
    "mlstm, widest heads": config(mlstm(dim=300, vdim=33, heads=1), width=40),
    "mlstm, one small head": config(mlstm(dim=1, vdim=1, heads=1)),
    "mlstm, odd sizes": config(with_mlp(mlstm(dim=7, vdim=5, heads=5, gate_cap=2.5), ff=51), width=45, vocab=61, side=5),
    "parallel": config(parallel()),
    "parallel, sizes on the tensor-core grid": config(parallel(window(dim=32, vdim=64, heads=8, kv_heads=2, rot={"base": 5e4, "dims": 32}),
                                                               light((0.6, 0.9, 0.98, 0.999), dim=64, vdim=32)), width=128),
    "parallel, one head each, no window": config(parallel(window(heads=1, kv_heads=1, mask=None), light((0.9,)))),
    "parallel, window of one and no first tokens": config(parallel(window(mask={"keep_first": 0, "size": 1}))),
    "parallel, more first tokens than window": config(parallel(window(mask={"keep_first": 40, "size": 6}))),
    "parallel, first tokens without a key in keep_first": config(parallel(window(mask={"size": 12}))),
    "parallel, a few dimensions turn": config(parallel(window(rot={"base": 300.0, "dims": 4}))),
    "parallel, odd sizes": config(parallel(window(dim=7, vdim=9, heads=3, kv_heads=3, rot={"base": 50.0, "dims": 6}), light((0.8, 0.4), dim=5, vdim=3)), width=37, side=1),
    "parallel, wide heads": config(parallel(window(dim=136, vdim=200, heads=2, kv_heads=1, scale=0.09, rot={"base": 1e4, "dims": 64}), light((0.9, 0.99), dim=136, vdim=72)), width=64),
    "parallel, widest heads": config(parallel(window(dim=264, vdim=270, heads=2, kv_heads=1, scale=0.06, rot={"base": 1e4, "dims": 264}), light((0.9,), dim=260, vdim=40)), width=64),
    "parallel, many heads per key": config(parallel(window(dim=16, vdim=8, heads=36, kv_heads=2, rot={"base": 1e4, "dims": 16}))),
    "parallel, decay of one and faster than any": config(parallel(right=light((1.0, 1e-4)))),
}


@pytest.mark.parametrize("name", SINGLE)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_layer(name, dtype):
    cfg = SINGLE[name]
    params = O.random_params(cfg, seed=3)
    toks = tokens(cfg, 150)
    want = O.forward(params, cfg, toks)
    m = build(cfg, params, dtype)
    for cuts in ([150], [70, 1], [40, 5, 9, 15, 64, 3], [1, 16, 17, 100]):
        check(run(m, toks, cuts), want, dtype, cuts)


def test_the_branches_as_mixers_of_their_own():
    """Window attention, lightning attention and mLSTM under the other design's norms (before and after each sublayer)."""
    from oracle import matulorn as M
    cfg = {"architecture": "Matulorn", "width": 40, "vocab": 61, "norm": {"eps": 1e-5, "groups": 2}, "layers": [
        {"type": "window_attention", "mixer": window(), "mlp": None}, {"type": "lightning", "mixer": light(), "mlp": None}, mlstm()]}
    from denograd_b200.hybrid import HybridTransformer
    m = HybridTransformer(cfg, "float32", 128)
    rng = np.random.default_rng(0)
    params = {k: O.bf16_round(rng.standard_normal(p.shape) * (1 if len(p.shape) == 1 else 1.2 / math.sqrt(p.shape[-1]))) for k, p in m.params.items()}
    m.load_state_dict(params)
    toks = tokens(cfg, 60)
    x = np.asarray(params["embed"], np.float64)[toks]
    for i, (lc, f) in enumerate(zip(cfg["layers"], (O.window_attention, O.lightning, O.mlstm))):
        n = lambda v, s: M.group_norm(v, np.asarray(params[f"l{i}.{s}"], np.float64), 2, 1e-5)  # noqa: E731
        x = x + n(f(n(x, "norm1"), M.sub(params, f"l{i}.mix."), lc["mixer"], 1e-5), "norm1b")
    want = M.group_norm(x, np.asarray(params["final.norm"], np.float64), 2, 1e-5) @ np.asarray(params["head"], np.float64).T
    for cuts in ([60], [31, 1], [2]):
        check(run(m, toks, cuts), want)


def test_layer_outputs():
    params = O.random_params(MIXED, seed=4)
    toks, layers = tokens(MIXED, 29), []
    O.forward(params, MIXED, toks, layer_outputs=layers)
    for n in (29, 2, 1):
        m = build(MIXED, params)
        got = m.layer_outputs(m.acquire_slot(), toks[:n])
        for g, w in zip(got, layers):
            assert np.abs(g - w[:n]).max() < 1e-4 * np.abs(w).max()


# ------------------------------------------------------------------------------------------------ kernels
@pytest.mark.parametrize("M,N,K", [(1, 40, 48), (2, 33, 200), (3, 130, 72), (17, 96, 64), (300, 260, 136), (129, 16, 1024), (700, 200, 264)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("act", ["none", "silu", "relu2", "side"])
def test_projection_epilogues(dev, M, N, K, dtype, act):
    """Activations on a run of columns, the token table's factor, and the last columns in 32 bits elsewhere."""
    from denograd_b200 import ffi
    from denograd_b200.device import Tensor
    from denograd_b200.hybrid import DTYPES
    rng = np.random.default_rng(1)
    ld, ldy, vocab, at, split = (K + 7) // 8 * 8, (N + 7) // 8 * 8, 23, 5, N - 7
    x, w = np.zeros((M, ld), np.float32), np.zeros((N, ld), np.float32)
    x[:, :K], w[:, :K] = O.bf16_round(rng.standard_normal((M, K))), O.bf16_round(rng.standard_normal((N, K)) / np.sqrt(K))
    bias, table = rng.standard_normal(N).astype(np.float32), O.bf16_round(rng.standard_normal((vocab, N + 9)))
    toks = rng.integers(0, vocab, M).astype(np.int32)
    t = lambda a: Tensor.zeros(a.shape, dtype, dev).assign(a)  # noqa: E731
    tx, tw, tt, tb, tk = t(x), t(w), t(table), Tensor(bias, device=dev), Tensor(toks, device=dev)
    y, y2 = Tensor.zeros((M, ldy), dtype, dev), Tensor.zeros((M, 9), "float32", dev)
    d = ffi.DenseDesc(DTYPES[dtype], ffi.DENSE_STORE, N, K, ld, ld, ldy, 0, 0.0, 0, tx.ptr, tw.ptr, 0, 0, tb.ptr, 0, 0, y.ptr)
    v = x.astype(np.float64) @ w.T.astype(np.float64) + bias
    if act == "silu":
        d.act, d.act_lo, d.act_hi = ffi.ACT_SILU, 3, N - 11
        v[:, 3:N - 11] = O.silu(v[:, 3:N - 11])
    elif act == "relu2":
        d.act = ffi.ACT_RELU2
        v = np.maximum(v, 0) ** 2
    elif act == "side":
        d.act, d.side, d.tokens, d.ld_side, d.col_side, d.vocab = ffi.ACT_GELU_SIDE, tt.ptr, tk.ptr, N + 9, at, vocab
        v = O.gelu_tanh(v) * table[toks][:, at:at + N]
    d.split, d.ld2, d.y2 = split, 9, y2.ptr
    dev.call("jg_dense", C.byref(ffi.Batch(M, 1, 0, 0, -1, 0)), d)
    top = np.abs(v).max()
    assert np.abs(y.numpy()[:, :split] - v[:, :split]).max() < (3e-5 if dtype == "float32" else 5e-3) * top
    assert np.abs(y2.numpy()[:, :7] - v[:, split:]).max() < 3e-5 * top  # 32 bits whatever the element type
    assert (y.numpy()[:, split:N] == 0).all() and (y2.numpy()[:, 7:] == 0).all()


@pytest.mark.parametrize("H,vd,groups", [(3, 20, 3), (3, 20, 1), (1, 7, 1), (8, 512, 8), (16, 8, 16), (40, 12, 40)])
@pytest.mark.parametrize("R", [1, 2, 5])
@pytest.mark.parametrize("lead", [0, 24])
def test_gated_norm(dev, H, vd, groups, R, lead):
    """Division, group norm and output gate as a kernel and as the prologue of a projection, with columns ahead of them."""
    from denograd_b200 import ffi
    from denograd_b200.device import Tensor
    rng = np.random.default_rng(2)
    n, N = H * vd, 33
    o, den, gate, w = rng.standard_normal((R, n)), 0.1 + rng.random((R, H)), 3 * rng.standard_normal((R, n + 5)), 1 + rng.standard_normal(n)
    for with_den in (True, False):
        v = o / np.repeat(den, vd, axis=1) if with_den else o
        v = v.reshape(R, groups, -1)
        want = (v / np.sqrt((v * v).mean(-1, keepdims=True) + 1e-3)).reshape(R, n) * w * O.sigmoid(gate[:, :n]) * 0.7
        to, td, tg, tw = (Tensor(a.astype(np.float32), device=dev) for a in (o, den, gate, w))
        g = ffi.GatedDesc(ffi.JG_F32, H, vd, groups, n + 5, 0, 1e-3, 0.7, to.ptr, td.ptr if with_den else 0, tg.ptr, tw.ptr)
        ld = (lead + n + 7) // 8 * 8
        out = Tensor.zeros((R, ld), "float32", dev)
        b = ffi.Batch(R, 1, 0, 0, -1, 0)
        dev.call("jg_gated_norm", C.byref(b), g, out.ptr + 4 * lead, ld)
        assert np.abs(out.numpy()[:, lead:lead + n] - want).max() < 2e-5 * np.abs(want).max()
        x, mat = rng.standard_normal((R, ld)).astype(np.float32), np.zeros((N, ld), np.float32)
        mat[:, :lead + n] = rng.standard_normal((N, lead + n)) / np.sqrt(lead + n)
        if R <= 2:
            tx, tm, y = Tensor(x, device=dev), Tensor(mat, device=dev), Tensor.zeros((R, 40), "float32", dev)
            d = ffi.DenseDesc(ffi.JG_F32, ffi.DENSE_STORE, N, lead + n, ld, ld, 40, 1, 0.0, 0, tx.ptr if lead else 0, tm.ptr, 0, 0, 0, 0, 0, y.ptr)
            d.gated, d.lead = g, lead
            dev.call("jg_dense", C.byref(b), d)
            row = np.concatenate([x[:, :lead], want], 1)
            assert np.abs(y.numpy()[:, :N] - row @ mat[:, :lead + n].T).max() < 5e-5


def linear_state(dev, q, k, v, dtype, cuts, gates=None, cap=5.0, decay=None, slot=1):
    """jg_linear_state on one sequence in portions: read-outs and divisors."""
    from denograd_b200 import ffi
    from denograd_b200.device import Tensor
    from denograd_b200.hybrid import DTYPES
    (T, H, d), vd = q.shape, v.shape[-1]
    up = lambda n: (n + 7) // 8 * 8  # noqa: E731
    cq, cv, cg = up(H * d), up(H * vd), 0
    ld = 2 * cq + cv
    rows = np.zeros((T, ld), np.float32)
    rows[:, :H * d], rows[:, cq:cq + H * d], rows[:, 2 * cq:2 * cq + H * vd] = q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)
    cols, es = vd + (gates is not None), 4 if dtype == "float32" else 2
    st = Tensor(np.full((3, H, cols, (d + 3) // 4 * 4), 7.0, np.float32), device=dev), Tensor(np.full((3, 2, H), 9.0, np.float32), device=dev)
    dec = Tensor(np.asarray(decay if decay is not None else np.ones(H), np.float32), device=dev)
    seq, out, dens, at, i = Tensor(np.array([slot], np.int32), device=dev), [], [], 0, 0
    while at < T:
        n = min(cuts[min(i, len(cuts) - 1)], T - at)
        x = Tensor.zeros((n, ld), dtype, dev).assign(rows[at:at + n])
        g = Tensor(gates[at:at + n].astype(np.float32), device=dev) if gates is not None else None
        o, den, pos = Tensor.zeros((n, H * vd), "float32", dev), Tensor(np.ones((n, H), np.float32), device=dev), Tensor(np.array([at], np.int32), device=dev)
        scratch = Tensor.zeros((16 * n * H,), "uint8", dev)
        desc = ffi.LinearDesc(DTYPES[dtype], H, d, vd, ld, 0, 0.5, cap, x.ptr, x.ptr + es * cq, x.ptr + 2 * es * cq, g.ptr if g else 0, dec.ptr, st[0].ptr, st[1].ptr, scratch.ptr,
                              o.ptr, den.ptr)
        dev.call("jg_linear_state", C.byref(ffi.Batch(1, n, pos.ptr, seq.ptr, at, 0)), desc)
        out.append(o.numpy().reshape(n, H, vd))
        dens.append(den.numpy())
        at, i = at + n, i + 1
    return np.concatenate(out), np.concatenate(dens)


def plain_linear_state(q, k, v, gates=None, cap=5.0, decay=None):
    (T, H, d), vd = q.shape, v.shape[-1]
    S, n, m, out, den = np.zeros((H, d, vd)), np.zeros((H, d)), np.zeros(H), np.zeros((T, H, vd)), np.ones((T, H))
    for t in range(T):
        for a in range(H):
            keep, put = (1.0 if decay is None else decay[a]), 1.0
            if gates is not None:
                i, f = cap * np.tanh(gates[t, a] / cap), float(O.log_sigmoid(cap * np.tanh(gates[t, H + a] / cap)))
                new = max(f + m[a], i)
                keep, put, m[a] = math.exp(f + m[a] - new), math.exp(i - new), new
            S[a] = keep * S[a] + put * np.outer(k[t, a], v[t, a])
            n[a] = keep * n[a] + put * k[t, a]
            out[t, a] = S[a].T @ (0.5 * q[t, a])
            if gates is not None:
                den[t, a] = max(abs(n[a] @ (0.5 * q[t, a])), math.exp(-m[a])) + 1e-6
    return out, den


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,vd", [(2, 64, 64), (3, 24, 40), (2, 128, 96), (1, 256, 40), (2, 100, 7), (1, 5, 3), (1, 600, 9)])
@pytest.mark.parametrize("kind", ["decay", "gates", "strong gates"])
def test_linear_recurrence(dev, dtype, H, d, vd, kind):
    """A slot full of other numbers, portions within and across the blocks of 16, 64 and 256 tokens, an odd and an even number
    of tokens (the running maximum changes places), and gates far out on both sides."""
    rng = np.random.default_rng(d + vd)
    T = 300
    q, k, v = (O.bf16_round(rng.standard_normal((T, H, n))).astype(np.float64) for n in (d, d, vd))
    gates = None if kind == "decay" else rng.standard_normal((T, 2 * H)).astype(np.float32)
    if kind == "strong gates":  # long runs of forgetting and of keeping, inputs from almost nothing to a lot
        gates = (6 * gates + np.repeat(rng.choice([-9.0, 9.0], (T // 20, 2 * H)), 20, axis=0)).astype(np.float32)
    decay = np.linspace(0.3, 0.995, H) if kind == "decay" else None
    want, want_den = plain_linear_state(q, k, v, gates, decay=decay)
    size, tol = np.sqrt((want * want).mean(axis=(0, 2))), 2e-5 if dtype == "float32" else 1e-4  # the inputs are bf16 numbers in both
    for cuts in ([300], [64, 1, 16, 63, 65], [1], [2, 3, 17]):
        got, den = linear_state(dev, q, k, v, dtype, cuts, gates, decay=decay)
        off = np.abs(got - want).max(axis=2) / size
        assert off.max() < 10 * tol, (cuts, np.unravel_index(off.argmax(), off.shape), off.max())
        off = np.abs(den - want_den) / np.maximum(want_den, size)
        assert off.max() < 10 * tol, (cuts, np.unravel_index(off.argmax(), off.shape), off.max())


@pytest.mark.parametrize("dtype,d", [("float32", 5), ("bfloat16", 8), ("bfloat16", 5)])
def test_gates_over_many_blocks(dev, dtype, d):
    """Portions longer than the 1024 tokens the gates are scanned in at a time, and what they leave for the next one."""
    rng = np.random.default_rng(4)
    T, H = 2300, 2
    q, k, v = (O.bf16_round(rng.standard_normal((T, H, n))).astype(np.float64) for n in (d, d, 8))
    gates = (4 * rng.standard_normal((T, 2 * H)) + np.array([-1.0, 1.0, 6.0, 3.0])).astype(np.float32)
    want, want_den = plain_linear_state(q, k, v, gates, cap=12.0)
    size, tol = np.sqrt((want * want).mean(axis=(0, 2))), 2e-4 if dtype == "float32" else 1e-3
    for cuts in ([2300], [1025, 1, 1100, 3], [2047, 1]):
        got, den = linear_state(dev, q, k, v, dtype, cuts, gates, cap=12.0)
        assert (np.abs(got - want).max(axis=2) / size).max() < tol, cuts
        assert (np.abs(den - want_den) / np.maximum(want_den, size)).max() < tol, cuts


def test_the_state_stays_in_32_bits():
    """A sum that bf16 could not carry: a thousand additions of 1 to a state of 2^12, decay one, then one token at a time."""
    from denograd_b200.device import Device
    dev, T = Device["CUDA"], 1100
    q, k, v = np.zeros((T, 1, 8)), np.zeros((T, 1, 8)), np.ones((T, 1, 8))
    k[:, 0, 0], q[:, 0, 0] = 1.0, 2.0
    v[0] = 4096.0
    for cuts in ([1100], [1000, 1], [64]):
        got, _ = linear_state(dev, q, k, v, "bfloat16", cuts, decay=np.ones(1))
        want = 4096.0 + np.arange(T)
        assert np.abs(got[:, 0] - want[:, None]).max() < 0.2, cuts  # read through 16 bits on the tensor cores
        assert abs(got[-1, 0, 0] - want[-1]) < (0.2 if cuts[-1] != 1 else 1e-3)


# ------------------------------------------------------------------------------------------------ cuts, slots, pages
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_and_decoding_agree(dtype):
    params = O.random_params(MIXED, seed=5)
    toks = tokens(MIXED, 170)
    want = O.forward(params, MIXED, toks)
    # small pages and a small row limit: the rings of the attention layers wrap many times over 170 tokens
    m = build(MIXED, params, dtype, page_size=16, max_rows=40)
    assert [r.pinned for r in m.states.rings] == [1, 1, 2]
    for cuts in ([170], [1], [2], [3], [5, 7, 2, 31, 16, 1, 1, 2, 17], [100, 1], [64, 2, 64, 1]):
        check(run(m, toks, cuts), want, dtype, cuts)
    m = build(MIXED, params, dtype, jit=False)
    check(run(m, toks, [40, 1]), want, dtype)


def test_long_sequences():
    """Portions of many blocks, then decoding far from the start, in 32 bits and in bf16."""
    cfg = config(with_mlp(mlstm(dim=32, vdim=32, heads=2)), parallel(window(dim=16, vdim=16, heads=4, rot={"base": 1e4, "dims": 16}, mask={"keep_first": 4, "size": 50}),
                                                                    light((0.9, 0.999), dim=32, vdim=32)))
    params = O.random_params(cfg, seed=6)
    toks = tokens(cfg, 700)
    want = O.forward(params, cfg, toks)
    for dtype in ("float32", "bfloat16"):
        m = build(cfg, params, dtype, max_context=768, page_size=32, max_rows=300)
        for cuts in ([700], [129, 128, 257, 1], [300, 16, 17, 15, 65, 1]):
            check(run(m, toks, cuts), want, dtype, cuts)


def test_slots_and_pages_are_reused_in_any_order():
    params = O.random_params(MIXED, seed=7)
    m = build(MIXED, params, page_size=16, max_rows=32)
    seqs = [tokens(MIXED, n, seed=n) for n in (57, 3, 91, 20, 1, 64)]
    want = [O.forward(params, MIXED, s) for s in seqs]
    for i in (0, 1, 2, 3, 4, 5, 2, 0):
        slots = [m.acquire_slot() for _ in range(1 + i % 3)]  # different slots and pages each time
        assert error(run(m, seqs[i], [9, 1, 1, 4], slot=slots[-1]), want[i]) < F32_TOL
        for s in slots:
            m.release_slot(s)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_interleaved_requests(dtype):
    params = O.random_params(MIXED, seed=8)
    m = build(MIXED, params, dtype, page_size=16, max_rows=32)
    seqs = [tokens(MIXED, n, seed=10 + n) for n in (61, 34, 45)]
    want = [O.forward(params, MIXED, s) for s in seqs]
    slots, at, got = [m.acquire_slot() for _ in seqs], [0, 0, 0], [[], [], []]
    rng = np.random.default_rng(0)
    while any(at[i] < len(seqs[i]) for i in range(3)):
        i = int(rng.choice([j for j in range(3) if at[j] < len(seqs[j])]))
        n = min(int(rng.choice([1, 1, 2, 5, 13, 20])), len(seqs[i]) - at[i])
        got[i].append(m.feed(slots[i], seqs[i][at[i]:at[i] + n], at[i], range(n)))
        at[i] += n
    for g, w in zip(got, want):
        check(np.concatenate(g), w, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("B", [2, 3])
def test_batch_rows_against_each_alone(B, dtype):
    """Batch rows of the model's own API: prompts and decode steps, each row against the oracle on its own."""
    params = O.random_params(MIXED, seed=9)
    m = build(MIXED, params, dtype)
    toks = np.array([tokens(MIXED, 90, seed=30 + b) for b in range(B)], np.int32)
    want = [O.forward(params, MIXED, t) for t in toks]
    at, got, ref = 0, [], []
    for n in (23, 2, 1, 1, 1, 20, 1, 1, 40):
        m.call(toks[:, at:at + n], at)
        at += n
        got.append(m.last_logits(B))
        ref.append(np.stack([w[at - 1] for w in want]))
    check(np.concatenate(got), np.concatenate(ref), dtype)


def test_state_goes_on_from_where_it_is_or_starts_anew():
    params = O.random_params(MIXED, seed=9)
    m = build(MIXED, params)
    s = m.acquire_slot()
    m.feed(s, tokens(MIXED, 9), 0)
    for bad in (4, 12):
        with pytest.raises(ValueError):
            m.feed(s, [1], bad)
    toks = tokens(MIXED, 12, seed=5)
    assert error(run(m, toks, [5, 1], slot=s), O.forward(params, MIXED, toks)) < F32_TOL  # position 0: a new sequence


# ------------------------------------------------------------------------------------------------ edges that one key decides
def needle_model(size, first, seed=11, sharp=60.0):
    """One layer in which token 2 looks for token 1 far more than for anything else, so that whether the key is seen decides the
    logits: the queries of token 2 and the keys of token 1 share a direction that is not rotated and that others lack."""
    left = window(heads=2, kv_heads=1, dim=16, vdim=24, mask={"keep_first": first, "size": size} if size else None, rot={"base": 500.0, "dims": 8}, scale=0.5)
    cfg = config(parallel(left, light((0.5,), dim=8, vdim=8), 1.0, 0.2), width=64, vocab=16)
    p = O.random_params(cfg, seed)
    x = np.asarray(p["embed"], np.float64) * cfg["embedding"]["scale"]
    basis = np.linalg.pinv(x)  # basis[:, t] . x[t'] = (t == t'): 16 tokens in 64 dimensions
    P = "l0.mix.left."
    for n in ("q", "k"):
        p[P + n + ".norm"][:] = 1.0
        p[P + n + ".b"][:] = 0.3 * p[P + n + ".b"]
    for h in range(2):
        p[P + "q"][h * 16 + 15] += sharp * basis[:, 2]
    p[P + "k"][15] += sharp * basis[:, 1]
    return cfg, {k: O.bf16_round(v) for k, v in p.items()}


def needle_tokens(n, key, query, seed=5):
    t = np.random.default_rng(seed).integers(3, 16, n)
    t[key], t[query] = 1, 2
    return t.tolist()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [9, 16, 64])
@pytest.mark.parametrize("key", [4, 14, 15, 16, 31])
def test_window_edge(dtype, size, key):
    """The last position that still sees a key and the first that does not, with the key around page borders and behind the kept
    tokens: whole, cut right before the query, cut between key and query, and decoded."""
    cfg, p = needle_model(size, 3)
    m = build(cfg, p, dtype, page_size=16, max_rows=32)
    tol = F32_TOL if dtype == "float32" else BF16_TOL
    for back, seen in ((1, True), (size - 1, True), (size, False), (size + 1, False)):
        query = key + back
        toks = needle_tokens(query + 3, key, query)
        want = O.forward(p, cfg, toks)
        if back in (size - 1, size):  # the comparison below would notice
            wrong = O.forward(p, cfg, toks, faults=["window_short" if seen else "window_long"])
            assert error(wrong[query:query + 1], want[query:query + 1]) > 4 * tol
        for cuts in ([len(toks)], [query, 2, 1], [key + 1, 1], [max(1, query - 1), 2, 1]):
            assert error(run(m, toks, cuts)[query], want[query]) < tol, (back, cuts)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("first", [1, 15, 16, 17, 33])
def test_first_tokens(dtype, first):
    """The last token that is kept and the first that is not, from far away, with kept tokens ending inside, at and behind a page."""
    cfg, p = needle_model(9, first)
    m = build(cfg, p, dtype, page_size=16, max_rows=32)
    tol = F32_TOL if dtype == "float32" else BF16_TOL
    for key, fault in ((0, None), (first - 1, "one_less_first"), (first, "one_more_first")):
        for query in (first + 9, first + 30, 150):
            toks = needle_tokens(query + 2, key, query)
            want = O.forward(p, cfg, toks)
            if fault:
                wrong = O.forward(p, cfg, toks, faults=[fault])
                assert error(wrong[query:query + 1], want[query:query + 1]) > 4 * tol
            for cuts in ([len(toks)], [query, 1], [query - 1, 2], [20, 20, 7, 1]):
                assert error(run(m, toks, cuts)[query], want[query]) < tol, (key, query, cuts)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_key_without_a_window(dtype):
    cfg, p = needle_model(0, 0)
    m = build(cfg, p, dtype, page_size=16)
    tol = F32_TOL if dtype == "float32" else BF16_TOL
    for key, query in ((0, 200), (17, 230), (127, 128)):
        toks = needle_tokens(query + 1, key, query)
        want = O.forward(p, cfg, toks)
        gone = O.forward(p, cfg, [4 if t == 1 else t for t in toks])
        assert error(gone[query:], want[query:]) > 4 * tol
        for cuts in ([query + 1], [query, 1], [64, 64, 64, 2]):
            assert error(run(m, toks, cuts)[query], want[query]) < tol


def weak_inputs():
    """An mLSTM layer whose input gates are nearly shut from the first token on: the divisor's floor decides how large the head is
    against eps, which the norm behind it would otherwise hide."""
    cfg = config(mlstm(gate_cap=20.0), eps=1e-3)
    params = O.random_params(cfg, seed=5)
    params["l0.mix.i.b"][:], params["l0.mix.f.b"][:] = -5.0, 6.0
    return cfg, params


@pytest.mark.parametrize("fault", ["no_floor", "state_lost", "norm_per_head", "head_map", "no_side", "one_less_first", "window_short"])
def test_the_comparison_notices(fault):
    """Mistakes planted in the oracle stand out from the tolerance the other tests use."""
    cfg, params = weak_inputs() if fault in ("no_floor") else (MIXED, O.random_params(MIXED, seed=5))
    toks = tokens(cfg, 60)
    want, wrong = O.forward(params, cfg, toks), O.forward(params, cfg, toks, faults=[fault])
    for cuts in ([60], [21, 1]):
        got = run(build(cfg, params), toks, cuts)
        assert error(got, want) < F32_TOL and error(got, wrong) > 20 * F32_TOL
    check(run(build(cfg, params, "bfloat16"), toks, [30, 1]), want, "bfloat16")


def test_first_positions_in_a_full_slot():
    """A new sequence in a slot that an earlier request left full."""
    params = O.random_params(MIXED, seed=12)
    m = build(MIXED, params, max_batch=1)
    run(m, tokens(MIXED, 90, seed=2), [90])
    for n in (1, 2, 3, 5, 6, 20):
        toks = tokens(MIXED, n, seed=40 + n)
        want = O.forward(params, MIXED, toks)
        for cuts in ([n], [1], [2, 1]):
            assert error(run(m, toks, cuts), want) < F32_TOL


# ------------------------------------------------------------------------------------------------ drivers
def driver(cfg, params, dtype="float32", **kw):
    from denograd_b200.rigazen import Rigazen
    return Rigazen(cfg, dtype, max_context=256, max_batch=2, **kw).load_state_dict(params)


def greedy(params, cfg, prompt, n):
    toks, margins = list(prompt), []
    for _ in range(n):
        l = O.forward(params, cfg, toks)[-1]
        top = np.sort(l)[-2:]
        margins.append((top[1] - top[0]) / l.std())
        toks.append(int(l.argmax()))
    return toks[len(prompt):], margins


def test_greedy_generation():
    params = O.random_params(MIXED, seed=14)
    prompts = [tokens(MIXED, 12, seed=s) for s in (1, 2)]
    refs = [greedy(params, MIXED, p, 40) for p in prompts]
    assert min(min(r[1]) for r in refs) > 1e-3  # no near-ties: the ids must match
    want = np.array([r[0] for r in refs])
    llm = driver(MIXED, params, temperature=0)
    for batched in (False, True):
        llm.reset()
        assert (llm.generate(np.array(prompts, np.int32), 40, batched=batched) == want).all()
        assert (llm.model.last_logits(2).argmax(1) == want[:, -1]).all()
    llm.reset()
    first = llm.prefill(np.array(prompts, np.int32)).numpy()
    loop = llm.model.decode_loop(first, llm.start_pos, 20)
    assert (loop == want[:, 1:21]).all()
    loop = llm.model.decode_loop(want[:, 20], llm.start_pos + 20, 12, resume=True)
    assert (loop == want[:, 21:33]).all()
    # one row: the fused decode step
    llm.reset()
    assert (llm.generate(np.array(prompts[0], np.int32), 40) == want[:1]).all()


def test_prefix_reuse_and_sampling():
    params = O.random_params(MIXED, seed=13)
    llm = driver(MIXED, params, temperature=0)
    a, b = tokens(MIXED, 20, seed=3), tokens(MIXED, 15, seed=4)
    for prompt in (a, a + b, a + b[:3], b, a):
        llm.start_pos = 0
        out = llm._prefill(prompt, batched=True)
        assert out.numpy()[0] == O.forward(params, MIXED, prompt)[-1].argmax(), prompt
    llm.temperature, llm.top_k, llm.top_p = 0.8, 1, 0.5  # one candidate: the draw is the greedy pick
    llm.start_pos, llm.last_seen_toks = 0, []
    assert llm._prefill(b, batched=True).numpy()[0] == O.forward(params, MIXED, b)[-1].argmax()
    llm.top_k = 0
    tok = llm._call(5)
    assert 0 <= tok < MIXED["vocab"]


def test_trace_replay_and_command_line(tmp_path):
    """The programs a user starts: bin/trace_run in both element types, and generation from a model folder."""
    params = O.random_params(MIXED, seed=14)
    folder, out = tmp_path / "m", tmp_path / "out"
    folder.mkdir()
    out.mkdir()
    (folder / "config.json").write_text(json.dumps(MIXED))
    write_safetensors_bf16(str(folder / "model.safetensors"), params)
    toks = tokens(MIXED, 50)
    want = O.forward(params, MIXED, toks)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:30], "want": [0, 29, 7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[30:31], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[31:33], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": toks[33:], "want": [16]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": toks[:2], "want": [1]}], "end": ["b"]}]
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", 2 * BF16_TOL)):
        p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr
        assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
        for i, rows in ((0, [0, 29, 7]), (1, [30]), (3, [49]), (4, [1])):
            got = np.fromfile(out / f"{i}.f32", "<f4").reshape(len(rows), -1)
            assert error(got, want[rows]) < tol
            (out / f"{i}.f32").unlink()
        assert not (out / "2.f32").exists()
    p = subprocess.run([sys.executable, "-m", "denograd_b200", "generate", "--model", str(folder), "--dtype", "float32", "--tokens",
                        ",".join(map(str, toks[:9])), "--max-new", "5"], capture_output=True, text=True, cwd=ROOT, timeout=600)
    assert p.returncode == 0, p.stderr
    assert p.stdout.split() == [str(t) for t in greedy(params, MIXED, toks[:9], 5)[0]]
