"""Matulorn on the device against the plain restatement in oracle/matulorn.py: each mechanism alone and all together, in 32
bits (tight) and as served (bf16), whole prompts, portions, decoding, reused slots and pages, keys at every kind of edge,
and the drivers on top."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import matulorn as O
from tests.util import ROOT, write_safetensors_bf16

pytestmark = pytest.mark.gpu

YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}
F32_TOL, BF16_TOL = 2e-4, 0.06


def latent(**kw):
    c = {"dim": 24, "heads": 3, "kv_rank": 40, "mask": {"size": 11}, "rot": {"base": 5000.0, "dims": 16, "scaling": YARN}, "rot_dim": 16,
         "scale": 0.2, "vdim": 20}
    c.update(kw)
    return {"type": "latent_attention", "mixer": c, "mlp": None}


def delta(**kw):
    c = {"conv": 4, "dim": 20, "heads": 6, "kv_heads": 2, "vdim": 28}
    c.update(kw)
    return {"type": "delta", "mixer": c, "mlp": None}


def mingru(width=56):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": None}


def with_mlp(layer, ff=72, limit=1.5):
    return dict(layer, mlp={"kind": "dense", "ff": ff, "limit": limit})


def config(*layers, width=48, vocab=97, groups=3, eps=1e-5):
    return {"architecture": "Matulorn", "layers": list(layers), "norm": {"eps": eps, "groups": groups}, "vocab": vocab, "width": width}


MIXED = config(with_mlp(latent()), delta(), with_mlp(mingru()), with_mlp(delta(heads=2, kv_heads=2, dim=36, vdim=12, conv=2)), mingru(40),
               latent(heads=5, dim=8, rot_dim=8, rot={"base": 100.0, "dims": 8, "scaling": None}, vdim=16, kv_rank=24, mask={"size": 30}))


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
    """32 bits: every row.  bf16: all rows together, and no row far off (a row whose delta output is nearly zero before its
    norm magnifies rounding)."""
    worst = error(got, want)
    if dtype == "float32":
        assert worst < F32_TOL, (what, worst)
        return
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    total = float(np.sqrt((d * d).mean() / (w * w).mean()))
    assert total < BF16_TOL and worst < 10 * BF16_TOL, (what, total, worst)


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
    "mingru": config(mingru()),
    "mingru wide, one group": config(mingru(width=200), width=64, groups=1),
    "mingru, mlp, odd sizes": config(with_mlp(mingru(37), ff=51), width=44, groups=4, vocab=61),
    "delta": config(delta()),
    "delta, one head each, one tap": config(delta(heads=1, kv_heads=1, dim=8, vdim=8, conv=1)),
    "delta, ungrouped, wide": config(delta(heads=2, kv_heads=2, dim=72, vdim=100, conv=3)),
    "delta, large heads": config(delta(heads=2, kv_heads=1, dim=136, vdim=260, conv=5)),
    "latent": config(latent()),
    "latent, no window, no scaling": config(latent(mask=None, rot={"base": 300.0, "dims": 16, "scaling": None})),
    "latent, window of one": config(latent(mask={"size": 1})),
    "latent, part of the key part turns": config(latent(rot={"base": 300.0, "dims": 8, "scaling": dict(YARN, factor=1.0)})),
    "latent, odd sizes": config(latent(heads=1, dim=7, rot_dim=6, rot={"base": 50.0, "dims": 6, "scaling": YARN}, vdim=5, kv_rank=9)),
    "latent, wide": config(latent(heads=4, dim=64, rot_dim=32, rot={"base": 1e4, "dims": 32, "scaling": YARN}, vdim=64, kv_rank=160, mask={"size": 40}),
                           width=128, groups=2),
    "latent, many heads": config(latent(heads=20, dim=16, rot_dim=8, rot={"base": 1e4, "dims": 8, "scaling": YARN}, vdim=72, kv_rank=264, mask={"size": 50})),
    "latent, many heads, short latent": config(latent(heads=33, dim=8, rot_dim=8, rot={"base": 1e4, "dims": 8, "scaling": YARN}, vdim=8, kv_rank=72)),
    "latent, long latent": config(latent(heads=2, dim=16, kv_rank=600)),
    "mlp with a tight clamp": config(with_mlp(mingru(24), ff=40, limit=0.3)),
}


@pytest.mark.parametrize("name", SINGLE)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_layer(name, dtype):
    cfg = SINGLE[name]
    params = O.random_params(cfg, seed=3)
    toks = tokens(cfg, 70)
    want = O.forward(params, cfg, toks)
    m = build(cfg, params, dtype)
    check(run(m, toks, [70]), want, dtype)
    check(run(m, toks, [33, 1]), want, dtype)
    check(run(m, toks, [5, 9, 15]), want, dtype)  # portions below the size that expands keys and values


def test_layer_outputs():
    params = O.random_params(MIXED, seed=4)
    toks, layers = tokens(MIXED, 29), []
    O.forward(params, MIXED, toks, layer_outputs=layers)
    for n in (29, 2, 1):
        m = build(MIXED, params)
        got = m.layer_outputs(m.acquire_slot(), toks[:n])
        for g, w in zip(got, layers):
            assert np.abs(g - w[:n]).max() < 1e-4 * np.abs(w).max()


@pytest.mark.parametrize("D,groups", [(48, 1), (48, 4), (60, 4), (4096, 1), (96, 96), (40, 20)])
@pytest.mark.parametrize("R", [1, 2, 5])
def test_stream_step(dev, D, groups, R):
    """Post-norm of a sublayer, residual sum and the next norm, with and without a row list."""
    import ctypes as C

    from denograd_b200 import ffi
    from denograd_b200.device import Tensor
    rng = np.random.default_rng(0)
    x, y = rng.standard_normal((R + 2, D)).astype(np.float32), (5 * rng.standard_normal((R + 2, D))).astype(np.float32)
    wa, wn = (1 + rng.standard_normal(D)).astype(np.float32), (1 + rng.standard_normal(D)).astype(np.float32)
    rows = np.array([R + 1 - i for i in range(R)], np.int32)
    want_x = x + O.group_norm(y.astype(np.float64), wa, groups, 1e-3)
    want_h = O.group_norm(want_x, wn, groups, 1e-3)
    ld = (D + 7) // 8 * 8
    tx, ty, ta, tn, tr = (Tensor(v, device=dev) for v in (x, y, wa, wn, rows))
    out, h = Tensor.zeros((R + 2, D), "float32", dev), Tensor.zeros((R, ld), "float32", dev)
    b = ffi.Batch(R, 1, 0, 0, -1, 0)
    for use_rows in (False, True):
        st = ffi.StreamDesc(D, groups, 1e-3, 0, tx.ptr, ty.ptr, ta.ptr, out.ptr, tn.ptr, tr.ptr if use_rows else 0)
        dev.call("jg_stream_norm", C.byref(b), st, h.ptr, ld, ffi.JG_F32)
        sel = rows if use_rows else np.arange(R)
        assert np.abs(h.numpy()[:, :D] - want_h[sel]).max() < 2e-5 * np.abs(want_h).max()
        assert np.abs(out.numpy()[sel] - want_x[sel]).max() < 2e-5 * np.abs(want_x).max()


@pytest.mark.parametrize("M,N,K", [(1, 40, 48), (2, 33, 200), (1, 3000, 1024), (2, 513, 4104), (3, 130, 72), (17, 96, 64), (40, 257, 136), (100, 64, 1000),
                                   (300, 384, 520), (5, 128, 2048), (129, 1, 8)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("glu", [False, True])
def test_projection(dev, M, N, K, dtype, glu):
    import ctypes as C

    from denograd_b200 import ffi
    from denograd_b200.device import Tensor
    from denograd_b200.hybrid import DTYPES
    rng = np.random.default_rng(1)
    ld, ldy = (K + 7) // 8 * 8, (N + 7) // 8 * 8
    x = np.zeros((M, ld), np.float32)
    w = np.zeros((2, N, ld), np.float32)
    x[:, :K], w[:, :, :K] = O.bf16_round(rng.standard_normal((M, K))), O.bf16_round(rng.standard_normal((2, N, K)) / np.sqrt(K))
    bias = rng.standard_normal((2, N)).astype(np.float32)
    t = lambda a: Tensor.zeros(a.shape, dtype, dev).assign(a)  # noqa: E731
    tx, tw, tb = t(x), [t(w[0]), t(w[1])], [Tensor(b, device=dev) for b in bias]
    y = Tensor.zeros((2 * M, ldy), dtype if glu else "float32", dev)
    d = ffi.DenseDesc(DTYPES[dtype], ffi.DENSE_GLU if glu else ffi.DENSE_STORE, N, K, ld, ld, ldy, 0 if glu else 1, 0.7, 0, tx.ptr, tw[0].ptr, tw[1].ptr, 0,
                      tb[0].ptr, tb[1].ptr, 0, y.ptr)
    dev.call("jg_dense", C.byref(ffi.Batch(M, 1, 0, 0, -1, 0)), d)
    a, b = (x.astype(np.float64) @ w[i].T.astype(np.float64) + bias[i] for i in range(2))
    if glu:
        g, u = np.minimum(a, 0.7), np.clip(b, -0.7, 0.7)
        a = g * O.sigmoid(1.702 * g) * (u + 1)
    assert np.abs(y.numpy()[:M, :N] - a).max() < (2e-5 if dtype == "float32" or not glu else 2e-2)


# ------------------------------------------------------------------------------------------------ cuts, slots, pages
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_and_decoding_agree(dtype):
    params = O.random_params(MIXED, seed=5)
    toks = tokens(MIXED, 150)
    want = O.forward(params, MIXED, toks)
    # small pages and a small row limit: the rings of both attention layers wrap many times over 150 tokens
    m = build(MIXED, params, dtype, page_size=16, max_rows=40)
    for cuts in ([150], [1], [2], [3], [5, 7, 2, 31, 16, 1, 1, 2, 17], [100, 1], [64, 2, 64, 1]):
        check(run(m, toks, cuts), want, dtype, cuts)
    m = build(MIXED, params, dtype, jit=False)
    check(run(m, toks, [40, 1]), want, dtype)


@pytest.mark.parametrize("width,scan", [(mingru(70), "mingru"), (delta(), "delta")])
def test_long_recurrences(width, scan):
    """Portions longer than one block of the scans, then more portions, then decoding."""
    cfg = config(width)
    params = O.random_params(cfg, seed=6)
    toks = tokens(cfg, 420)
    want = O.forward(params, cfg, toks)
    m = build(cfg, params, max_context=512)
    for cuts in ([420], [129, 128, 130, 1], [300, 16, 17, 15, 1]):
        assert error(run(m, toks, cuts), want) < F32_TOL, cuts


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


def test_interleaved_requests():
    params = O.random_params(MIXED, seed=8)
    m = build(MIXED, params, page_size=16, max_rows=32)
    seqs = [tokens(MIXED, n, seed=10 + n) for n in (61, 34, 47)]
    want = [O.forward(params, MIXED, s) for s in seqs]
    slots, at, got = [m.acquire_slot() for _ in seqs], [0, 0, 0], [[], [], []]
    rng = np.random.default_rng(0)
    while any(at[i] < len(seqs[i]) for i in range(3)):
        i = int(rng.choice([j for j in range(3) if at[j] < len(seqs[j])]))
        n = min(int(rng.choice([1, 1, 2, 5, 13])), len(seqs[i]) - at[i])
        got[i].append(m.feed(slots[i], seqs[i][at[i]:at[i] + n], at[i], range(n)))
        at[i] += n
    for g, w in zip(got, want):
        assert error(np.concatenate(g), w) < F32_TOL


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("B", [2, 3])
def test_batch_rows_against_each_alone(B, dtype):
    """Batch rows of the model's own API: a prompt and decode steps, each row against the oracle on its own."""
    params = O.random_params(MIXED, seed=9)
    m = build(MIXED, params, dtype)
    toks = np.array([tokens(MIXED, 60, seed=30 + b) for b in range(B)], np.int32)
    want = [O.forward(params, MIXED, t) for t in toks]
    at, got, ref = 0, [], []
    for n in (23, 2, 1, 1, 1, 20, 1, 1):
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
    with pytest.raises(ValueError):
        m.feed(s, [1] * 300, 12)


# ------------------------------------------------------------------------------------------------ edges that one key decides
def needle_model(window, seed=11, rot_key=False):
    """One latent layer in which token 2, and only it, looks for token 1: a rank-one term makes their score stand out, so that
    whether the key is seen decides the logits."""
    layer = latent(mask={"size": window} if window else None, heads=2, scale=0.25)
    cfg = config(layer, width=48, vocab=16)
    p = O.random_params(cfg, seed)
    c = layer["mixer"]
    h = O.group_norm(p["embed"].astype(np.float64), p["l0.norm1"], cfg["norm"]["groups"], cfg["norm"]["eps"])
    basis = np.linalg.pinv(h)  # basis[:, t] . h[t'] = (t == t'): 16 tokens in 48 dimensions
    sub = O.sub(p, "l0.mix.")
    lat = O.rms((h[1] @ sub["dkv"].T)[:c["kv_rank"]], cfg["norm"]["eps"]) * sub["dkv.norm"]
    k = (lat @ sub["uk"].T).reshape(c["heads"], c["dim"])
    q = (h[2] @ sub["q"].T).reshape(c["heads"], -1)
    for n in range(c["heads"]):
        row = n * (c["dim"] + c["rot_dim"])
        aim = k[n] * (14.0 / c["scale"] / (k[n] @ k[n]))
        p["l0.mix.q"][row:row + c["dim"]] += np.outer(aim - q[n, :c["dim"]], basis[:, 2])
    p["l0.mix.q"] = O.bf16_round(p["l0.mix.q"])
    return cfg, p


def needle_tokens(n, key, query):
    t = np.random.default_rng(5).integers(3, 16, n)
    t[key], t[query] = 1, 2
    return t.tolist()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [9, 16, 64])
@pytest.mark.parametrize("key", [0, 14, 15, 16, 31])
def test_window_edge(dtype, window, key):
    """The last position that still sees a key and the first that does not, with the key around page borders: whole, cut
    right before the query, cut between key and query, and decoded."""
    cfg, p = needle_model(window)
    m = build(cfg, p, dtype, page_size=16, max_rows=32)
    tol = F32_TOL if dtype == "float32" else BF16_TOL
    for back, seen in ((1, True), (window - 1, True), (window, False), (window + 1, False)):
        query = key + back
        toks = needle_tokens(query + 3, key, query)
        want = O.forward(p, cfg, toks)
        wrong = O.forward(p, cfg, toks, faults=["window_short" if seen else "window_long"])
        if back in (window - 1, window):
            assert error(wrong[query], want[query]) > 10 * tol  # the comparison below would notice
        for cuts in ([len(toks)], [query, 2, 1], [key + 1, 1], [max(1, query - 1), 2, 1]):
            assert error(run(m, toks, cuts)[query], want[query]) < tol, (back, cuts)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_key_without_a_window(dtype):
    cfg, p = needle_model(0)
    m = build(cfg, p, dtype, page_size=16)
    tol = F32_TOL if dtype == "float32" else BF16_TOL
    for key, query in ((0, 200), (17, 230), (127, 128)):
        toks = needle_tokens(query + 1, key, query)
        want = O.forward(p, cfg, toks)
        gone = O.forward(p, cfg, [4 if t == 1 else t for t in toks])
        assert error(gone[query], want[query]) > 10 * tol
        for cuts in ([query + 1], [query, 1], [64, 64, 64, 2]):
            assert error(run(m, toks, cuts)[query], want[query]) < tol


@pytest.mark.parametrize("fault", ["no_sink", "rot_mscale", "head_map", "mingru_forgets"])
def test_the_comparison_notices(fault):
    """Mistakes planted in the oracle stand out from the tolerance the other tests use."""
    params = O.random_params(MIXED, seed=5)
    toks = tokens(MIXED, 40)
    want, wrong = O.forward(params, MIXED, toks), O.forward(params, MIXED, toks, faults=[fault])
    m = build(MIXED, params)
    got = run(m, toks, [40])
    assert error(got, want) < F32_TOL and error(got, wrong) > 20 * F32_TOL


def test_first_tokens_of_a_sequence():
    """Positions before the convolution's taps are filled, in a slot that an earlier request left full."""
    cfg = config(delta(conv=6), mingru(), latent())
    params = O.random_params(cfg, seed=12)
    m = build(cfg, params, max_batch=1)
    run(m, tokens(cfg, 50, seed=2), [50])
    for n in (1, 2, 3, 5, 6, 7):
        toks = tokens(cfg, n, seed=40 + n)
        want = O.forward(params, cfg, toks)
        for cuts in ([n], [1], [2, 1]):
            assert error(run(m, toks, cuts), want) < F32_TOL


# ------------------------------------------------------------------------------------------------ drivers
def driver(cfg, params, dtype="float32", **kw):
    from denograd_b200.matulorn import Matulorn
    return Matulorn(cfg, dtype, max_context=256, max_batch=2, **kw).load_state_dict(params)


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
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
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
