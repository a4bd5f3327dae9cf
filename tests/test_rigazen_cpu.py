"""Rigazen without a GPU: configuration, plans, pinned pages, parameters, checkpoints, and known answers of the oracle the GPU
tests compare with."""
import json
import math

import numpy as np
import pytest

from denograd_b200 import registry, synth
from denograd_b200.hybrid import Columns, HybridTransformer
from oracle import rigazen as O
from tests.fake_ffi import recording
from tests.util import write_safetensors_bf16

MLSTM = {"type": "mlstm", "mixer": {"dim": 12, "gate_cap": 8.0, "heads": 3, "vdim": 10}, "mlp": {"kind": "dense", "ff": 50}}
PARALLEL = {"type": "parallel", "mlp": None, "mixer": {
    "left": {"dim": 12, "heads": 4, "kv_heads": 2, "mask": {"keep_first": 18, "size": 21}, "rot": {"base": 1000.0, "dims": 8}, "scale": 0.3, "vdim": 10},
    "right": {"decay": [0.5, 0.9], "dim": 6, "heads": 2, "vdim": 14}, "left_scale": 0.5, "right_scale": 2.0}}
CFG = {"architecture": "Rigazen", "embedding": {"scale": 3.0}, "layers": [PARALLEL, MLSTM], "norm": {"eps": 1e-5}, "token_side": {"dim": 6}, "vocab": 33, "width": 40}


def test_pinned_pages():
    with recording():
        m = HybridTransformer(CFG, max_context=300, max_batch=3, page_size=16, max_rows=40)
        st, ring = m.states, m.states.rings[0]
        assert ring.pinned == 2 and ring.pages_per_slot == 2 + math.ceil((21 - 1 + 40) / 16) and ring.n_pages == 3 * ring.pages_per_slot
        a, b = st.acquire(), st.acquire()
        pages = ring._table[[a, b]].ravel().tolist()
        assert len(set(pages)) == len(pages)
        st.release(a)
        c, d = st.acquire(), st.acquire()
        assert sorted(ring._table[[b, c, d]].ravel().tolist()) == list(range(ring.n_pages))
        # every position that is still seen, and those of the longest portion, have places of their own
        def place(p):
            i = p // 16
            return (i if i < ring.pinned else ring.pinned + (i - ring.pinned) % (ring.pages_per_slot - ring.pinned)), p % 16
        for start in range(0, 260):
            seen = [p for p in range(start + 40) if p < 18 or p >= start - 20]
            assert len({place(p) for p in seen}) == len(seen)
        small = HybridTransformer(CFG, max_context=64, max_batch=1, page_size=16)
        assert small.states.rings[0].pinned == 0 and small.states.rings[0].pages_per_slot == 4  # the context fits
        del m, small


def names(m, rec, B, S):
    n0 = len(rec.calls)
    m.forward(np.zeros((B, S), np.int32), 0)
    return [c[0] for c in rec.kernels(n0) if not c[0].endswith(("_floats", "_bytes"))]


def test_plans():
    """One and two rows: norms, sums and what follows a recurrence are inside the projections; more rows: calls of their own."""
    with recording() as rec:
        m = HybridTransformer(CFG, max_context=64, max_batch=4)
        d, side = "jg_dense", ["jg_dense", "jg_dense"]
        fused = ["jg_stream_embed", d, "jg_window_attn", "jg_linear_state", d, *side, d, "jg_linear_state", d, d, d, *side, d, "jg_argmax_finalize"]
        assert names(m, rec, 1, 1) == fused and names(m, rec, 2, 1) == fused and names(m, rec, 1, 2) == fused
        n, g = "jg_stream_norm", "jg_gated_norm"
        rows = ["jg_stream_embed", n, d, "jg_window_attn", "jg_linear_state", g, d, n, *side, n, d, "jg_linear_state", g, d, n, d, d, n, *side]
        assert names(m, rec, 3, 1) == rows + [n, d, "jg_argmax_finalize"]
        assert names(m, rec, 1, 9) == rows + [d, "jg_argmax_finalize"]
        calls = [c[1] for c in m._chunk(1, 1).plans[(True, True)].calls if c and c[0] == d]
        inputs = [c.stream for c in calls if c.x == 0 and c.gated.o == 0]
        assert all(s.plain and s.w_norm == 0 for s in inputs) and len(inputs) == 5
        assert all(a.x_out == b.x for a, b in zip(inputs, inputs[1:]) if a.x_out)  # the stream moves on to the buffer that was written
        gated = [c for c in calls if c.gated.o]
        assert [c.lead for c in gated] == [40, 0] and [c.gated.groups for c in gated] == [1, 3] and [round(c.gated.scale, 6) for c in gated] == [2.0, 1.0]
        assert gated[0].gated.den == 0 and gated[1].gated.den
        del m


def test_parameters_follow_the_configuration():
    with recording():
        m = HybridTransformer(CFG, max_context=64)
        assert {k: p.shape for k, p in m.params.items()} == O.tensor_shapes(CFG)
        params = O.random_params(CFG)
        m.load_state_dict(params)
        assert m.head is m.embed
        with pytest.raises(KeyError):
            m.load_state_dict({k: v for k, v in params.items() if k != "l1.mix.f.b"})
        with pytest.raises(KeyError):
            m.load_state_dict(dict(params, head=params["embed"]))
        synth.fill_hybrid(m)
        assert m.params["final.norm"].offset == 1.0 and m.params["l0.side.norm"].offset == 0.0 and m.params["l1.mix.norm"].offset == 0.0
        bad = dict(PARALLEL, mixer=dict(PARALLEL["mixer"], right=dict(PARALLEL["mixer"]["right"], decay=[0.5])))
        for layers in ([bad], [dict(MLSTM, mlp={"kind": "moe"})], [dict(PARALLEL, mixer=dict(PARALLEL["mixer"], left=dict(PARALLEL["mixer"]["left"], kv_heads=3)))]):
            with pytest.raises(ValueError):
                HybridTransformer(dict(CFG, layers=layers), max_context=64)
        with pytest.raises(ValueError):
            HybridTransformer(dict(CFG, architecture="Nobody"), max_context=64)
        del m


def test_columns_wait_for_all_their_tensors():
    class Model:
        dtype = "float32"
    with recording():
        from denograd_b200.device import Device
        Model.dev, params = Device["CUDA"], {}
        c = Columns(Model, params, [("a", 5), ("b", 3)], 4)
        assert c.col0 == {"a": 0, "b": 8} and (c.K, c.ld) == (11, 16) and params["b"].ptr == c.ptr + 32
        sent = []
        c.weight.assign = lambda arr: sent.append(arr.copy())
        a, b = np.arange(20.0).reshape(4, 5), -np.arange(1.0, 13.0).reshape(4, 3)
        for order in ((("a", a), ("b", b)), (("b", b), ("a", a))):
            for name, v in order:
                assert not sent
                params[name].assign(v)
            w = sent.pop()
            assert (w[:, :5] == a).all() and (w[:, 5:8] == 0).all() and (w[:, 8:11] == b).all() and (w[:, 11:] == 0).all()


def test_registry_and_command_line(tmp_path, capsys):
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    write_safetensors_bf16(str(tmp_path / "model.safetensors"), O.random_params(CFG))
    with recording():
        llm = registry.load(str(tmp_path), max_context=64, temperature=0)
        assert type(llm).__name__ == "Rigazen" and llm.model.dtype == "bfloat16" and llm.model.embed_scale == 3.0
        del llm
    from denograd_b200.__main__ import main
    assert main(["info", "--model", str(tmp_path)]) == 0
    assert json.loads(capsys.readouterr().out)["architecture"] == "Rigazen"


def test_components():
    """A model's library holds the kernels of its mixers and not those of the others."""
    from denograd_b200 import build
    from denograd_b200.hybrid import MIXERS
    assert set(build.MIXER_COMPONENT) == set(MIXERS)
    assert build.component_of(["mlstm", "parallel"]) == "hybrid_branches" and build.component_of(["delta", "mingru"]) == "hybrid_recurrent"
    assert build.component_of(["delta", "mlstm"]) == "hybrid" and build.component_of(["unheard of"]) == "hybrid"
    assert "latent_attn.cu" not in build.COMPONENTS["hybrid_branches"] and "window_attn.cu" in build.COMPONENTS["hybrid_branches"]
    assert set(build.COMPONENTS["hybrid"]) <= set(build.SOURCES) and len(set(build.SOURCES)) == len(build.SOURCES)


# ------------------------------------------------------------------------------------------------ the oracle's known answers
def test_oracle_known_answers():
    y = O.rotate_half(np.arange(1.0, 7.0), 2, 4, 1.0)  # base 1: both pairs (0, 2) and (1, 3) turn by 2 radians, the rest passes
    c, s = math.cos(2), math.sin(2)
    assert np.allclose(y, [1 * c - 3 * s, 2 * c - 4 * s, 3 * c + 1 * s, 4 * c + 2 * s, 5, 6])
    assert np.allclose(O.gelu_tanh(np.array([0.0, 1.0, -1.0])), [0, 0.841192, -0.158808], atol=1e-6)
    assert np.allclose(O.log_sigmoid([0.0, 50.0, -50.0]), [-math.log(2), 0, -50])
    eye = np.eye(1)
    # mLSTM, one head of one dimension, gates at zero: i = 0, f = log 1/2, so S_t = S_{t-1} / 2 + k v and the same for n
    p = {"q": eye, "k": eye, "v": eye, "i": 0 * eye, "i.b": np.zeros(1), "f": 0 * eye, "f.b": np.zeros(1), "norm": np.ones(1), "g": 0 * eye, "o": eye}
    h = np.array([[2.0], [1.0]])
    out = O.mlstm(h, p, {"heads": 1, "dim": 1, "vdim": 1, "gate_cap": 5.0}, 1.0)
    o = [2 * 4 / (2 * 2 + 1e-6), 1 * (4 / 2 + 1) / (1 * (2 / 2 + 1) + 1e-6)]
    assert np.allclose(out[:, 0], [v / math.sqrt(v * v + 1) / 2 for v in o])
    # lightning, decay one half, silu on all three
    out = O.lightning(h, {k: p[k] for k in ("q", "k", "v", "norm", "g", "o")}, {"heads": 1, "dim": 1, "vdim": 1, "decay": [0.5]}, 1.0)
    a, b = (float(O.silu(np.float64(v))) for v in (2.0, 1.0))
    o = [a * a * a, b * (0.5 * a * a + b * b)]
    assert np.allclose(out[:, 0], [v / math.sqrt(v * v + 1) / 2 for v in o])
    # a window of one: every position sees itself and, with first tokens kept, those
    q = {"q": 0 * eye, "k": 0 * eye, "v": eye, "q.b": np.zeros(1), "k.b": np.zeros(1), "v.b": np.zeros(1), "q.norm": np.ones(1), "k.norm": np.ones(1), "o": eye}
    cfg = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "rot": {"dims": 0, "base": 1.0}, "scale": 1.0, "mask": {"size": 1, "keep_first": 0}}
    h = np.array([[1.0], [2.0], [4.0], [8.0]])
    assert np.allclose(O.window_attention(h, q, cfg, 1e-5)[:, 0], [1, 2, 4, 8])
    assert np.allclose(O.window_attention(h, q, dict(cfg, mask={"size": 1, "keep_first": 1}), 1e-5)[:, 0], [1, 1.5, 2.5, 4.5])
    assert np.allclose(O.window_attention(h, q, dict(cfg, mask={"size": 2, "keep_first": 1}), 1e-5)[:, 0], [1, 1.5, 7 / 3, 13 / 3])
