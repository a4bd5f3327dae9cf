"""Host side of the layer-list models without a GPU: slots and page rings, plans, configuration, checkpoints, the trace
replay's protocol, and known answers of the oracle the GPU tests compare with."""
import ctypes as C
import io
import json
import math

import numpy as np
import pytest

from denograd_b200 import ffi, registry
from denograd_b200.device import from_bf16_bits, to_bf16_bits
from denograd_b200.hybrid import HybridTransformer, yarn_table
from oracle import matulorn as O
from tests.fake_ffi import recording
from tests.util import write_safetensors_bf16

CFG = {"architecture": "Matulorn", "norm": {"eps": 1e-5, "groups": 2}, "vocab": 33, "width": 40, "layers": [
    {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 50, "limit": 3.0},
     "mixer": {"dim": 12, "heads": 3, "kv_rank": 20, "mask": {"size": 21}, "rot": {"base": 1000.0, "dims": 8, "scaling": None}, "rot_dim": 8, "scale": 0.3, "vdim": 10}},
    {"type": "delta", "mlp": None, "mixer": {"conv": 3, "dim": 12, "heads": 4, "kv_heads": 2, "vdim": 6}},
    {"type": "mingru", "mlp": {"kind": "dense", "ff": 24, "limit": 1.0}, "mixer": {"width": 30}}]}


def test_slots_and_page_rings():
    with recording():
        m = HybridTransformer(CFG, max_context=300, max_batch=3, page_size=16, max_rows=40)
        st, ring = m.states, m.states.rings[0]
        assert ring.pages_per_slot == math.ceil((21 - 1 + 40) / 16) and ring.n_pages == 3 * ring.pages_per_slot
        a, b = st.acquire(), st.acquire()
        pages = ring._table[[a, b]].ravel().tolist()
        assert len(set(pages)) == len(pages)
        st.advance(a, 0, 10)
        st.advance(a, 10, 5)
        with pytest.raises(ValueError):
            st.advance(a, 12, 1)
        with pytest.raises(ValueError):
            st.advance(a, 15, 290)
        st.advance(a, 0, 300)
        st.release(a)
        with pytest.raises(ValueError):
            st.release(a)
        c, d = st.acquire(), st.acquire()
        assert st.length[c] == 0
        pages = ring._table[[b, c, d]].ravel().tolist()
        assert sorted(pages) == list(range(ring.n_pages))
        with pytest.raises(ValueError):
            st.acquire()
        small = HybridTransformer(CFG, max_context=20, max_batch=1, page_size=16)
        assert small.states.rings[0].pages_per_slot == 2  # the context is shorter than the window
        del m, small


def test_plans():
    """The decode step of one row folds norms and the minGRU recurrence into the projections; more rows do not."""
    with recording() as rec:
        m = HybridTransformer(CFG, max_context=64, max_batch=4)
        names = lambda B, S: _run(m, rec, B, S)  # noqa: E731
        attn, mlp = ["jg_dense", "jg_latent_attn", "jg_dense"], ["jg_dense", "jg_dense"]
        fused = ["jg_stream_embed", *attn, *mlp, "jg_dense", "jg_delta_rule", "jg_dense", "jg_dense", "jg_dense", *mlp, "jg_dense", "jg_argmax_finalize"]
        assert names(1, 1) == fused and names(2, 1) == fused
        n = "jg_stream_norm"
        rows = ["jg_stream_embed", n, *attn, n, *mlp, n, "jg_dense", "jg_delta_rule", "jg_dense", n, "jg_dense", "jg_mingru_scan", "jg_dense", n, *mlp]
        assert names(3, 1) == rows + [n, "jg_dense", "jg_argmax_finalize"]
        assert names(1, 9) == rows + ["jg_dense", "jg_argmax_finalize"]
        two = names(1, 2)
        assert n not in two and "jg_mingru_scan" in two
        ws = m._chunk(1, 1)
        p = ws.plans[(True, True)]
        st = [c[1].stream for c in p.calls if c and c[0] == "jg_dense" and c[1].x == 0]
        assert all(a.x_out == b.x for a, b in zip(st, st[1:]) if a.x_out)  # the stream moves on to the buffer that was written
        assert all(s.x_out != s.x for s in st) and st[0].y == 0 and all(s.y for s in st[1:])
        del m, ws, p


def _run(m, rec, B, S):
    n0 = len(rec.calls)
    m.forward(np.zeros((B, S), np.int32), 0)
    return [c[0] for c in rec.kernels(n0) if not c[0].endswith(("_floats", "_bytes"))]


def test_parameters_follow_the_configuration():
    with recording():
        m = HybridTransformer(CFG, max_context=64)
        assert {k: p.shape for k, p in m.params.items()} == O.tensor_shapes(CFG)
        params = O.random_params(CFG)
        m.load_state_dict(params)
        with pytest.raises(KeyError):
            m.load_state_dict({k: v for k, v in params.items() if k != "l1.mix.A_log"})
        with pytest.raises(KeyError):
            m.load_state_dict(dict(params, more=np.zeros(3)))
        with pytest.raises(ValueError):
            m.load_state_dict(dict(params, head=params["head"][:-1]))
        with pytest.raises(ValueError):
            HybridTransformer(dict(CFG, layers=[{"type": "fir", "mixer": {}, "mlp": None}]))
        with pytest.raises(ValueError):
            HybridTransformer(CFG, dtype="float16")
        with pytest.raises(ValueError):
            HybridTransformer(dict(CFG, norm={"eps": 1e-5, "groups": 3}))
        del m


def test_descriptor_sizes_match_the_header():
    """Field by field, against the struct definitions in the header."""
    import re

    from tests.test_abi import HEADER
    src = re.sub(r"/\*.*?\*/", "", open(HEADER).read(), flags=re.S)
    for name, cls in (("jg_batch", ffi.Batch), ("jg_stream_desc", ffi.StreamDesc), ("jg_dense_desc", ffi.DenseDesc), ("jg_mingru_desc", ffi.MinGruDesc),
                      ("jg_delta_desc", ffi.DeltaDesc), ("jg_latent_desc", ffi.LatentDesc), ("jg_gated_desc", ffi.GatedDesc),
                      ("jg_linear_desc", ffi.LinearDesc), ("jg_window_desc", ffi.WindowDesc)):
        body = re.search(r"typedef struct \{([^}]*)\} " + name + ";", src).group(1)
        want = []
        for decl in body.split(";"):
            if decl.strip():
                kind, rest = decl.split(None, 1)
                want += [(n.strip(), kind) for n in rest.split(",")]
        kinds = {C.c_int32: "int32_t", C.c_uint64: "uint64_t", C.c_float: "float", ffi.StreamDesc: "jg_stream_desc", ffi.GatedDesc: "jg_gated_desc"}
        assert [(n, kinds[t]) for n, t in cls._fields_] == want, name


def test_bf16_values_survive(tmp_path):
    bits = np.arange(0, 1 << 16, 7, dtype=np.uint16)
    bits = bits[((bits >> 7) & 0xFF) != 0xFF]  # finite
    f = from_bf16_bits(bits)
    assert (to_bf16_bits(f) == bits).all()
    assert (from_bf16_bits(to_bf16_bits(np.float32([1 + 2.0 ** -8, 1 + 3 * 2.0 ** -8, -3.0e38]))) == O.bf16_round(np.float32([1 + 2.0 ** -8, 1 + 3 * 2.0 ** -8, -3.0e38]))).all()
    from denograd_b200.state import load_checkpoint
    path = str(tmp_path / "model.safetensors")
    write_safetensors_bf16(path, {"a": f.reshape(1, -1), "big": np.float32([[1e30, -1e-30]])})
    got = load_checkpoint(path, widen_bf16=True)
    assert got["a"].dtype == np.float32 and (got["a"] == f).all()
    assert (got["big"] == O.bf16_round(np.float32([[1e30, -1e-30]]))).all()  # outside the fp16 range


def test_registry(tmp_path):
    assert registry.architecture(CFG) == "Matulorn" and registry.architecture({"architectures": ["LlamaForCausalLM"]}) == "LlamaForCausalLM"
    with pytest.raises(ValueError):
        registry.architecture({"architectures": ["Nobody"]})
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    params = O.random_params(CFG)
    write_safetensors_bf16(str(tmp_path / "model.safetensors"), params)
    with recording():
        llm = registry.load(str(tmp_path), max_context=64, temperature=0)
        assert type(llm).__name__ == "Matulorn" and llm.model.dtype == "bfloat16" and llm.model.max_context == 64
        del llm
    llama = {"architectures": ["LlamaForCausalLM"], "hidden_size": 64, "num_attention_heads": 2, "num_hidden_layers": 1, "rms_norm_eps": 1e-5,
             "vocab_size": 50, "intermediate_size": 96}
    (tmp_path / "config.json").write_text(json.dumps(llama))
    with pytest.raises(registry.UnsupportedDtype):
        registry.load(str(tmp_path), "float32")
    from denograd_b200.trace import main
    assert main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path)]) == 3


class FakeModel:
    """Logits name the request's slot, the position and the token."""
    def __init__(self):
        self.free, self.log = [1, 0], []

    def acquire_slot(self):
        return self.free.pop()

    def release_slot(self, s):
        self.free.append(s)

    def feed(self, slot, toks, at, want):
        self.log.append((slot, list(toks), at))
        return np.array([[slot, at + w, toks[w]] for w in want], np.float32).reshape(len(want), 3)


def test_trace_protocol(tmp_path):
    from denograd_b200.trace import replay
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [9], "want": []}]},
             {"step": 2, "entries": [{"id": "a", "tokens": [8], "want": [0]}, {"id": "b", "tokens": [3, 4], "want": [1]}], "end": ["a"]},
             {"step": 7, "entries": [{"id": "c", "tokens": [1], "want": [0]}], "end": ["b", "c"]}]
    said, m = [], FakeModel()
    replay(m, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2", "done 7"] and sorted(m.free) == [0, 1]
    read = lambda i: np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, 3).tolist()  # noqa: E731
    assert read(0) == [[0, 0, 5], [0, 2, 7]] and not (tmp_path / "1.f32").exists()
    assert read(2) == [[0, 3, 8], [1, 2, 4]] and read(7) == [[0, 0, 1]]


def test_command_line_info(tmp_path, capsys):
    from denograd_b200.__main__ import main
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert main(["info", "--model", str(tmp_path)]) == 0
    assert json.loads(capsys.readouterr().out)["architecture"] == "Matulorn"


# ------------------------------------------------------------------------------------------------ the oracle's known answers
def test_oracle_known_answers():
    f, g = O.yarn_frequencies(8, 100.0, None)
    assert np.allclose(f, [1, 100 ** -0.25, 0.1, 100 ** -0.75]) and g == 1.0
    f, g = O.yarn_frequencies(8, 100.0, {"factor": 1.0, "original": 64, "fast": 8, "slow": 1})
    assert np.allclose(f, [1, 100 ** -0.25, 0.1, 100 ** -0.75]) and g == 1.0
    f, g = O.yarn_frequencies(8, 100.0, {"factor": 8.0, "original": 4, "fast": 1e6, "slow": 1e5})  # every wavelength is long
    assert np.allclose(f, np.array([1 / 8, 100 ** -0.25 / 8, 0.1 / 8, 100 ** -0.75 / 8])) or f[0] == 1.0
    assert math.isclose(g, 0.1 * math.log(8) + 1)
    x = np.arange(1.0, 6.0)
    y = O.rotate(x, 1, np.array([math.pi / 2, 0.0]), 1.0)
    assert np.allclose(y, [-3, 2, 1, 4, 5])  # pair (0, 2) turned by a quarter, pair (1, 3) not at all, the rest passes
    c = O.short_conv(np.array([[1.0], [0], [0], [2.0]]), np.array([[0.25, 0.5, 1.0]]))
    assert np.allclose(c[:, 0], [1, 0.5, 0.25, 2])
    n = O.group_norm(np.array([3.0, 4.0, 0.0, 2.0]), np.array([1.0, 1, 1, 2]), 2, 0.0)
    assert np.allclose(n, [3 / math.sqrt(12.5), 4 / math.sqrt(12.5), 0, 2 * math.sqrt(2)])


def test_rotary_tables_agree():
    for s in (None, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}, {"factor": 2.0, "original": 4096, "fast": 32.0, "slow": 1.0}):
        f, g = O.yarn_frequencies(16, 5000.0, s)
        t = yarn_table(16, 5000.0, s, 50)
        a = np.arange(50)[:, None] * f
        assert np.abs(t[..., 0] - np.cos(a) * g).max() < 1e-6 and np.abs(t[..., 1] - np.sin(a) * g).max() < 1e-6
