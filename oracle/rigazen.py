"""Plain restatement of the Rigazen decoder in numpy float64, one function per mechanism, one token or one score at a time
where that is the clearest way to say it.  Test infrastructure only: it shares no code with denograd_b200 and keeps no
cache — every call starts from the whole token sequence.

Parameters are a dict name -> array under the checkpoint's tensor names; a configuration is the checkpoint's config.json
as a dict.  ``faults`` lets a test plant a mistake here (a window one longer, a first token that is dropped, a lost state,
...) and see that the comparison notices it.
"""
from __future__ import annotations

import math

import numpy as np

from .matulorn import F, bf16_round, rms, sigmoid, silu, sub


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def log_sigmoid(z):
    return -np.logaddexp(0.0, -np.asarray(z, F))


def rotate_half(x, pos, dims, base):
    """Entries i and i + dims/2 of a vector turn by pos * base^(-2i/dims); entries from `dims` on stay."""
    y = np.array(x, F)
    half = dims // 2
    for i in range(half):
        a = pos * base ** (-2.0 * i / dims)
        u, v = x[i], x[i + half]
        y[i], y[i + half] = u * math.cos(a) - v * math.sin(a), v * math.cos(a) + u * math.sin(a)
    return y


def mlstm(h, p, cfg, eps, faults=()):
    H, d, vd, cap = cfg["heads"], cfg["dim"], cfg["vdim"], cfg["gate_cap"]
    T = h.shape[0]
    q = (h @ p["q"].T).reshape(T, H, d) * d ** -0.5
    k, v = (h @ p["k"].T).reshape(T, H, d), (h @ p["v"].T).reshape(T, H, vd)
    gate_i = cap * np.tanh((h @ p["i"].T + p["i.b"]) / cap)
    gate_f = log_sigmoid(cap * np.tanh((h @ p["f"].T + p["f.b"]) / cap))
    S, n = np.zeros((H, d, vd), F), np.zeros((H, d), F)
    m = np.zeros(H, F)
    o = np.empty((T, H, vd), F)
    for t in range(T):
        if "state_lost" in faults and t % 7 == 3:
            S[:], n[:] = 0.0, 0.0
        for a in range(H):
            new = max(gate_f[t, a] + m[a], gate_i[t, a])
            keep, put = math.exp(gate_f[t, a] + m[a] - new), math.exp(gate_i[t, a] - new)
            S[a] = keep * S[a] + put * np.outer(k[t, a], v[t, a])
            n[a] = keep * n[a] + put * k[t, a]
            m[a] = new
            floor = 0.0 if "no_floor" in faults else math.exp(-new)
            o[t, a] = S[a].T @ q[t, a] / (max(abs(n[a] @ q[t, a]), floor) + 1e-6)
    o = rms(o, eps).reshape(T, H * vd) * p["norm"] * sigmoid(h @ p["g"].T)
    return o @ p["o"].T


def window_attention(h, p, cfg, eps, faults=()):
    H, G, d, vd = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]
    q, k, v = (h @ p[n].T + p[n + ".b"] for n in "qkv")
    if "norm_per_head" in faults:
        q = rms(q.reshape(T, H, d), eps).reshape(T, H * d) * p["q.norm"]
    else:
        q = rms(q, eps) * p["q.norm"]
    k = rms(k, eps) * p["k.norm"]
    q, k, v = q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, vd)
    rot = cfg["rot"]
    q = np.array([[rotate_half(q[t, a], t, rot["dims"], rot["base"]) for a in range(H)] for t in range(T)])
    k = np.array([[rotate_half(k[t, a], t, rot["dims"], rot["base"]) for a in range(G)] for t in range(T)])
    mask = cfg.get("mask") or {}
    size, first = mask.get("size"), mask.get("keep_first") or 0
    if size is not None:
        size += 1 if "window_long" in faults else (-1 if "window_short" in faults else 0)
    first += 1 if "one_more_first" in faults else (-1 if "one_less_first" in faults else 0)
    o = np.zeros((T, H, vd), F)
    for i in range(T):
        seen = [j for j in range(i + 1) if size is None or i - j < size or j < first]
        for a in range(H):
            g = a % G if "head_map" in faults else a // (H // G)
            s = k[seen, g] @ q[i, a] * cfg["scale"]
            e = np.exp(s - s.max())
            o[i, a] = e / e.sum() @ v[seen, g]
    return o.reshape(T, H * vd) @ p["o"].T


def lightning(h, p, cfg, eps, faults=()):
    H, d, vd = cfg["heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]
    q, k, v = (silu(h @ p[n].T).reshape(T, H, -1) for n in "qkv")
    S, o = np.zeros((H, d, vd), F), np.empty((T, H, vd), F)
    for t in range(T):
        if "state_lost" in faults and t % 7 == 3:
            S[:] = 0.0
        for a in range(H):
            S[a] = cfg["decay"][a] * S[a] + np.outer(k[t, a], v[t, a])
            o[t, a] = S[a].T @ q[t, a]
    o = rms(o, eps).reshape(T, H * vd) if "norm_per_head" in faults else rms(o.reshape(T, H * vd), eps)
    return (o * p["norm"] * sigmoid(h @ p["g"].T)) @ p["o"].T


def parallel(h, p, cfg, eps, faults=()):
    left = window_attention(h, sub(p, "left."), cfg["left"], eps, faults)
    right = lightning(h, sub(p, "right."), cfg["right"], eps, faults)
    return cfg["left_scale"] * left + cfg["right_scale"] * right


def squared_relu_ff(h, p):
    return np.maximum(h @ p["up"].T, 0.0) ** 2 @ p["down"].T


def token_side(x, e, p, eps):
    y = (gelu_tanh(x @ p["gate"].T) * e) @ p["proj"].T
    return rms(y, eps) * p["norm"]


MIXERS = {"mlstm": mlstm, "parallel": parallel}


def forward(params, config, tokens, faults=(), layer_outputs=None):
    """Logits [tokens, vocab] in float64 of one sequence from its first token on."""
    eps, tokens = config["norm"]["eps"], np.asarray(tokens)
    g = {k: np.asarray(v, F) for k, v in params.items()}
    x = g["embed"][tokens] * config["embedding"]["scale"]
    n = config["token_side"]["dim"]
    for i, lc in enumerate(config["layers"]):
        L = f"l{i}."
        x = x + rms(MIXERS[lc["type"]](x, sub(g, L + "mix."), lc["mixer"], eps, faults), eps) * (1.0 + g[L + "norm1"])
        if lc.get("mlp"):
            x = x + rms(squared_relu_ff(x, sub(g, L + "mlp.")), eps) * (1.0 + g[L + "norm2"])
        if "no_side" not in faults:
            x = x + token_side(x, g["side.embed"][tokens, i * n:(i + 1) * n], sub(g, L + "side."), eps)
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return rms(x, eps) * (1.0 + g["final.norm"]) @ g["embed"].T


# ------------------------------------------------------------------------------------------------ random models
def tensor_shapes(config):
    """name -> shape of every tensor of a model with this configuration."""
    D, V, n = config["width"], config["vocab"], config["token_side"]["dim"]
    s = {"embed": (V, D), "side.embed": (V, n * len(config["layers"])), "final.norm": (D,)}
    for i, lc in enumerate(config["layers"]):
        L, M, m = f"l{i}.", f"l{i}.mix.", lc["mixer"]
        s[L + "norm1"] = (D,)
        if lc["type"] == "mlstm":
            H, qk, v = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
            s.update({M + "q": (qk, D), M + "k": (qk, D), M + "v": (v, D), M + "g": (v, D), M + "o": (D, v), M + "norm": (v,)})
            s.update({M + "i": (H, D), M + "i.b": (H,), M + "f": (H, D), M + "f.b": (H,)})
        elif lc["type"] == "parallel":
            a, r, P, Q = m["left"], m["right"], M + "left.", M + "right."
            for name, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                s[P + name], s[P + name + ".b"] = (rows, D), (rows,)
                if name != "v":
                    s[P + name + ".norm"] = (rows,)
            s[P + "o"] = (D, a["heads"] * a["vdim"])
            qk, v = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            s.update({Q + "q": (qk, D), Q + "k": (qk, D), Q + "v": (v, D), Q + "g": (v, D), Q + "o": (D, v), Q + "norm": (v,)})
        else:
            raise ValueError(lc["type"])
        if lc.get("mlp"):
            f = lc["mlp"]["ff"]
            s.update({L + "norm2": (D,), L + "mlp.up": (f, D), L + "mlp.down": (D, f)})
        s.update({L + "side.gate": (n, D), L + "side.proj": (D, n), L + "side.norm": (D,)})
    return s


def random_params(config, seed=0):
    """bfloat16-representable float32 weights at scales that keep every mechanism visible in the logits."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2") or name == "final.norm":
            v = 0.2 * rng.standard_normal(shape)
        elif leaf == "norm":
            v = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name.endswith("f.b"):
            v = 2.0 + rng.standard_normal(shape)
        elif leaf == "b":
            v = 0.3 * rng.standard_normal(shape)
        elif name == "embed":
            v = rng.standard_normal(shape) / config["embedding"]["scale"]
        elif name == "side.embed":
            v = rng.standard_normal(shape)
        else:
            v = rng.standard_normal(shape) * (1.2 / math.sqrt(shape[-1]))
        out[name] = bf16_round(v)
    return out
