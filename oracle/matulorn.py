"""Plain restatement of the Matulorn decoder in numpy float64, one function per mechanism, one token or one score at a time
where that is the clearest way to say it.  Test infrastructure only: it shares no code with denograd_b200 and keeps no
cache — every call starts from the whole token sequence.

Parameters are a dict name -> array under the checkpoint's tensor names; a configuration is the checkpoint's config.json
as a dict.  ``faults`` lets a test plant a mistake here (a window one longer, a sink left out, ...) and see that the
comparison notices it.
"""
from __future__ import annotations

import math

import numpy as np

F = np.float64


def sigmoid(z):
    z = np.asarray(z, F)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def group_norm(x, w, groups, eps):
    """RMS norm of each of `groups` equal consecutive parts of the last axis, then times w."""
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return rms(parts, eps).reshape(x.shape) * w


def yarn_frequencies(dims, base, scaling):
    """Rotary frequencies of the dims/2 pairs and the factor on cos and sin."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], F)
    if not scaling:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    out = np.empty_like(f)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / scaling["factor"] * ramp + f[i] * (1.0 - ramp)
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, pos, freqs, mscale):
    """Half-split rotary on the first 2 * len(freqs) entries of a vector at position `pos`."""
    n = len(freqs)
    c, s = np.cos(pos * freqs) * mscale, np.sin(pos * freqs) * mscale
    y = np.array(x, F)
    u, v = x[:n], x[n:2 * n]
    y[:n], y[n:2 * n] = u * c - v * s, v * c + u * s
    return y


def mingru(h, p, cfg, eps, faults=()):
    z = sigmoid(h @ p["z"].T + p["z.b"])
    u = h @ p["x"].T + p["x.b"]
    cand = np.where(u >= 0, u + 0.5, sigmoid(u))
    g = silu(h @ p["g"].T)
    state = np.zeros(h.shape[:0] + (p["z"].shape[0],), F)
    out = np.empty((h.shape[0], state.shape[0]), F)
    for t in range(h.shape[0]):
        if "mingru_forgets" in faults and t % 7 == 3:
            state = np.zeros_like(state)
        state = (1.0 - z[t]) * state + z[t] * cand[t]
        out[t] = state * g[t]
    return out @ p["o"].T


def latent_attention(h, p, cfg, eps, faults=()):
    H, dim, rd, vd, rank = cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    window = (cfg.get("mask") or {}).get("size")
    if window is not None:
        window += 1 if "window_long" in faults else (-1 if "window_short" in faults else 0)
    T = h.shape[0]
    q = (h @ p["q"].T).reshape(T, H, dim + rd)
    ckr = h @ p["dkv"].T
    c = rms(ckr[:, :rank], eps) * p["dkv.norm"]
    freqs, ms = yarn_frequencies(cfg["rot"]["dims"], cfg["rot"]["base"], cfg["rot"].get("scaling"))
    if "rot_mscale" in faults:
        ms = 1.0
    kr = np.stack([rotate(ckr[t, rank:], t, freqs, ms) for t in range(T)])
    kn = (c @ p["uk"].T).reshape(T, H, dim)
    v = (c @ p["uv"].T).reshape(T, H, vd)
    out = np.zeros((T, H, vd), F)
    for i in range(T):
        j0 = 0 if window is None else max(0, i - window + 1)
        for n in range(H):
            qr = rotate(q[i, n, dim:], i, freqs, ms)
            s = (kn[j0:i + 1, n] @ q[i, n, :dim] + kr[j0:i + 1] @ qr) * cfg["scale"]
            sink = p["sink"][n]
            m = max(float(s.max()), float(sink))
            e = np.exp(s - m)
            denom = e.sum() + (0.0 if "no_sink" in faults else math.exp(sink - m))
            out[i, n] = (e / denom) @ v[j0:i + 1, n]
    return out.reshape(T, H * vd) @ p["o"].T


def short_conv(x, w):
    """Causal per-channel convolution over time: w[:, -1] is the current row's tap, rows before the first are zero."""
    taps = w.shape[1]
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                y[t] += w[:, j] * x[src]
    return y


def gated_delta(h, p, cfg, eps, faults=()):
    H, G, dim, vd = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]
    q = silu(short_conv(h @ p["q"].T, p["q.conv"])).reshape(T, G, dim)
    k = silu(short_conv(h @ p["k"].T, p["k.conv"])).reshape(T, G, dim)
    v = silu(short_conv(h @ p["v"].T, p["v.conv"])).reshape(T, H, vd)
    q = q / np.sqrt((q * q).sum(-1, keepdims=True) + 1e-6) * dim ** -0.5
    k = k / np.sqrt((k * k).sum(-1, keepdims=True) + 1e-6)
    beta = sigmoid(h @ p["b"].T)
    decay = np.exp(-np.exp(p["A_log"]) * softplus(h @ p["a"].T + p["dt_bias"]))
    S = np.zeros((H, dim, vd), F)
    o = np.empty((T, H, vd), F)
    rep = H // G
    for t in range(T):
        for n in range(H):
            g = n // rep if "head_map" not in faults else n % G
            S[n] = decay[t, n] * S[n]
            u = beta[t, n] * (v[t, n] - S[n].T @ k[t, g])
            S[n] = S[n] + np.outer(k[t, g], u)
            o[t, n] = S[n].T @ q[t, g]
    o = rms(o, eps) * p["norm"] * silu(h @ p["g"].T).reshape(T, H, vd)
    return o.reshape(T, H * vd) @ p["o"].T


def dense_ff(h, p, cfg):
    lim = cfg["limit"]
    g = np.minimum(h @ p["gate"].T + p["gate.b"], lim)
    u = np.clip(h @ p["up"].T + p["up.b"], -lim, lim)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ p["down"].T + p["down.b"]


MIXERS = {"mingru": mingru, "latent_attention": latent_attention, "delta": gated_delta}


def sub(params, prefix):
    return {k[len(prefix):]: np.asarray(v, F) for k, v in params.items() if k.startswith(prefix)}


def forward(params, config, tokens, faults=(), layer_outputs=None):
    """Logits [tokens, vocab] in float64 of one sequence from its first token on."""
    eps, groups = config["norm"]["eps"], config["norm"]["groups"]
    x = np.asarray(params["embed"], F)[np.asarray(tokens)]
    for i, lc in enumerate(config["layers"]):
        L = f"l{i}."
        norm = lambda v, name: group_norm(v, np.asarray(params[L + name], F), groups, eps)  # noqa: E731
        y = MIXERS[lc["type"]](norm(x, "norm1"), sub(params, L + "mix."), lc["mixer"], eps, faults)
        x = x + norm(y, "norm1b")
        if lc.get("mlp"):
            x = x + norm(dense_ff(norm(x, "norm2"), sub(params, L + "mlp."), lc["mlp"]), "norm2b")
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return group_norm(x, np.asarray(params["final.norm"], F), groups, eps) @ np.asarray(params["head"], F).T


# ------------------------------------------------------------------------------------------------ random models
def tensor_shapes(config):
    """name -> shape of every tensor of a model with this configuration."""
    D, V = config["width"], config["vocab"]
    s = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    for i, lc in enumerate(config["layers"]):
        L, m = f"l{i}.", lc["mixer"]
        s[L + "norm1"] = s[L + "norm1b"] = (D,)
        M = L + "mix."
        if lc["type"] == "mingru":
            W = m["width"]
            for n in "zxg":
                s[M + n] = (W, D)
            s[M + "z.b"] = s[M + "x.b"] = (W,)
            s[M + "o"] = (D, W)
        elif lc["type"] == "latent_attention":
            H = m["heads"]
            s[M + "q"] = (H * (m["dim"] + m["rot_dim"]), D)
            s[M + "dkv"] = (m["kv_rank"] + m["rot_dim"], D)
            s[M + "dkv.norm"] = (m["kv_rank"],)
            s[M + "uk"], s[M + "uv"] = (H * m["dim"], m["kv_rank"]), (H * m["vdim"], m["kv_rank"])
            s[M + "sink"] = (H,)
            s[M + "o"] = (D, H * m["vdim"])
        elif lc["type"] == "delta":
            H, G = m["heads"], m["kv_heads"]
            for n, c in (("q", G * m["dim"]), ("k", G * m["dim"]), ("v", H * m["vdim"])):
                s[M + n], s[M + n + ".conv"] = (c, D), (c, m["conv"])
            s[M + "b"] = s[M + "a"] = (H, D)
            s[M + "A_log"] = s[M + "dt_bias"] = (H,)
            s[M + "norm"], s[M + "g"], s[M + "o"] = (m["vdim"],), (H * m["vdim"], D), (D, H * m["vdim"])
        else:
            raise ValueError(lc["type"])
        if lc.get("mlp"):
            s[L + "norm2"] = s[L + "norm2b"] = (D,)
            f = lc["mlp"]["ff"]
            s.update({L + "mlp.gate": (f, D), L + "mlp.gate.b": (f,), L + "mlp.up": (f, D), L + "mlp.up.b": (f,),
                      L + "mlp.down": (D, f), L + "mlp.down.b": (D,)})
    return s


def bf16_round(a):
    """Nearest bfloat16 (ties to even) of float32 values, as float32."""
    b = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return (((b + 0x7FFF + ((b >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32)


def random_params(config, seed=0):
    """bfloat16-representable float32 weights at scales that keep every mechanism visible in the logits."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".", 1)[1] if name.startswith("l") else name
        if leaf.endswith("norm") or "norm" in leaf.rsplit(".", 1)[-1]:
            v = 1.0 + 0.2 * rng.standard_normal(shape)
        elif leaf.endswith(".conv"):
            v = rng.standard_normal(shape) * 0.5
        elif leaf.endswith("sink"):
            v = rng.standard_normal(shape)
        elif leaf.endswith("A_log"):
            v = np.log(rng.uniform(0.02, 2.0, shape))
        elif leaf.endswith("dt_bias"):
            v = rng.standard_normal(shape) - 1.0
        elif leaf.endswith(".b") and len(shape) == 1:
            v = 0.3 * rng.standard_normal(shape)
        elif name == "embed":
            v = rng.standard_normal(shape)
        else:
            v = rng.standard_normal(shape) * (1.6 / math.sqrt(shape[-1]))
        out[name] = bf16_round(v)
    return out
