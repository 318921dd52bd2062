"""Plain restatement of the Siladra family in numpy float64: one function per mechanism, whole sequences only, no cache, no step
function, nothing shared with the product path.  Tests compare the native library against it.

A Siladra layer wraps each sublayer in two RMS norms: x += rms_b(mixer(rms_a(x))), then the same around the feed-forward; a layer may
be another layer once more (the same weights, a state of its own).  Mixers: "mlstm" (a matrix memory per head with exponential input
gates and logistic forget gates, both capped, kept in range by a running maximum that starts at 0), "parallel" (grouped softmax
attention with biased, normed, YaRN-rotated queries and keys beside a selective state-space scan; each output normed, half of their
sum) and "delta" (a decayed memory per head that is corrected towards v along k; q, k, v pass short convolutions and silu, q and k are
unit vectors).  Feed-forward: SiLU-gated experts, the largest router outputs of a token weighted by their own softmax, or none."""
from __future__ import annotations

import math

import numpy as np


def to_float(bits):
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def logistic(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * logistic(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def causal_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros in front of the sequence"""
    taps = w.shape[1]
    y = np.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < u.shape[0]:
            y[back:] += w[:, j] * u[:u.shape[0] - back]
    return y


# ------------------------------------------------------------------------------------------------ matrix memory with exponential gates
def mlstm_scan(q, k, v, i, f, book=None):
    """q, k [T, D], v [T, V], log gates i, f [T] of one head -> [T, V]"""
    T, D = q.shape
    S, n, m = np.zeros((D, v.shape[1])), np.zeros(D), 0.0
    out = np.zeros((T, v.shape[1]))
    for t in range(T):
        new = max(f[t] + m, i[t])
        keep, take = math.exp(f[t] + m - new), math.exp(i[t] - new)
        S = keep * S + take * np.outer(k[t], v[t])
        n = keep * n + take * k[t]
        m = new
        out[t] = (S.T @ q[t]) / (max(abs(n @ q[t]), math.exp(-m)) + 1e-6)
        if book is not None:
            book.setdefault("m", []).append(m)
            book.setdefault("nq", []).append(n @ q[t])
    return out


def mlstm(h, T, c, eps, book=None):
    n, H, D, V, cap = h.shape[0], c["heads"], c["dim"], c["vdim"], c["gate_cap"]
    q, k, v = (h @ T["q"].T).reshape(n, H, D) * D ** -0.5, (h @ T["k"].T).reshape(n, H, D), (h @ T["v"].T).reshape(n, H, V)
    i, f = soft_cap(h @ T["i"].T + T["i.b"], cap), -softplus(-soft_cap(h @ T["f"].T + T["f.b"], cap))
    o = np.stack([mlstm_scan(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a], None if book is None else book.setdefault(a, {})) for a in range(H)], axis=1)
    return unit_rms(o, eps).reshape(n, H * V) * T["norm"] * logistic(h @ T["g"].T) @ T["o"].T


# ------------------------------------------------------------------------------------------------ attention beside a selective scan
def yarn(dims, base, scaling):
    """(frequencies of the dims / 2 pairs, factor on cos and sin)"""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    factor, orig = float(scaling["factor"]), float(scaling["original"])
    at = lambda turns: dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(at(scaling["fast"])), 0), min(math.ceil(at(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(v, freqs, amp):
    """v [T, heads, n]: entries (2i, 2i + 1) turn by t * freqs[i] and are scaled by amp; entries beyond the pairs stay"""
    out = np.array(v, np.float64)
    pos = np.arange(v.shape[0], dtype=np.float64)[:, None]
    for i, f in enumerate(freqs):
        c, s = np.cos(pos * f) * amp, np.sin(pos * f) * amp
        out[..., 2 * i] = v[..., 2 * i] * c - v[..., 2 * i + 1] * s
        out[..., 2 * i + 1] = v[..., 2 * i + 1] * c + v[..., 2 * i] * s
    return out


def attention(h, T, c, eps, book=None):
    n, H, G, D, V = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = rms_norm((h @ T["q"].T + T["q.b"]).reshape(n, H, D), T["q.norm"], eps)
    k = rms_norm((h @ T["k"].T + T["k.b"]).reshape(n, G, D), T["k.norm"], eps)
    v = (h @ T["v"].T + T["v.b"]).reshape(n, G, V)
    rot = c.get("rot")
    if rot and rot.get("dims"):
        turn = yarn(int(rot["dims"]), rot["base"], rot.get("scaling"))
        q, k = rotate(q, *turn), rotate(k, *turn)
    out = np.zeros((n, H, V))
    for a in range(H):
        g = a // (H // G)
        s = np.where(np.tril(np.ones((n, n), bool)), q[:, a] @ k[:, g].T * c["scale"], -np.inf)
        w = np.exp(s - s.max(axis=-1, keepdims=True))
        w /= w.sum(axis=-1, keepdims=True)
        out[:, a] = w @ v[:, g]
        if book is not None:
            book.setdefault("weights", {})[a] = w
    return out.reshape(n, H * V) @ T["o"].T


def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, inner], A [inner, N], B, C [T, N], D [inner] -> [T, inner]"""
    S, out = np.zeros(A.shape), np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t]
        out[t] = S @ C[t] + D * x[t]
    return out


def mamba(h, T, c):
    inner, N, rank = c["inner"], c["state"], c["dt_rank"]
    xz = h @ T["in"].T
    x, z = silu(causal_conv(xz[:, :inner], T["conv"]) + T["conv.b"]), xz[:, inner:]
    p = x @ T["x"].T
    dt = softplus(p[:, :rank] @ T["dt"].T + T["dt.b"])
    y = selective_scan(x, dt, -np.exp(T["A_log"]), p[:, rank:rank + N], p[:, rank + N:], T["D"])
    return y * silu(z) @ T["o"].T


def parallel(h, T, c, eps, book=None):
    left = attention(h, sub(T, "left."), c["left"], eps, book)
    right = mamba(h, sub(T, "right."), c["right"])
    return 0.5 * (rms_norm(left, T["left.out"], eps) + rms_norm(right, T["right.out"], eps))


# ------------------------------------------------------------------------------------------------ gated delta rule
def delta_scan(q, k, v, beta, g):
    """q, k [T, D], v [T, V], beta, g [T] of one head -> [T, V]"""
    S, out = np.zeros((q.shape[1], v.shape[1])), np.zeros((q.shape[0], v.shape[1]))
    for t in range(q.shape[0]):
        S = g[t] * S
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def delta(h, T, c, eps):
    n, H, G, D, V = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (silu(causal_conv(h @ T[t].T, T[t + ".conv"])) for t in ("q", "k", "v"))
    q, k, v = unit(q.reshape(n, G, D)) * D ** -0.5, unit(k.reshape(n, G, D)), v.reshape(n, H, V)
    beta = logistic(h @ T["b"].T)
    g = np.exp(-np.exp(T["A_log"]) * softplus(h @ T["a"].T + T["dt_bias"]))
    o = np.stack([delta_scan(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], beta[:, a], g[:, a]) for a in range(H)], axis=1)
    return (rms_norm(o, T["norm"], eps) * silu(h @ T["g"].T).reshape(n, H, V)).reshape(n, H * V) @ T["o"].T


# ------------------------------------------------------------------------------------------------ experts, the model
def route(z, top):
    """router outputs z [T, E] -> (choices [T, top], weights [T, top]): the largest outputs, the softmax over them alone"""
    idx = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    s = np.take_along_axis(z, idx, axis=-1)
    w = np.exp(s - s.max(axis=-1, keepdims=True))
    return idx, w / w.sum(axis=-1, keepdims=True)


def experts(h, T, c, book=None):
    idx, w = route(np.stack([h @ row for row in T["router"]], axis=-1), c["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(idx[t], w[t]):
            out[t] += wt * (T[f"e{e}.down"] @ (silu(T[f"e{e}.gate"] @ h[t]) * (T[f"e{e}.up"] @ h[t])))
    if book is not None:
        book["choices"], book["mix"] = idx, w
    return out


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, layer_outputs=None, book=None):
    """tensors: name -> float64 arrays.  Returns logits [n, vocab]; layer_outputs (a list) receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = tensors["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    for i, l in enumerate(cfg["layers"]):
        p = f"l{l.get('weights_of', i) if l.get('weights_of') is not None else i}."
        h, T, c = rms_norm(x, tensors[p + "norm1"], eps), sub(tensors, p + "mix."), l["mixer"]
        bk = None if book is None else book.setdefault(i, {})
        y = {"mlstm": lambda: mlstm(h, T, c, eps, bk), "parallel": lambda: parallel(h, T, c, eps, bk), "delta": lambda: delta(h, T, c, eps)}[l["type"]]()
        x = x + rms_norm(y, tensors[p + "norm1b"], eps)
        if l.get("mlp"):
            y = experts(rms_norm(x, tensors[p + "norm2"], eps), sub(tensors, p + "mlp."), l["mlp"], bk)
            x = x + rms_norm(y, tensors[p + "norm2b"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return rms_norm(x, tensors["final.norm"], eps) @ tensors["head"].T


def greedy(cfg, tensors, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(np.argmax(forward(cfg, tensors, toks)[-1])))
    return toks[len(prompt):]
