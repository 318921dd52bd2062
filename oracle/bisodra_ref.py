"""Plain restatement of the Bisodra family in numpy float64: one function per mechanism, whole sequences only, no cache, no step
function, nothing shared with the product path.  Tests compare the native library against it.

A Bisodra layer wraps each sublayer in two bias-free layer norms: x += ln_b(mixer(ln_a(x))), then the same around the feed-forward.
Mixers: "attention" (grouped K/V heads whose keys double as values; q and k pass a short causal convolution per channel right behind
their biased projections; no rotation -- a head-wise slope times the distance is taken off every score; a sliding window beside a
number of first tokens that stay visible; one more 1 in the softmax denominator; an element-wise sigmoid gate; an output projection
with a bias) and "latent_attention" (queries through a normed latent, keys and values up-projected from one normed latent per token
plus one rotated key part shared by the heads, rotary frequencies blended by YaRN, causal softmax, the same kind of gate; the latent
and the rotated part may be an earlier layer's).  Feed-forward: down(gelu(up h)) with the erf form of GELU, or none.  The embedding
is scaled on the way in and, unscaled, is the output matrix; logits carry a constant factor."""
from __future__ import annotations

import math

import numpy as np


def to_float(bits):
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def layer_norm(x, w, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def logistic(z):
    return 1.0 / (1.0 + np.exp(-z))


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def causal_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros in front of the sequence"""
    taps = w.shape[1]
    y = np.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def visible(i, j, size, keep):
    """does position i see key j: causal, within the last `size` positions or among the first `keep`; size 0: all earlier ones"""
    return j <= i and (size <= 0 or i - j < size or j < keep)


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def masked_softmax(scores, mask, extra):
    """rows of softmax weights over the visible keys; extra: a constant added to the denominator (in units of exp(score))"""
    w = np.zeros_like(scores)
    for i in range(scores.shape[0]):
        on = mask[i]
        top = scores[i, on].max()
        if extra > 0.0:
            top = max(top, 0.0)
        e = np.exp(scores[i, on] - top)
        w[i, on] = e / (e.sum() + extra * np.exp(-top))
    return w


def windowed_attention(h, T, m, book=None):
    """mixer "attention" """
    n = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    size, keep = int((m.get("mask") or {}).get("size") or 0), int((m.get("mask") or {}).get("keep_first") or 0)
    q, k = h @ T["q"].T + T["q.b"], h @ T["k"].T + T["k.b"]
    if m.get("conv"):
        q, k = causal_conv(q, T["q.conv"]), causal_conv(k, T["k.conv"])
    q, k = q.reshape(n, H, D), k.reshape(n, G, D)
    mask = np.array([[visible(i, j, size, keep) for j in range(n)] for i in range(n)])
    dist = np.subtract.outer(np.arange(n), np.arange(n)).astype(np.float64)
    out = np.zeros((n, H, D))
    for a in range(H):
        g = a // (H // G)
        w = masked_softmax(q[:, a] @ k[:, g].T * m["scale"] - slopes(H)[a] * dist, mask, 1.0)
        out[:, a] = w @ k[:, g]
        if book is not None:
            book.setdefault("weights", {})[a] = w
    o = out.reshape(n, H * D) * logistic(h @ T["g"].T)
    return o @ T["o"].T + T["o.b"]


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
    """v [T, ..., n]: entries (i, i + len(freqs)) of the last axis turn by t * freqs[i] and are scaled by amp; later entries stay"""
    out = np.array(v, np.float64)
    half = len(freqs)
    pos = np.arange(v.shape[0], dtype=np.float64).reshape((-1,) + (1,) * (v.ndim - 2))
    for i in range(half):
        c, s = np.cos(pos * freqs[i]) * amp, np.sin(pos * freqs[i]) * amp
        out[..., i] = v[..., i] * c - v[..., i + half] * s
        out[..., i + half] = v[..., i + half] * c + v[..., i] * s
    return out


def latent_of(h, T, m, eps):
    """what a layer with a down-projection of its own leaves for itself and later layers: (latent [n, rank], rotated key part [n, rot])"""
    z = h @ T["dkv"].T
    rot = m.get("rot")
    part = z[:, m["kv_rank"]:]
    if rot and rot.get("dims"):
        part = rotate(part, *yarn(int(rot["dims"]), rot["base"], rot.get("scaling")))
    return rms_norm(z[:, :m["kv_rank"]], T["dkv.norm"], eps), part


def latent_attention(h, T, m, eps, kv, book=None):
    """mixer "latent_attention" over a given (latent, rotated key part)"""
    n = h.shape[0]
    H, D, Dr, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = kv
    q = (rms_norm(h @ T["dq"].T, T["dq.norm"], eps) @ T["uq"].T).reshape(n, H, D + Dr)
    rot = m.get("rot")
    qr = q[..., D:]
    if rot and rot.get("dims"):
        qr = rotate(qr, *yarn(int(rot["dims"]), rot["base"], rot.get("scaling")))
    k, v = (c @ T["uk"].T).reshape(n, H, D), (c @ T["uv"].T).reshape(n, H, V)
    mask = np.array([[j <= i for j in range(n)] for i in range(n)])
    out = np.zeros((n, H, V))
    for a in range(H):
        w = masked_softmax((q[:, a, :D] @ k[:, a].T + qr[:, a] @ kr.T) * m["scale"], mask, 0.0)
        out[:, a] = w @ v[:, a]
        if book is not None:
            book.setdefault("weights", {})[a] = w
    return out.reshape(n, H * V) * logistic(h @ T["g"].T) @ T["o"].T


def dense_ff(h, T):
    return gelu(h @ T["up"].T) @ T["down"].T


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, layer_outputs=None, book=None):
    """tensors: name -> float64 arrays.  Returns logits [n, vocab]; layer_outputs (a list) receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = tensors["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    kept = {}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        h = layer_norm(x, tensors[p + "norm1"], eps)
        T = sub(tensors, p + "mix.")
        bk = None if book is None else book.setdefault(i, {})
        if l["type"] == "attention":
            y = windowed_attention(h, T, m, bk)
        elif l["type"] == "latent_attention":
            src = i if m.get("kv_from") is None else int(m["kv_from"])
            if src == i:
                kept[i] = latent_of(h, T, m, eps)
            y = latent_attention(h, T, m, eps, kept[src], bk)
        else:
            raise ValueError(l["type"])
        x = x + layer_norm(y, tensors[p + "norm1b"], eps)
        if l.get("mlp"):
            y = dense_ff(layer_norm(x, tensors[p + "norm2"], eps), sub(tensors, p + "mlp."))
            x = x + layer_norm(y, tensors[p + "norm2b"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return layer_norm(x, tensors["final.norm"], eps) @ tensors["embed"].T * float(cfg["logit_scale"])


def greedy(cfg, tensors, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(np.argmax(forward(cfg, tensors, toks)[-1])))
    return toks[len(prompt):]
