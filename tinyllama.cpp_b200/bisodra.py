"""Bisodra: reader of the family's config.json, its tensor inventory, synthetic weights.

A Bisodra model is a list of sandwich layers: x += norm1b(mixer(norm1(x))), then x += norm2b(ff(norm2(x))), all four norms layer norms
with a weight and no bias, over a scaled embedding that is also (unscaled) the output matrix; logits carry a constant factor.
config.json lists the layers; each names its mixer --
"attention": softmax attention with grouped K/V heads whose values ARE its keys; biased q and k projections, each followed by a short
causal convolution per channel; no rotation, a head-wise slope times the distance is taken off every score; a sliding window beside a
number of first tokens that stay visible; one more 1 in the softmax denominator; an element-wise sigmoid gate; a biased output projection;
"latent_attention": queries through a normed latent, keys and values up-projected from one normed latent per token plus one rotated key
part shared by the heads, YaRN-scaled rotary pairs (i, i + dims/2), causal, an element-wise sigmoid gate; with "kv_from" the latent and the
rotated key part are those of an earlier layer's cache --
and its feed-forward: down(gelu(up h)) with the erf form of GELU, or none.  This module turns config.json into the flat description the
native library takes (seq.SeqModel); every size and constant comes from the config."""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np

from . import safetensors_io as st
from .seq import BLOCK_SANDWICH, FF_GELU, MIX_LATENT_ATTN, MIX_SOFTMAX_ATTN, NORM_LAYER_NB, ROT_HALVES, ROT_SCALE_YARN

ARCHITECTURE = "Bisodra"
GATE_PER_ENTRY = 2
SINK_ONE = 2
# what a layer needs to share with the layer whose latents it reads
LATENT_CACHE_KEYS = ("kv_rank", "rope_dim", "rot_dims", "rot_base", "rot_layout", "rot_scaling", "rot_factor", "rot_low", "rot_high", "rot_original")


def _windowed(i: int, m: dict) -> dict:
    b = {"kind": MIX_SOFTMAX_ATTN, "name": "", "heads": int(m["heads"]), "kv_heads": int(m.get("kv_heads", m["heads"])), "dim": int(m["dim"]),
         "vdim": int(m.get("vdim", m["dim"])), "scale": float(m["scale"]), "kv_from": -1, "maps": 1, "bias": 1, "out_bias": 1, "conv": int(m.get("conv") or 0),
         "v_from_k": 1, "slopes": 1, "sink": SINK_ONE, "gated": GATE_PER_ENTRY}
    if b["heads"] % b["kv_heads"]:
        raise ValueError(f"layer {i}: {b['heads']} query heads do not divide into {b['kv_heads']} key/value heads")
    if b["vdim"] != b["dim"]:
        raise ValueError(f"layer {i}: the values are the keys, but vdim {b['vdim']} is not dim {b['dim']}")
    mask = m.get("mask")
    if mask:
        b["window"], b["keep_first"] = int(mask.get("size") or 0), int(mask.get("keep_first") or 0)
        if b["window"] < 0 or b["keep_first"] < 0 or (mask.get("size") is not None and b["window"] == 0):
            raise ValueError(f"layer {i}: a window of {mask.get('size')} tokens beside the first {mask.get('keep_first')}")
    return b


def _latent(i: int, m: dict) -> dict:
    b = {"kind": MIX_LATENT_ATTN, "name": "", "heads": int(m["heads"]), "dim": int(m["dim"]), "rope_dim": int(m["rot_dim"]), "vdim": int(m["vdim"]),
         "kv_rank": int(m["kv_rank"]), "q_rank": int(m["q_rank"]), "scale": float(m["scale"]), "gated": GATE_PER_ENTRY, "kv_from": -1}
    rot = m.get("rot")
    if rot and b["rope_dim"] > 0:
        b.update(rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), rot_layout=ROT_HALVES)
        if b["rot_dims"] > b["rope_dim"] or b["rot_dims"] % 2:
            raise ValueError(f"layer {i}: {b['rot_dims']} rotated entries do not fit a rotated part of {b['rope_dim']}")
        sc = rot.get("scaling")
        if sc:
            b.update(rot_scaling=ROT_SCALE_YARN, rot_factor=float(sc["factor"]), rot_original=float(sc["original"]), rot_high=float(sc["fast"]), rot_low=float(sc["slow"]))
            if min(b["rot_factor"], b["rot_original"], b["rot_high"], b["rot_low"]) <= 0.0 or b["rot_base"] <= 1.0:
                raise ValueError(f"layer {i}: frequency scaling {sc} over base {b['rot_base']}")
    if m.get("kv_from") is not None:
        b["kv_from"] = int(m["kv_from"])
        if not 0 <= b["kv_from"] < i:
            raise ValueError(f"layer {i}: kv_from {b['kv_from']} is not an earlier layer")
    return b


MIXERS = {"attention": _windowed, "latent_attention": _latent}


def describe(cfg: dict) -> dict:
    """config.json (parsed) -> description for seq.SeqModel."""
    if cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config: {cfg.get('architecture')!r}")
    d = {"vocab": int(cfg["vocab"]), "width": int(cfg["width"]), "eps": float(cfg["norm"]["eps"]), "final_norm": 4, "tied_head": 1,
         "embed_scale": float((cfg.get("embedding") or {}).get("scale", 1.0)), "logit_scale": float(cfg.get("logit_scale", 1.0)), "layers": []}
    if d["embed_scale"] == 0.0 or d["logit_scale"] == 0.0:
        raise ValueError(f"embedding scale {d['embed_scale']}, logit scale {d['logit_scale']}")
    for i, l in enumerate(cfg["layers"]):
        if l.get("type") not in MIXERS:
            raise ValueError(f"layer {i}: unknown type {l.get('type')!r}")
        lay = {"style": BLOCK_SANDWICH, "norm_kind": NORM_LAYER_NB, "branches": [MIXERS[l["type"]](i, l["mixer"])], "ff": 0}
        mlp = l.get("mlp")
        if mlp:
            if mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            lay.update(ff=int(mlp["ff"]), ff_kind=FF_GELU)
        d["layers"].append(lay)
    for i, lay in enumerate(d["layers"]):            # a shared cache must fit the layer that reads it
        b = lay["branches"][0]
        if b["kv_from"] >= 0:
            src = d["layers"][b["kv_from"]]["branches"][0]
            if src["kind"] != MIX_LATENT_ATTN or src["kv_from"] >= 0:
                raise ValueError(f"layer {i}: kv_from {b['kv_from']} is not a latent-attention layer with latents of its own")
            if any(src.get(k) != b.get(k) for k in LATENT_CACHE_KEYS):
                raise ValueError(f"layer {i}: latent size or rotation differ from those of layer {b['kv_from']}, whose cache it reads")
    return d


def tensor_shapes(desc: dict) -> dict:
    """name -> shape of every tensor of a checkpoint of this description (all bfloat16)."""
    W, out = desc["width"], {}
    out["embed"] = (desc["vocab"], W)
    for i, l in enumerate(desc["layers"]):
        p, b = f"l{i}.", l["branches"][0]
        mp = p + "mix."
        H, D, V = b["heads"], b["dim"], b["vdim"]
        if b["kind"] == MIX_LATENT_ATTN:
            hd = D + b["rope_dim"]
            out.update({mp + "dq": (b["q_rank"], W), mp + "dq.norm": (b["q_rank"],), mp + "uq": (H * hd, b["q_rank"])})
            if b["kv_from"] < 0:
                out.update({mp + "dkv": (b["kv_rank"] + b["rope_dim"], W), mp + "dkv.norm": (b["kv_rank"],)})
            out.update({mp + "uk": (H * D, b["kv_rank"]), mp + "uv": (H * V, b["kv_rank"]), mp + "g": (H * V, W), mp + "o": (W, H * V)})
        else:
            G = b["kv_heads"]
            out.update({mp + "q": (H * D, W), mp + "q.b": (H * D,), mp + "k": (G * D, W), mp + "k.b": (G * D,)})
            if b["conv"]:
                out.update({mp + "q.conv": (H * D, b["conv"]), mp + "k.conv": (G * D, b["conv"])})
            out.update({mp + "g": (H * V, W), mp + "o": (W, H * V), mp + "o.b": (W,)})
        for q in ("1", "1b") + (("2", "2b") if l["ff"] else ()):
            out[p + "norm" + q] = (W,)
        if l["ff"]:
            out.update({p + "mlp.up": (l["ff"], W), p + "mlp.down": (W, l["ff"])})
    out["final.norm"] = (W,)
    return out


def synth_tensors(desc: dict, seed: int = 0, gain: float = 1.0) -> dict:
    """Random weights (bfloat16 bit patterns): matrices ~ N(0, gain^2 / fan_in), norm weights around one, small biases, convolutions around
    a leading last tap, an embedding whose scaled rows have unit entries."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(desc).items():
        leaf = name.split(".")[-1]
        if leaf == "b":
            a = 0.2 * rng.standard_normal(shape)
        elif leaf.startswith("norm"):
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif leaf == "conv":
            a = 0.4 * rng.standard_normal(shape)
            a[:, -1] += 0.8
        elif name == "embed":
            a = rng.standard_normal(shape) / abs(desc["embed_scale"])
        else:
            a = rng.standard_normal(shape) * gain / np.sqrt(shape[-1])
        out[name] = st.f32_to_bf16_bits(np.asarray(a, np.float32))
    return out


def read_checkpoint(model_dir) -> tuple[dict, dict]:
    """(description, name -> bfloat16 bit patterns) of a folder with config.json and model.safetensors."""
    model_dir = Path(model_dir)
    desc = describe(json.loads((model_dir / "config.json").read_text()))
    return desc, st.read_as_bf16(model_dir / "model.safetensors", tensor_shapes(desc), ARCHITECTURE)


def write_checkpoint(model_dir, cfg: dict, tensors: dict) -> None:
    model_dir = Path(model_dir)
    model_dir.mkdir(parents=True, exist_ok=True)
    (model_dir / "config.json").write_text(json.dumps(cfg, indent=1))
    st.write(model_dir / "model.safetensors", {k: ("BF16", v) for k, v in tensors.items()})


def windowed_layer(heads=4, kv_heads=2, dim=16, conv=3, window=12, keep_first=5, scale=None, mlp=None) -> dict:
    """One "attention" entry of config["layers"]."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "scale": float(dim ** -0.5 if scale is None else scale)}
    if window:
        m["mask"] = {"size": window, "keep_first": keep_first}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent_layer(heads=3, dim=10, rot_dim=6, vdim=14, kv_rank=24, q_rank=20, rot_base=10000.0, yarn=(4.0, 32.0, 4.0, 1.0), scale=None, kv_from=None, mlp=None) -> dict:
    """One "latent_attention" entry; yarn: (factor, original, fast, slow) or None."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": float((dim + rot_dim) ** -0.5 if scale is None else scale),
         "rot": {"dims": rot_dim, "base": rot_base}}
    if yarn:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense_mlp(ff=40) -> dict:
    return {"kind": "dense", "ff": ff}


def make_config(vocab=96, width=48, layers=None, eps=1e-5, embed_scale=6.0, logit_scale=0.5) -> dict:
    """A config.json dictionary for tests, benchmarks and examples."""
    if layers is None:
        layers = [windowed_layer(mlp=dense_mlp()), latent_layer(mlp=dense_mlp(56)), windowed_layer(window=7, keep_first=2, conv=2), latent_layer(kv_from=1, heads=2, mlp=dense_mlp())]
    return {"architecture": ARCHITECTURE, "vocab": vocab, "width": width, "embedding": {"scale": embed_scale}, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}
