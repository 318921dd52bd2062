"""Siladra: reader of the family's config.json, its tensor inventory, synthetic weights.

A Siladra model is a list of sandwich layers: x += norm1b(mixer(norm1(x))), then x += norm2b(ff(norm2(x))), all four norms RMS norms with
a plain weight, over a scaled embedding; the output matrix is a tensor of its own.  A layer with "weights_of": j is layer j once more --
the same tensors, a cache and state of its own.  config.json lists the layers; each names its mixer --
"mlstm": a matrix memory per head with capped exponential input gates and logistic forget gates under a running maximum, a normaliser,
a norm per head and a sigmoid gate;
"parallel": two mixers on the same input, "left" softmax attention with grouped K/V heads, biased and normed queries and keys and YaRN-scaled
rotary pairs (2i, 2i + 1), "right" a selective scan behind a short convolution; each output normed, the mean of the two;
"delta": the gated delta rule behind short convolutions with silu, unit-length queries and keys shared by groups of heads --
and its feed-forward: SiLU-gated experts, of which a token uses the `top` with the largest router outputs weighted by their own softmax,
or none.  This module turns config.json into the flat description the native library takes (seq.SeqModel); every size and constant
comes from the config."""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np

from . import safetensors_io as st
from .seq import (BLOCK_SANDWICH, FF_GATED_EXPERTS, MIX_DELTA, MIX_MLSTM, MIX_SOFTMAX_ATTN, MIX_SSM, NORM_RMS, ROT_INTERLEAVED, ROT_SCALE_YARN, ROUTE_SOFTMAX)

ARCHITECTURE = "Siladra"
QK_NORM_WEIGHTED = 2
FINAL_RMS = 5


def _grouped(i: int, heads: int, kv_heads: int) -> None:
    if kv_heads < 1 or heads % kv_heads:
        raise ValueError(f"layer {i}: {heads} heads do not divide into {kv_heads} key/value heads")


def _taps(i: int, m: dict) -> int:
    if int(m["conv"]) < 1:
        raise ValueError(f"layer {i}: a convolution of {m['conv']} taps")
    return int(m["conv"])


def _mlstm(i: int, m: dict) -> dict:
    b = {"kind": MIX_MLSTM, "name": "", "heads": int(m["heads"]), "dim": int(m["dim"]), "vdim": int(m["vdim"]), "gate_cap": float(m["gate_cap"])}
    if b["gate_cap"] <= 0.0:
        raise ValueError(f"layer {i}: gates capped at {b['gate_cap']}")
    b["scale"] = b["dim"] ** -0.5
    return b


def _delta(i: int, m: dict) -> dict:
    b = {"kind": MIX_DELTA, "name": "", "heads": int(m["heads"]), "kv_heads": int(m.get("kv_heads", m["heads"])), "dim": int(m["dim"]), "vdim": int(m["vdim"]), "conv": _taps(i, m)}
    _grouped(i, b["heads"], b["kv_heads"])
    b["scale"] = b["dim"] ** -0.5
    return b


def _attention(i: int, m: dict, name: str) -> dict:
    b = {"kind": MIX_SOFTMAX_ATTN, "name": name, "heads": int(m["heads"]), "kv_heads": int(m.get("kv_heads", m["heads"])), "dim": int(m["dim"]), "vdim": int(m["vdim"]),
         "scale": float(m["scale"]), "kv_from": -1, "maps": 1, "bias": 1, "qk_norm": QK_NORM_WEIGHTED}
    _grouped(i, b["heads"], b["kv_heads"])
    rot = m.get("rot")
    if rot and int(rot["dims"]) > 0:
        b.update(rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), rot_layout=ROT_INTERLEAVED)
        if b["rot_dims"] > b["dim"] or b["rot_dims"] % 2:
            raise ValueError(f"layer {i}: {b['rot_dims']} rotated entries do not fit heads of {b['dim']}")
        sc = rot.get("scaling")
        if sc:
            b.update(rot_scaling=ROT_SCALE_YARN, rot_factor=float(sc["factor"]), rot_original=float(sc["original"]), rot_high=float(sc["fast"]), rot_low=float(sc["slow"]))
            if min(b["rot_factor"], b["rot_original"], b["rot_high"], b["rot_low"]) <= 0.0 or b["rot_base"] <= 1.0:
                raise ValueError(f"layer {i}: frequency scaling {sc} over base {b['rot_base']}")
    return b


def _ssm(i: int, m: dict, name: str) -> dict:
    b = {"kind": MIX_SSM, "name": name, "inner": int(m["inner"]), "state": int(m["state"]), "dt_rank": int(m["dt_rank"]), "conv": _taps(i, m)}
    if min(b["inner"], b["state"], b["dt_rank"]) < 1:
        raise ValueError(f"layer {i}: a scan of {b['inner']} channels, {b['state']} states, step rank {b['dt_rank']}")
    return b


MIXERS = {"mlstm": lambda i, m: [_mlstm(i, m)], "delta": lambda i, m: [_delta(i, m)],
          "parallel": lambda i, m: [_attention(i, m["left"], "left"), _ssm(i, m["right"], "right")]}


def describe(cfg: dict) -> dict:
    """config.json (parsed) -> description for seq.SeqModel."""
    if cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config: {cfg.get('architecture')!r}")
    d = {"vocab": int(cfg["vocab"]), "width": int(cfg["width"]), "eps": float(cfg["norm"]["eps"]), "final_norm": FINAL_RMS,
         "embed_scale": float((cfg.get("embedding") or {}).get("scale", 1.0)), "layers": []}
    if d["embed_scale"] == 0.0:
        raise ValueError("an embedding scale of 0")
    for i, l in enumerate(cfg["layers"]):
        if l.get("type") not in MIXERS:
            raise ValueError(f"layer {i}: unknown type {l.get('type')!r}")
        lay = {"style": BLOCK_SANDWICH, "norm_kind": NORM_RMS, "branches": MIXERS[l["type"]](i, l["mixer"]), "ff": 0, "join_norm": int(l["type"] == "parallel")}
        mlp = l.get("mlp")
        if mlp:
            if mlp.get("kind") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            r = mlp["router"]
            lay.update(ff=int(mlp["expert"]["ff"]), ff_kind=FF_GATED_EXPERTS, experts=int(r["experts"]), top=int(r["top"]), route_kind=ROUTE_SOFTMAX)
            if not 1 <= lay["top"] <= min(lay["experts"], 64):
                raise ValueError(f"layer {i}: {lay['top']} of {lay['experts']} experts per token")
        if l.get("weights_of") is not None:
            j = int(l["weights_of"])
            if not 0 <= j < i:
                raise ValueError(f"layer {i}: weights_of {j} is not an earlier layer")
            j = d["layers"][j].get("weights_of", j)              # the layer that holds the tensors
            if {k: v for k, v in d["layers"][j].items() if k != "weights_of"} != lay:
                raise ValueError(f"layer {i} differs from layer {j}, whose weights it uses")
            lay["weights_of"] = j
        d["layers"].append(lay)
    return d


def tensor_shapes(desc: dict) -> dict:
    """name -> shape of every tensor of a checkpoint of this description (all bfloat16)."""
    W, out = desc["width"], {}
    out["embed"] = (desc["vocab"], W)
    for i, l in enumerate(desc["layers"]):
        if l.get("weights_of") is not None:
            continue
        p = f"l{i}."
        for b in l["branches"]:
            mp = p + "mix." + (b["name"] + "." if b["name"] else "")
            if b["kind"] == MIX_SSM:
                n, N, r = b["inner"], b["state"], b["dt_rank"]
                out.update({mp + "in": (2 * n, W), mp + "conv": (n, b["conv"]), mp + "conv.b": (n,), mp + "x": (r + 2 * N, n), mp + "dt": (n, r), mp + "dt.b": (n,),
                            mp + "A_log": (n, N), mp + "D": (n,), mp + "o": (W, n)})
            else:
                H, G, D, V = b["heads"], b.get("kv_heads", b["heads"]), b["dim"], b["vdim"]
                if b["kind"] == MIX_SOFTMAX_ATTN:
                    out.update({mp + "q": (H * D, W), mp + "q.b": (H * D,), mp + "k": (G * D, W), mp + "k.b": (G * D,), mp + "v": (G * V, W), mp + "v.b": (G * V,),
                                mp + "q.norm": (D,), mp + "k.norm": (D,)})
                elif b["kind"] == MIX_MLSTM:
                    out.update({mp + "q": (H * D, W), mp + "k": (H * D, W), mp + "v": (H * V, W), mp + "g": (H * V, W), mp + "i": (H, W), mp + "i.b": (H,), mp + "f": (H, W), mp + "f.b": (H,),
                                mp + "norm": (H * V,)})
                else:
                    for t, n in (("q", G * D), ("k", G * D), ("v", H * V)):
                        out.update({mp + t: (n, W), mp + t + ".conv": (n, b["conv"])})
                    out.update({mp + "g": (H * V, W), mp + "b": (H, W), mp + "a": (H, W), mp + "A_log": (H,), mp + "dt_bias": (H,), mp + "norm": (V,)})
                out[mp + "o"] = (W, H * V)
            if l["join_norm"]:
                out[mp + "out"] = (W,)
        for q in ("1", "1b") + (("2", "2b") if l["ff"] else ()):
            out[p + "norm" + q] = (W,)
        if l["ff"]:
            out[p + "mlp.router"] = (l["experts"], W)
            for e in range(l["experts"]):
                out.update({f"{p}mlp.e{e}.gate": (l["ff"], W), f"{p}mlp.e{e}.up": (l["ff"], W), f"{p}mlp.e{e}.down": (W, l["ff"])})
    out["final.norm"] = (W,)
    out["head"] = (desc["vocab"], W)
    return out


def synth_tensors(desc: dict, seed: int = 0, gain: float = 1.0) -> dict:
    """Random weights (bfloat16 bit patterns): matrices ~ N(0, gain^2 / fan_in), norm weights around one, small biases, convolutions around
    a leading last tap, an embedding whose scaled rows have unit entries; decays spread from a few to a few hundred tokens."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(desc).items():
        leaf = name.split(".")[-1]
        if leaf == "b" and len(shape) == 1:
            a = 0.2 * rng.standard_normal(shape)
            if name.endswith(".f.b"):
                a = rng.uniform(1.0, 5.0, shape)
            elif name.endswith(".dt.b"):
                a = rng.uniform(-4.5, -1.0, shape)
        elif leaf.startswith("norm") or leaf == "out":
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif leaf == "conv":
            a = 0.4 * rng.standard_normal(shape)
            a[:, -1] += 0.8
        elif leaf == "A_log":
            a = np.log(np.arange(1, shape[-1] + 1)) + 0.1 * rng.standard_normal(shape) if len(shape) == 2 else rng.uniform(-1.0, 1.5, shape)
        elif leaf == "dt_bias":
            a = rng.uniform(-5.0, -1.0, shape)
        elif leaf == "D":
            a = 1.0 + 0.2 * rng.standard_normal(shape)
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


# ------------------------------------------------------------------ entries of config["layers"]
def mlstm_layer(heads=3, dim=20, vdim=28, gate_cap=9.0, mlp=None) -> dict:
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}, "mlp": mlp}


def delta_layer(heads=4, kv_heads=2, dim=24, vdim=20, conv=3, mlp=None) -> dict:
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def parallel_layer(heads=4, kv_heads=2, dim=16, vdim=12, rot_dims=12, rot_base=500.0, yarn=(4.0, 64.0, 4.0, 1.0), scale=None, inner=40, state=6, dt_rank=5, conv=3, mlp=None) -> dict:
    """yarn: (factor, original, fast, slow) or None."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(dim ** -0.5 if scale is None else scale), "rot": {"dims": rot_dims, "base": rot_base}}
    if yarn:
        left["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "parallel", "mixer": {"left": left, "right": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}, "mlp": mlp}


def moe_mlp(ff=24, experts=5, top=2) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def again(layers, j: int) -> dict:
    """layer j once more"""
    return {**{k: v for k, v in layers[j].items() if k != "weights_of"}, "weights_of": j}


def make_config(vocab=96, width=48, layers=None, eps=1e-5, embed_scale=6.0) -> dict:
    """A config.json dictionary for tests, benchmarks and examples."""
    if layers is None:
        layers = [delta_layer(mlp=moe_mlp()), parallel_layer(mlp=moe_mlp(32, 6, 3)), mlstm_layer()]
        layers += [again(layers, 1), again(layers, 0)]
    return {"architecture": ARCHITECTURE, "vocab": vocab, "width": width, "embedding": {"scale": embed_scale}, "norm": {"eps": eps}, "layers": layers}
