"""CPU-side pieces of the Bisodra family: the config reader on every constant and on absent sections, the tensor inventory, the
registry and checkpoint folder, and closed forms of the restatement's own building blocks (oracle/bisodra_ref.py)."""
import math

import numpy as np
import pytest

from oracle import bisodra_ref as R
from tinyllama_cpp_b200 import bisodra as BI, registry, seq


def test_describe_reads_every_constant():
    layers = [BI.latent_layer(heads=5, dim=9, rot_dim=4, vdim=11, kv_rank=30, q_rank=14, rot_base=777.0, yarn=(3.5, 99.0, 16.0, 2.0), scale=0.21, mlp=BI.dense_mlp(44)),
              BI.windowed_layer(heads=6, kv_heads=3, dim=10, conv=5, window=19, keep_first=7, scale=0.3),
              BI.latent_layer(heads=2, dim=6, rot_dim=4, vdim=8, kv_rank=30, q_rank=10, rot_base=777.0, yarn=(3.5, 99.0, 16.0, 2.0), scale=0.4, kv_from=0)]
    d = BI.describe(BI.make_config(vocab=70, width=36, layers=layers, eps=2e-4, embed_scale=5.5, logit_scale=0.3))
    assert (d["vocab"], d["width"], d["eps"], d["final_norm"], d["tied_head"], d["embed_scale"], d["logit_scale"]) == (70, 36, 2e-4, 4, 1, 5.5, 0.3)
    assert all(l["style"] == seq.BLOCK_SANDWICH and l["norm_kind"] == seq.NORM_LAYER_NB for l in d["layers"])
    a = d["layers"][0]["branches"][0]
    assert (a["kind"], a["heads"], a["dim"], a["rope_dim"], a["vdim"], a["kv_rank"], a["q_rank"], a["scale"], a["gated"], a["kv_from"]) == (seq.MIX_LATENT_ATTN, 5, 9, 4, 11, 30, 14, 0.21, 2, -1)
    assert (a["rot_dims"], a["rot_base"], a["rot_layout"], a["rot_scaling"]) == (4, 777.0, seq.ROT_HALVES, seq.ROT_SCALE_YARN)
    assert (a["rot_factor"], a["rot_original"], a["rot_high"], a["rot_low"]) == (3.5, 99.0, 16.0, 2.0)
    assert (d["layers"][0]["ff"], d["layers"][0]["ff_kind"]) == (44, seq.FF_GELU) and d["layers"][1]["ff"] == 0
    b = d["layers"][1]["branches"][0]
    assert (b["kind"], b["heads"], b["kv_heads"], b["dim"], b["vdim"], b["scale"]) == (seq.MIX_SOFTMAX_ATTN, 6, 3, 10, 10, 0.3)
    assert (b["conv"], b["window"], b["keep_first"], b["v_from_k"], b["slopes"], b["sink"], b["bias"], b["out_bias"], b["gated"]) == (5, 19, 7, 1, 1, 2, 1, 1, 2)
    assert d["layers"][2]["branches"][0]["kv_from"] == 0
    s = BI.tensor_shapes(d)
    assert s["l1.mix.q.conv"] == (60, 5) and s["l1.mix.k.conv"] == (30, 5) and s["l1.mix.g"] == (60, 36) and s["l1.mix.o.b"] == (36,) and "l1.mix.v" not in s
    assert s["l0.mix.dkv"] == (34, 36) and s["l0.mix.uq"] == (65, 14) and s["l0.mix.g"] == (55, 36) and s["l0.mlp.up"] == (44, 36)
    assert "l2.mix.dkv" not in s and "l2.mix.dkv.norm" not in s and s["l2.mix.uk"] == (12, 30) and "head" not in s and "final.norm.b" not in s
    assert "l1.norm2" not in s and s["l0.norm2b"] == (36,)


def test_absent_sections_and_bad_values():
    d = BI.describe(BI.make_config(layers=[BI.windowed_layer(conv=0, window=0), BI.latent_layer(yarn=None)]))
    a, b = (l["branches"][0] for l in d["layers"])
    assert a.get("window", 0) == 0 and a.get("keep_first", 0) == 0 and a["conv"] == 0 and "l0.mix.q.conv" not in BI.tensor_shapes(d)
    assert b.get("rot_factor", 0.0) == 0.0 and b["rot_dims"] == 6
    mix = lambda i: (lambda c: c["layers"][i]["mixer"])
    for bad in (lambda c: mix(1)(c).__setitem__("kv_from", 1), lambda c: c["layers"][0].__setitem__("type", "attention_3"), lambda c: mix(0)(c).__setitem__("kv_heads", 3),
                lambda c: mix(0)(c).__setitem__("vdim", 8), lambda c: mix(0)(c)["mask"].__setitem__("size", 0), lambda c: mix(0)(c)["mask"].__setitem__("keep_first", -1),
                lambda c: mix(1)(c)["rot"].__setitem__("dims", 8), lambda c: mix(1)(c)["rot"]["scaling"].__setitem__("factor", 0), lambda c: c.__setitem__("architecture", "Other"),
                lambda c: c["layers"][0].__setitem__("mlp", {"kind": "moe"}), lambda c: mix(3)(c).__setitem__("kv_from", 0), lambda c: mix(3)(c).__setitem__("kv_rank", 23),
                lambda c: mix(3)(c)["rot"].__setitem__("base", 5.0), lambda c: c.__setitem__("logit_scale", 0.0)):
        c2 = BI.make_config()
        BI.describe(c2)
        bad(c2)
        with pytest.raises(ValueError):
            BI.describe(c2)


def test_registry_and_checkpoint_folder(tmp_path):
    cfg = BI.make_config()
    t = BI.synth_tensors(BI.describe(cfg), 1)
    BI.write_checkpoint(tmp_path / "m", cfg, t)
    assert registry.family_of(tmp_path / "m") == "Bisodra" and "Bisodra" in registry.STEPWISE
    desc, back = BI.read_checkpoint(tmp_path / "m")
    assert set(back) == set(BI.tensor_shapes(desc)) and all(np.array_equal(back[k], t[k]) for k in t)


def test_enumerators_follow_the_header():
    import re
    from pathlib import Path
    hdr = (Path(__file__).resolve().parent.parent / "include" / "gten_b200_seq.h").read_text()
    enums = dict(re.findall(r"(GTB_[A-Z0-9_]+) = (\d+)", hdr))
    for name, value in (("NORM_LAYER_NB", seq.NORM_LAYER_NB), ("FF_GELU", seq.FF_GELU), ("ROT_SCALE_WAVES", seq.ROT_SCALE_WAVES), ("ROT_SCALE_YARN", seq.ROT_SCALE_YARN)):
        assert int(enums["GTB_" + name]) == value, name

    def fields(struct):                       # names in the header's order
        body = re.search(r"typedef struct \{((?:(?!typedef struct).)*?)\} %s;" % struct, hdr, re.S).group(1)
        body = re.sub(r"/\*.*?\*/", "", body, flags=re.S)
        return [re.sub(r"\[.*?\]|\*", "", n).strip().split()[-1] for decl in body.split(";") if decl.strip() for n in decl.split(",")]
    assert fields("gtb_seq_branch") == [f[0] for f in seq.BranchC._fields_]
    assert fields("gtb_seq_layer") == [f[0] for f in seq.LayerC._fields_]
    assert fields("gtb_seq_config") == [f[0] for f in seq.ConfigC._fields_]


# ------------------------------------------------------------------ the restatement's closed forms
def test_norms_and_gelu():
    rng = np.random.default_rng(0)
    x = rng.standard_normal((5, 12)) * 3 + 2
    y = R.layer_norm(x, np.ones(12), 0.0)
    assert np.allclose(y.mean(-1), 0.0) and np.allclose((y * y).mean(-1), 1.0) and np.allclose(R.layer_norm(x + 7.0, np.ones(12), 0.0), y)
    assert np.allclose((R.rms_norm(x, np.ones(12), 0.0) ** 2).mean(-1), 1.0)
    z = np.linspace(-5, 5, 41)
    assert np.allclose(R.gelu(z) - R.gelu(-z), z) and np.isclose(R.gelu(np.array([1.0]))[0], 0.8413447460685429)


def test_gelu_of_the_product_epilogue():
    """The polynomial of the tensor-core epilogue, with the constants of its source, in float32 against the error function."""
    import re
    from pathlib import Path
    src = (Path(__file__).resolve().parent.parent / "tinyllama.cpp_b200" / "csrc" / "gtb_seq_gemm.cu").read_text()
    body = re.search(r"float sq_gelu_erf\(float z\) \{(.*?)\n\}", src, re.S).group(1)
    root, p, a5, a4, a3, a2, a1 = (np.float32(x) for x in re.findall(r"(-?0\.7071\d+|-?\d\.\d{6,})f", body)[:7])
    z = np.linspace(-8, 8, 20001).astype(np.float32)
    x = np.abs(z) * root
    t = np.float32(1) / (p * x + np.float32(1))
    q = ((((a5 * t + a4) * t + a3) * t + a2) * t + a1) * t * np.exp(-x * x)
    got = np.float32(0.5) * z * np.where(z < 0, q, np.float32(2) - q)
    err = np.abs(got - R.gelu(z.astype(np.float64)))
    assert err.max() < 1e-6 and np.abs(q - [math.erfc(v) for v in x.astype(np.float64)]).max() < 5e-7


def test_convolution_is_causal_and_linear():
    rng = np.random.default_rng(1)
    u, w = rng.standard_normal((9, 4)), rng.standard_normal((4, 3))
    y = R.causal_conv(u, w)
    assert np.allclose(y[0], w[:, 2] * u[0]) and np.allclose(y[1], w[:, 2] * u[1] + w[:, 1] * u[0])
    for c in range(4):
        assert np.allclose(y[:, c], np.convolve(u[:, c], w[c, ::-1])[:9])
    v = u.copy()
    v[6] += 1.0
    assert np.allclose(R.causal_conv(v, w)[:6], y[:6]) and not np.allclose(R.causal_conv(v, w)[6:9], y[6:9])
    assert np.allclose(R.causal_conv(u, w[:, 2:]), u * w[:, 2])


def test_visibility_slopes_and_softmax():
    see = lambda i, size, keep: [j for j in range(12) if R.visible(i, j, size, keep)]
    assert see(8, 3, 2) == [0, 1, 6, 7, 8] and see(8, 3, 0) == [6, 7, 8] and see(1, 3, 5) == [0, 1] and see(4, 0, 0) == [0, 1, 2, 3, 4] and see(7, 4, 6) == list(range(8))
    assert np.allclose(R.slopes(8), [2.0 ** -(h + 1) for h in range(8)]) and np.allclose(R.slopes(1), [2.0 ** -8]) and np.isclose(R.slopes(3)[0], 2.0 ** (-8 / 3))
    rng = np.random.default_rng(2)
    s = rng.standard_normal((4, 4))
    mask = np.tril(np.ones((4, 4), bool))
    assert np.allclose(R.masked_softmax(s, mask, 0.0).sum(-1), 1.0)
    w = R.masked_softmax(s, mask, 1.0)
    assert np.isclose(w[0, 0], np.exp(s[0, 0]) / (1 + np.exp(s[0, 0]))) and np.isclose(w[3].sum(), np.exp(s[3]).sum() / (1 + np.exp(s[3]).sum())) and w[0, 1] == 0.0


def test_yarn_frequencies():
    f, amp = R.yarn(8, 100.0, None)
    assert amp == 1.0 and np.allclose(f, [100.0 ** (-i / 4) for i in range(4)])
    # at(turns) = 8 ln(64 / (2 pi turns)) / (2 ln 100): 1.01 for 3 turns, 2.41 for 0.6 -> the ramp runs from pair 1 to pair 3
    g, amp = R.yarn(8, 100.0, {"factor": 4.0, "original": 64.0, "fast": 3.0, "slow": 0.6})
    assert np.isclose(amp, 1.0 + 0.1 * math.log(4.0))
    assert np.allclose(g, f * [1.0, 1.0, 0.5 + 0.125, 0.25])
    low, _ = R.yarn(8, 100.0, {"factor": 4.0, "original": 1.0, "fast": 32.0, "slow": 1.0})         # every wavelength is long: pair 0 starts the ramp
    assert np.isclose(low[0], f[0]) and np.allclose(low[1:], f[1:] / 4.0)
    v = np.random.default_rng(3).standard_normal((6, 2, 10))
    r = R.rotate(v, g, 1.5)
    assert np.allclose(r[..., 8:], v[..., 8:]) and np.allclose(r[0, :, :8], 1.5 * v[0, :, :8])
    assert np.allclose(np.hypot(r[..., 1], r[..., 5]), 1.5 * np.hypot(v[..., 1], v[..., 5]))


def test_shared_latents_and_absorbed_scores():
    """Scores through the up-projected keys equal those of the query carried through the up-projection, over the latents themselves."""
    rng = np.random.default_rng(4)
    m = BI.latent_layer(heads=2, dim=5, rot_dim=4, vdim=6, kv_rank=7, q_rank=8)["mixer"]
    Wd = 10
    T = {"dq": rng.standard_normal((8, Wd)), "dq.norm": np.ones(8), "uq": rng.standard_normal((18, 8)), "dkv": rng.standard_normal((11, Wd)), "dkv.norm": np.ones(7),
         "uk": rng.standard_normal((10, 7)), "uv": rng.standard_normal((12, 7)), "g": np.zeros((12, Wd)), "o": np.eye(12)}
    h = rng.standard_normal((6, Wd))
    c, kr = R.latent_of(h, T, m, 1e-6)
    got = R.latent_attention(h, T, m, 1e-6, (c, kr)).reshape(6, 2, 6)
    q = (R.rms_norm(h @ T["dq"].T, 1.0, 1e-6) @ T["uq"].T).reshape(6, 2, 9)
    qr = R.rotate(q[..., 5:], *R.yarn(4, 10000.0, m["rot"]["scaling"]))
    for a in range(2):
        s = (q[:, a, :5] @ T["uk"][5 * a:5 * a + 5] @ c.T + qr[:, a] @ kr.T) * m["scale"]
        w = R.masked_softmax(s, np.tril(np.ones((6, 6), bool)), 0.0)
        assert np.allclose(got[:, a], 0.5 * (w @ c) @ T["uv"][6 * a:6 * a + 6].T)
