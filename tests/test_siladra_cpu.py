"""CPU-side pieces of the Siladra family: the config reader on every constant, on absent sections and on bad values, the tensor
inventory, the registry and checkpoint folder, and closed forms of the restatement's own building blocks (oracle/siladra_ref.py)."""
import math

import numpy as np
import pytest

from oracle import siladra_ref as R
from tinyllama_cpp_b200 import registry, seq
from tinyllama_cpp_b200 import siladra as SI


def test_describe_reads_every_constant():
    layers = [SI.parallel_layer(heads=6, kv_heads=3, dim=10, vdim=7, rot_dims=8, rot_base=777.0, yarn=(3.5, 99.0, 16.0, 2.0), scale=0.21, inner=44, state=9, dt_rank=4, conv=5, mlp=SI.moe_mlp(33, 7, 3)),
              SI.mlstm_layer(heads=3, dim=11, vdim=13, gate_cap=6.5), SI.delta_layer(heads=8, kv_heads=2, dim=9, vdim=15, conv=2, mlp=SI.moe_mlp(10, 4, 1))]
    layers += [SI.again(layers, 0), SI.again(layers, 2)]
    d = SI.describe(SI.make_config(vocab=70, width=36, layers=layers, eps=2e-4, embed_scale=5.5))
    assert (d["vocab"], d["width"], d["eps"], d["final_norm"], d["embed_scale"]) == (70, 36, 2e-4, 5, 5.5)
    assert all(l["style"] == seq.BLOCK_SANDWICH and l["norm_kind"] == seq.NORM_RMS for l in d["layers"])
    a, b = d["layers"][0]["branches"]
    assert (a["kind"], a["name"], a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], a["bias"], a["qk_norm"]) == (seq.MIX_SOFTMAX_ATTN, "left", 6, 3, 10, 7, 0.21, 1, 2)
    assert (a["rot_dims"], a["rot_base"], a["rot_layout"], a["rot_scaling"]) == (8, 777.0, seq.ROT_INTERLEAVED, seq.ROT_SCALE_YARN)
    assert (a["rot_factor"], a["rot_original"], a["rot_high"], a["rot_low"]) == (3.5, 99.0, 16.0, 2.0)
    assert (b["kind"], b["name"], b["inner"], b["state"], b["dt_rank"], b["conv"]) == (seq.MIX_SSM, "right", 44, 9, 4, 5)
    l0 = d["layers"][0]
    assert (l0["join_norm"], l0["ff"], l0["ff_kind"], l0["experts"], l0["top"], l0["route_kind"]) == (1, 33, seq.FF_GATED_EXPERTS, 7, 3, seq.ROUTE_SOFTMAX)
    m = d["layers"][1]["branches"][0]
    assert (m["kind"], m["heads"], m["dim"], m["vdim"], m["gate_cap"], m["scale"]) == (seq.MIX_MLSTM, 3, 11, 13, 6.5, 11 ** -0.5) and d["layers"][1]["ff"] == 0
    q = d["layers"][2]["branches"][0]
    assert (q["kind"], q["heads"], q["kv_heads"], q["dim"], q["vdim"], q["conv"], q["scale"]) == (seq.MIX_DELTA, 8, 2, 9, 15, 2, 9 ** -0.5)
    assert [l.get("weights_of") for l in d["layers"]] == [None, None, None, 0, 2]
    s = SI.tensor_shapes(d)
    assert not any(k.startswith(("l3.", "l4.")) for k in s) and s["head"] == (70, 36)
    assert s["l0.mix.left.q"] == (60, 36) and s["l0.mix.left.v.b"] == (21,) and s["l0.mix.left.k.norm"] == (10,) and s["l0.mix.left.out"] == (36,) and s["l0.mix.left.o"] == (36, 42)
    assert s["l0.mix.right.in"] == (88, 36) and s["l0.mix.right.x"] == (22, 44) and s["l0.mix.right.dt"] == (44, 4) and s["l0.mix.right.A_log"] == (44, 9) and s["l0.mix.right.conv"] == (44, 5)
    assert s["l1.mix.norm"] == (39,) and s["l1.mix.i.b"] == (3,) and "l1.norm2" not in s and s["l2.mix.norm"] == (15,) and s["l2.mix.v.conv"] == (120, 2) and s["l2.mix.k"] == (18, 36)
    assert s["l0.mlp.e6.down"] == (36, 33) and s["l2.mlp.router"] == (4, 36) and "l1.mlp.router" not in s and "l0.mix.out" not in s


def test_a_layer_run_a_third_time_names_the_layer_with_the_tensors():
    base = [SI.mlstm_layer(), SI.delta_layer()]
    layers = base + [SI.again(base, 0)]
    layers.append({**layers[2], "weights_of": 2})
    assert [l.get("weights_of") for l in SI.describe(SI.make_config(layers=layers))["layers"]] == [None, None, 0, 0]


def test_absent_sections_and_bad_values():
    c = SI.make_config(layers=[SI.parallel_layer(yarn=None), SI.parallel_layer(rot_dims=0)])
    del c["layers"][1]["mixer"]["left"]["rot"], c["layers"][1]["mixer"]["left"]["kv_heads"], c["embedding"]
    d = SI.describe(c)
    assert d["layers"][0]["branches"][0].get("rot_factor", 0.0) == 0.0 and d["layers"][0]["branches"][0]["rot_dims"] == 12 and d["embed_scale"] == 1.0
    assert d["layers"][1]["branches"][0].get("rot_dims", 0) == 0 and d["layers"][1]["branches"][0]["kv_heads"] == 4
    mix = lambda i: (lambda c: c["layers"][i]["mixer"])
    for bad in (lambda c: c.__setitem__("architecture", "Other"), lambda c: c["layers"][0].__setitem__("type", "delta_2"), lambda c: mix(0)(c).__setitem__("kv_heads", 3),
                lambda c: mix(0)(c).__setitem__("conv", 0), lambda c: mix(1)(c)["left"].__setitem__("kv_heads", 3), lambda c: mix(1)(c)["left"]["rot"].__setitem__("dims", 18),
                lambda c: mix(1)(c)["left"]["rot"].__setitem__("dims", 5), lambda c: mix(1)(c)["left"]["rot"]["scaling"].__setitem__("factor", 0), lambda c: mix(1)(c)["right"].__setitem__("state", 0),
                lambda c: mix(2)(c).__setitem__("gate_cap", 0.0), lambda c: c["layers"][0].__setitem__("mlp", {"kind": "dense"}), lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 9),
                lambda c: c["layers"][3].__setitem__("weights_of", 3), lambda c: c["layers"][3].__setitem__("weights_of", -1), lambda c: c["layers"][4].__setitem__("weights_of", 1),
                lambda c: c["embedding"].__setitem__("scale", 0.0)):
        import copy
        c2 = copy.deepcopy(SI.make_config())
        SI.describe(c2)
        bad(c2)
        with pytest.raises(ValueError):
            SI.describe(c2)


def test_registry_and_checkpoint_folder(tmp_path):
    cfg = SI.make_config()
    t = SI.synth_tensors(SI.describe(cfg), 1)
    SI.write_checkpoint(tmp_path / "m", cfg, t)
    assert registry.family_of(tmp_path / "m") == "Siladra" and "Siladra" in registry.STEPWISE
    desc, back = SI.read_checkpoint(tmp_path / "m")
    assert set(back) == set(SI.tensor_shapes(desc)) and all(np.array_equal(back[k], t[k]) for k in t)


def test_enumerators_follow_the_header():
    import re
    from pathlib import Path
    hdr = (Path(__file__).resolve().parent.parent / "include" / "gten_b200_seq.h").read_text()
    enums = dict(re.findall(r"(GTB_[A-Z0-9_]+) = (\d+)", hdr))
    for name in ("MIX_MLSTM", "MIX_DELTA", "MIX_SSM", "ROUTE_LOGISTIC", "ROUTE_SOFTMAX", "FF_GATED_EXPERTS"):
        assert int(enums["GTB_" + name]) == getattr(seq, name), name


# ------------------------------------------------------------------ the restatement's closed forms
def test_matrix_memory_is_a_weighted_sum_over_the_past():
    """With F_t the sum of log forget gates, o = sum_s e^(F_t - F_s + i_s) (q.k_s) v_s / max(|sum_s e^(..) q.k_s|, 1), whatever the running maximum."""
    rng = np.random.default_rng(0)
    T, D, V = 30, 5, 4
    q, k, v, i, f = rng.standard_normal((T, D)), rng.standard_normal((T, D)), rng.standard_normal((T, V)), rng.standard_normal(T) * 2, -rng.uniform(0, 2, T)
    F = np.cumsum(f)
    book = {}
    got = R.mlstm_scan(q, k, v, i, f, book)
    for t in range(T):
        w = np.exp(F[t] - F[:t + 1] + i[:t + 1]) * (k[:t + 1] @ q[t])
        assert np.allclose(got[t], w @ v[:t + 1] / max(abs(w.sum()), 1.0), rtol=1e-4, atol=1e-9)
    m = 0.0
    for t in range(T):
        m = max(f[t] + m, i[t])
        assert np.isclose(book["m"][t], m)
    assert np.allclose(R.soft_cap(np.array([-1e3, 0.0, 1e3]), 7.0), [-7.0, 0.0, 7.0]) and np.isclose(R.soft_cap(np.array([0.01]), 7.0)[0], 0.01, rtol=1e-5)


def test_delta_rule_overwrites_what_a_key_held():
    k = R.unit(np.random.default_rng(1).standard_normal((1, 6)))
    q = np.repeat(k, 3, 0)
    v = np.array([[1.0, 2.0], [5.0, -3.0], [0.5, 0.5]])
    one = R.delta_scan(q, q, v, np.ones(3), np.ones(3))
    assert np.allclose(one, v, atol=1e-5)                       # beta 1, no decay: the key now holds the new value
    half = R.delta_scan(q, q, v, np.full(3, 0.5), np.ones(3))
    assert np.allclose(half[1], 0.5 * (0.5 * v[0]) + 0.5 * v[1], atol=1e-5)
    decayed = R.delta_scan(q, q, v, np.array([1.0, 0.0, 0.0]), np.array([1.0, 0.25, 0.5]))
    assert np.allclose(decayed, [v[0], 0.25 * v[0], 0.125 * v[0]], atol=1e-5)
    assert np.allclose(np.linalg.norm(R.unit(np.random.default_rng(2).standard_normal((4, 9))), axis=-1), 1.0, atol=1e-6)


def test_delta_rule_in_chunks():
    """The triangular system of a chunk (unit lower, strictly lower part beta_t e^(b_t - b_s) k_t.k_s) reproduces the walk from any state."""
    rng = np.random.default_rng(3)
    T, D, V = 12, 5, 4
    q, k, v = rng.standard_normal((2 * T, D)), R.unit(rng.standard_normal((2 * T, D))), rng.standard_normal((2 * T, V))
    beta, g = rng.uniform(0, 1, 2 * T), rng.uniform(0.3, 1, 2 * T)
    want = R.delta_scan(q, k, v, beta, g)
    S, out = np.zeros((D, V)), []
    for c in (slice(0, T), slice(T, 2 * T)):
        b = np.cumsum(np.log(g[c]))
        w = np.tril(np.exp(b[:, None] - b[None, :]))
        A = np.tril(beta[c][:, None] * w * (k[c] @ k[c].T), -1)
        U = np.linalg.solve(np.eye(T) + A, beta[c][:, None] * (v[c] - np.exp(b)[:, None] * (k[c] @ S)))
        out.append(np.exp(b)[:, None] * (q[c] @ S) + (w * (q[c] @ k[c].T)) @ U)
        S = np.exp(b[-1]) * S + k[c].T @ (np.exp(b[-1] - b)[:, None] * U)
    assert np.allclose(np.concatenate(out), want)


def test_selective_scan_and_convolution():
    x, dt = np.ones((5, 1)), np.full((5, 1), 0.5)
    y = R.selective_scan(x, dt, np.array([[-2.0]]), np.full((5, 1), 3.0), np.full((5, 1), 0.25), np.array([10.0]))
    s = 0.0
    for t in range(5):
        s = math.exp(-1.0) * s + 1.5
        assert np.isclose(y[t, 0], 0.25 * s + 10.0)
    rng = np.random.default_rng(4)
    u, w = rng.standard_normal((9, 4)), rng.standard_normal((4, 3))
    c = R.causal_conv(u, w)
    for ch in range(4):
        assert np.allclose(c[:, ch], np.convolve(u[:, ch], w[ch, ::-1])[:9])
    assert np.allclose(R.causal_conv(u[:1], w), u[:1] * w[:, 2])


def test_router_norms_and_rotation():
    z = np.array([[1.0, 3.0, 3.0, -2.0], [0.0, 0.0, 0.0, 0.0]])
    idx, w = R.route(z, 3)
    assert idx.tolist() == [[1, 2, 0], [0, 1, 2]] and np.allclose(w[1], 1 / 3) and np.allclose(w[0], np.exp([0, 0, -2]) / (2 + math.exp(-2)))
    x = np.random.default_rng(5).standard_normal((5, 12)) * 3
    assert np.allclose((R.rms_norm(x, np.ones(12), 0.0) ** 2).mean(-1), 1.0) and np.allclose(R.softplus(np.array([-800.0, 0.0, 800.0])), [0.0, math.log(2.0), 800.0])
    f, amp = R.yarn(8, 100.0, {"factor": 4.0, "original": 64.0, "fast": 3.0, "slow": 0.6})
    assert np.isclose(amp, 1.0 + 0.1 * math.log(4.0)) and np.allclose(f, [100.0 ** (-i / 4) for i in range(4)] * np.array([1.0, 1.0, 0.625, 0.25]))
    v = np.random.default_rng(6).standard_normal((6, 2, 10))
    r = R.rotate(v, f, 1.5)
    assert np.allclose(r[..., 8:], v[..., 8:]) and np.allclose(r[0, :, :8], 1.5 * v[0, :, :8])
    assert np.allclose(np.hypot(r[..., 2], r[..., 3]), 1.5 * np.hypot(v[..., 2], v[..., 3])) and np.allclose(r[2, 0, 0], 1.5 * (v[2, 0, 0] * math.cos(2.0) - v[2, 0, 1] * math.sin(2.0)))
