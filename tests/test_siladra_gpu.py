"""The Siladra family on the layer-list library (libgten_b200_seq.so) against the plain numpy restatement in oracle/siladra_ref.py.

Every test makes its own small configuration and random weights.  float32 mode is held to rounding (1e-4 of the logits' spread);
bfloat16 mode to a loose bound that a wrong key, a lost state or a chunk's edge still breaks by orders of magnitude.  Where random
weights would hide a fault (one far token among hundreds, a floor in a denominator, the start of a running maximum) the test plants it:
one input channel marks a token, a gate or a key reads that channel, and the restatement confirms that it decides the answer."""
import json

import numpy as np
import pytest

pytestmark = pytest.mark.gpu

from oracle import siladra_ref as R  # noqa: E402
from tinyllama_cpp_b200 import safetensors_io as st  # noqa: E402
from tinyllama_cpp_b200 import siladra as SI  # noqa: E402


@pytest.fixture(scope="module")
def lib():
    from tinyllama_cpp_b200 import build, seq
    build.build(target="seq")
    seq.init(0)
    return seq


def make(lib, cfg, mode="float32", seed=0, n_slots=3, max_ctx=512, max_rows=0, tweak=None, **synth):
    desc = SI.describe(cfg)
    t = SI.synth_tensors(desc, seed, **synth)
    if tweak:
        tweak(t)
    m = lib.SeqModel(desc, lib.MODE_BY_NAME[mode], n_slots, max_ctx, max_rows).load(t)
    return m, {k: R.to_float(v) for k, v in t.items()}


def rows_rel(got, want):
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())


def rel(got, want):
    """Largest row: rms of the difference after removing each row's mean, over the rms spread of the expected rows."""
    return float(rows_rel(got, want).max())


TOL = {"float32": 1e-4, "bfloat16": 6e-2}
MODES = ["float32", "bfloat16"]


def close(got, want, mode, frac=0.85):
    """Within TOL on every row in float32.  In bfloat16 a few rows are ill-conditioned: a head whose read-out nearly cancels is scaled to unit RMS all the
    same, and a close choice between two experts may flip (and colours the rows after it).  There most rows (`frac`) are held to TOL, the median to half
    of it, and the rest to being of the logits' own size; a lost state or a wrong edge breaks most rows."""
    if mode == "float32":
        return rel(got, want) < TOL[mode]
    rows = rows_rel(got, want)
    return float(np.mean(rows < TOL[mode])) >= frac and float(np.median(rows)) < 0.5 * TOL[mode] and float(rows.max()) < 2.0


def toks(seed, n, vocab, lo=0):
    return np.random.default_rng(3000 + seed).integers(lo, vocab, n).astype(np.int32)


def put(t, name, fn):
    a = st.bf16_bits_to_f32(t[name]).astype(np.float64)
    fn(a)
    t[name] = st.f32_to_bf16_bits(a.astype(np.float32))


ML, PA, DE, E = SI.mlstm_layer, SI.parallel_layer, SI.delta_layer, SI.moe_mlp

# ------------------------------------------------------------------ each mechanism alone
VARIANTS = {
    "mlstm": [ML()],
    "mlstm_one_head": [ML(heads=1, dim=33, vdim=17)],
    "mlstm_odd_sizes": [ML(heads=5, dim=7, vdim=3)],
    "mlstm_wide_values": [ML(heads=2, dim=16, vdim=150)],
    "mlstm_tight_cap": [ML(gate_cap=0.7)],
    "mlstm_chunks_of_32": [ML(heads=2, dim=170, vdim=40)],
    "mlstm_beyond_the_chunk_kernels": [ML(heads=1, dim=300, vdim=24)],
    "delta": [DE()],
    "delta_one_query_head": [DE(heads=6, kv_heads=1, dim=10, vdim=9)],
    "delta_all_own_heads": [DE(heads=3, kv_heads=3, dim=40, vdim=33)],
    "delta_one_tap": [DE(conv=1)],
    "delta_two_taps": [DE(conv=2)],
    "delta_four_taps": [DE(conv=4, heads=2, kv_heads=1, dim=64, vdim=64)],
    "delta_seven_taps": [DE(conv=7)],
    "delta_chunks_of_32": [DE(heads=2, kv_heads=1, dim=136, vdim=48)],
    "delta_wide_values": [DE(heads=2, kv_heads=2, dim=20, vdim=300)],
    "delta_beyond_the_chunk_kernels": [DE(heads=2, kv_heads=1, dim=260, vdim=20)],
    "parallel": [PA()],
    "parallel_one_kv_head": [PA(heads=5, kv_heads=1, dim=8, vdim=20, rot_dims=8)],
    "parallel_all_own_keys": [PA(heads=3, kv_heads=3, dim=12, vdim=7, rot_dims=4)],
    "parallel_plain_rotation": [PA(yarn=None)],
    "parallel_no_rotation": [PA(rot_dims=0)],
    "parallel_every_frequency_divided": [PA(rot_dims=16, yarn=(4.0, 6.0, 32.0, 2.0), scale=0.9)],
    "parallel_no_frequency_divided": [PA(rot_dims=16, yarn=(4.0, 1e6, 2.0, 1.0), scale=0.9)],
    "parallel_factor_one": [PA(yarn=(1.0, 32.0, 4.0, 1.0))],
    "scan_one_state": [PA(state=1, inner=30, dt_rank=1)],
    "scan_seven_states_one_tap": [PA(state=7, inner=37, dt_rank=9, conv=1)],
    "scan_16_states": [PA(state=16, inner=80, dt_rank=70, conv=4)],
    "scan_33_states": [PA(state=33, inner=24, dt_rank=2, conv=6)],
    "scan_100_states": [PA(state=100, inner=19, dt_rank=3, conv=2)],
    "scan_200_states": [PA(state=200, inner=10, dt_rank=4)],
    "experts": [ML(mlp=E())],
    "experts_top_1": [DE(mlp=E(ff=40, experts=4, top=1))],
    "experts_all": [ML(mlp=E(ff=17, experts=3, top=3))],
    "experts_one": [ML(mlp=E(ff=32, experts=1, top=1))],
    "experts_40_of_45": [ML(mlp=E(ff=8, experts=45, top=40))],
    "all": None,
}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("variant", list(VARIANTS))
def test_mechanisms_one_at_a_time(lib, mode, variant):
    cfg = SI.make_config(vocab=101, width=72, layers=VARIANTS[variant])
    m, W = make(lib, cfg, mode, seed=3)
    m.set_option("capture", 1)
    t = toks(1, 140, cfg["vocab"])
    trace = []
    want = R.forward(cfg, W, t, trace)
    got = m.step([(0, t)], range(len(t)))
    assert m.n_runs == len(trace)
    if mode == "float32" or not any(l.get("mlp") for l in cfg["layers"]):
        for u in range(m.n_runs):                # the stream after every layer
            for r in (0, 20, 63, 64, len(t) - 1):
                assert rel(m.read_capture(u, r)[None], trace[u][r][None]) < TOL[mode], (u, r)
    assert close(got, want, mode)
    one = np.concatenate([m.step([(1, t[i:i + 1])], [0]) for i in range(40)])
    assert close(one, want[:40], mode)


def test_embedding_scale_and_output_matrix(lib):
    for width, scale in ((64, 0.25), (56, 12.0)):
        cfg = SI.make_config(vocab=70, width=width, layers=[ML(), DE()], embed_scale=scale)
        for mode in MODES:
            m, W = make(lib, cfg, mode, seed=4)
            t = toks(9, 70, 70)
            want = R.forward(cfg, W, t)
            assert np.abs(m.step([(0, t)], range(70)) - want).max() < 6 * TOL[mode] * want.std(), (mode, width)


@pytest.mark.parametrize("width", [40, 42, 1100, 2100])
def test_joined_branches_at_every_width(lib, width):
    """The residual update that joins two branches: rows in registers (one and two groups of values a thread, and more), and rows that are walked."""
    cfg = SI.make_config(vocab=40, width=width, layers=[PA(mlp=E(ff=8, experts=3, top=1) if width == 40 else None), PA(heads=1, kv_heads=1, inner=24, dt_rank=3)])
    for mode in MODES:
        m, W = make(lib, cfg, mode, seed=5)
        t = toks(7, 70, 40)
        want = R.forward(cfg, W, t)
        assert close(m.step([(0, t)], range(70)), want, mode)
        got = np.concatenate([m.step([(1, t[i:i + 1])], [0]) for i in range(12)])
        assert close(got, want[:12], mode)
    other = {k: v for k, v in W.items()}
    other["l0.mix.left.out"], other["l0.mix.right.out"] = W["l0.mix.right.out"], W["l0.mix.left.out"]
    assert rel(R.forward(cfg, other, t), want) > 20 * TOL["float32"]


# ------------------------------------------------------------------ prefill = decode = portions
BOTH = [DE(conv=4, mlp=E()), PA(mlp=E(32, 6, 3)), ML(mlp=E(20, 4, 1)), DE(heads=3, kv_heads=1, dim=18, vdim=40, conv=6), PA(heads=2, kv_heads=1, state=20, conv=5)]
NO_FF = [DE(conv=4), PA(), ML(), DE(heads=3, kv_heads=1, dim=18, vdim=40, conv=6), PA(heads=2, kv_heads=1, state=20, conv=5)]


@pytest.mark.parametrize("mode", MODES)
def test_prefill_against_token_by_token(lib, mode):
    for layers in (BOTH, NO_FF):
        cfg = SI.make_config(vocab=90, width=64, layers=layers)
        m, W = make(lib, cfg, mode, seed=5)
        t = toks(2, 150, cfg["vocab"])
        whole = m.step([(0, t)], range(len(t)))
        one = np.concatenate([m.step([(1, t[i:i + 1])], [0]) for i in range(len(t))])
        want = R.forward(cfg, W, t)
        assert close(whole, want, mode) and close(one, want, mode)
        if layers is NO_FF:
            assert close(one, whole, mode)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", [[2, 2, 2, 3, 50, 2, 7, 1, 1, 30], [33, 1, 64, 2], [97, 3], [1] * 5 + [95], [70, 30], [2] * 50, [65, 16, 64, 17], [130, 2, 66]])
def test_portions_of_any_size(lib, mode, sizes):
    layers = NO_FF if mode == "bfloat16" else BOTH
    layers = layers + [SI.again(layers, 2), SI.again(layers, 0)]
    cfg = SI.make_config(vocab=77, width=48, layers=layers)
    m, W = make(lib, cfg, mode, seed=7)
    n = sum(sizes)
    t = toks(3, n, cfg["vocab"])
    want = R.forward(cfg, W, t)
    at, rows = 0, []
    for s in sizes:
        rows.append(m.step([(2, t[at:at + s])], range(s)))
        at += s
    assert m.position(2) == n
    assert close(np.concatenate(rows), want, mode)


def test_passes_inside_a_step_cut_anywhere(lib):
    """max_rows smaller than a step: the library cuts the step into passes; same logits."""
    t = toks(4, 200, 64)
    for mode, rows, layers in (("float32", 16, BOTH), ("bfloat16", 64, NO_FF), ("bfloat16", 40, NO_FF)):
        cfg = SI.make_config(vocab=64, width=64, layers=layers)
        m1, W = make(lib, cfg, mode, seed=9, max_rows=rows)
        m2, _ = make(lib, cfg, mode, seed=9)
        a = m1.step([(0, t), (1, t[:70])], range(270))
        b = m2.step([(0, t), (1, t[:70])], range(270))
        want = R.forward(cfg, W, t)
        assert close(a[:200], want, mode) and close(a[200:], want[:70], mode) and close(a, b, mode)


@pytest.mark.parametrize("n", [1, 2, 16, 17, 31, 32, 33, 63, 64, 65, 127, 128, 129, 257])
def test_chunk_borders_in_prompt_and_decode(lib, n):
    """Prompts that end just before, on and just behind a chunk's edge (64 rows, 32 for wide heads) and a few decoded tokens."""
    cfg = SI.make_config(vocab=64, width=64, layers=[ML(heads=2, dim=48, vdim=31), DE(heads=4, kv_heads=2, dim=32, vdim=64), ML(heads=1, dim=144, vdim=80), DE(heads=1, kv_heads=1, dim=130, vdim=16), PA()])
    for mode in MODES:
        m, W = make(lib, cfg, mode, seed=19)
        t = toks(30, n + 3, 64)
        want = R.forward(cfg, W, t)
        got = m.step([(0, t[:n])], range(n))
        got = np.concatenate([got] + [m.step([(0, t[n + i:n + i + 1])], [0]) for i in range(3)])
        assert rel(got, want) < TOL[mode]


# ------------------------------------------------------------------ batches, slots
@pytest.mark.parametrize("mode", MODES)
def test_batch_of_unequal_requests_equals_each_alone(lib, mode):
    cfg = SI.make_config(vocab=80, width=64, layers=BOTH if mode == "float32" else NO_FF)
    m, W = make(lib, cfg, mode, seed=11, n_slots=5)
    seqs = [toks(10 + i, n, 80) for i, n in enumerate((67, 5, 200, 1, 131))]
    first = [s[: max(1, len(s) // 2)] for s in seqs]
    out1 = m.step([(i, f) for i, f in enumerate(first)], range(sum(len(f) for f in first)))
    rest = [(i, s[len(f):]) for i, (s, f) in enumerate(zip(seqs, first)) if len(s) > len(f)]
    out2 = m.step(rest, range(sum(len(r) for _, r in rest)))
    at1, at2 = 0, 0
    for i, (s, f) in enumerate(zip(seqs, first)):
        want = R.forward(cfg, W, s)
        got = out1[at1:at1 + len(f)]
        at1 += len(f)
        if len(s) > len(f):
            got = np.concatenate([got, out2[at2:at2 + len(s) - len(f)]])
            at2 += len(s) - len(f)
        assert close(got, want, mode), i


@pytest.mark.parametrize("mode", MODES)
def test_decoding_beside_a_prompt(lib, mode):
    """Steps that mix single decoded rows with prompt portions, short enough for the row kernels and long enough for the chunked ones."""
    cfg = SI.make_config(vocab=80, width=64, layers=NO_FF)
    m, W = make(lib, cfg, mode, seed=12, n_slots=3)
    a, b, c = toks(14, 60, 80), toks(15, 150, 80), toks(16, 12, 80)
    wa, wb, wc = (R.forward(cfg, W, x) for x in (a, b, c))
    m.step([(0, a[:50])])
    ia, ib, ic = 50, 0, 0
    for nb, nc in ((3, 2), (90, 0), (2, 5), (55, 5)):
        segs, n = [(0, a[ia:ia + 1]), (1, b[ib:ib + nb])], 1 + nb
        if nc:
            segs.append((2, c[ic:ic + nc]))
        got = m.step(segs, range(n + nc))
        assert rel(got[:1], wa[ia:ia + 1]) < TOL[mode] and rel(got[1:n], wb[ib:ib + nb]) < TOL[mode]
        if nc:
            assert rel(got[n:], wc[ic:ic + nc]) < TOL[mode]
        ia, ib, ic = ia + 1, ib + nb, ic + nc


@pytest.mark.parametrize("mode", MODES)
def test_slot_freed_and_used_again(lib, mode):
    """States that hardly decay and convolutions that mostly read the past: a state, a running maximum or a history left behind would show."""
    from tinyllama_cpp_b200.scheduler import SlotManager

    def tweak(t):
        for k in t:
            if k.endswith(".conv"):
                put(t, k, lambda a: a.__setitem__((slice(None), 0), 1.5))
            elif k.endswith(".f.b"):
                put(t, k, lambda a: a.fill(6.0))
            elif k.endswith(".i.b"):
                put(t, k, lambda a: a.fill(3.0))
            elif k.endswith("dt_bias"):
                put(t, k, lambda a: a.fill(-7.0))
    cfg = SI.make_config(vocab=70, width=64, layers=[DE(conv=4), PA(conv=4), ML(), SI.again([DE(conv=4)], 0)])
    m, W = make(lib, cfg, mode, seed=13, n_slots=2, tweak=tweak)
    sm = SlotManager(m)
    a, b, c = toks(20, 90, 70), toks(21, 9, 70), toks(22, 75, 70)
    sa = sm.acquire("a")
    m.step([(sa, a)])
    sb = sm.acquire("b")
    m.step([(sb, b[:4])])
    sm.release("a")
    sc = sm.acquire("c")
    assert sc == sa
    got_c = m.step([(sc, c[:2]), (sb, b[4:])], range(2 + len(b) - 4))
    assert rel(got_c[:2], R.forward(cfg, W, c)[:2]) < TOL[mode]
    assert rel(got_c[2:], R.forward(cfg, W, b)[4:]) < TOL[mode]
    assert rel(m.step([(sc, c[2:])], range(len(c) - 2)), R.forward(cfg, W, c)[2:]) < TOL[mode]
    with pytest.raises(RuntimeError):
        sm.acquire("d")


def test_a_layer_run_again_keeps_a_state_of_its_own(lib):
    """Shared tensors, separate caches, states and histories: another layer's state in its place would change everything after it."""
    base = [DE(conv=4), PA(), ML()]
    cfg = SI.make_config(vocab=60, width=48, layers=base + [SI.again(base, i) for i in (0, 1, 2)])
    for mode in MODES:
        m, W = make(lib, cfg, mode, seed=14)
        assert m.n_runs == 6 and not any(k.startswith(("l3.", "l4.", "l5.")) for k in W)
        t = toks(23, 120, 60)
        want = R.forward(cfg, W, t)
        got = np.concatenate([m.step([(0, t[:80])], range(80)), m.step([(0, t[80:83])], range(3)), m.step([(0, t[83:])], range(37))])
        assert rel(got, want) < TOL[mode]


# ------------------------------------------------------------------ planted tokens: far keys, states that must last
NEEDLE, QUERY, C_NEEDLE, C_QUERY, C_ONE = 1, 2, 5, 9, 11


def planted(lib, kind, mode="float32", max_ctx=700, eps=1e-5):
    """One layer without a feed-forward.  Channel C_NEEDLE of the embedding is non-zero for token NEEDLE only and C_QUERY for token QUERY
    only.  "attention": head 0's query and its key read them with one strong entry.  "mlstm", "delta", "scan": the write of every token
    but NEEDLE is made small (input gate, beta, step size read C_NEEDLE; channel C_ONE is the same for every token), and nothing decays."""
    layers = {"attention": [PA(heads=2, kv_heads=1, dim=8, vdim=10, rot_dims=4, yarn=None, scale=1.5)], "scan": [PA(heads=2, kv_heads=1, dim=8, vdim=10, rot_dims=4, inner=24, conv=2)],
              "mlstm": [ML(heads=2, dim=12, vdim=10, gate_cap=30.0)], "delta": [DE(heads=2, kv_heads=1, dim=12, vdim=10, conv=2)]}[kind]
    cfg = SI.make_config(vocab=60, width=40, layers=layers, embed_scale=4.0, eps=eps)

    def row(r, col, value):
        def fn(a):
            a[r, :] = 0.0
            a[:, col] = 0.0
            a[r, col] = value
        return fn

    def tweak(t):
        def emb(a):
            a[:, C_NEEDLE] = 0.0
            a[:, C_QUERY] = 0.0
            a[:, C_ONE] = 0.4
            a[NEEDLE, C_NEEDLE] = 6.0
            a[QUERY, C_QUERY] = 6.0
        put(t, "embed", emb)
        put(t, "l0.norm1", lambda a: a.__setitem__([C_NEEDLE, C_QUERY], 1.0))
        p = "l0.mix."
        if kind == "attention":
            put(t, p + "left.q", row(6, C_QUERY, 3.0))
            put(t, p + "left.k", row(6, C_NEEDLE, 3.0))
            put(t, p + "left.q.b", lambda a: a.__setitem__(6, 0.0))
            put(t, p + "left.k.b", lambda a: a.__setitem__(6, 0.0))
            for n in ("q", "k"):
                put(t, p + f"left.{n}.norm", lambda a: a.__setitem__(6, 3.0))
        elif kind == "scan":
            # steps of a few ten-thousandths, of the order of one at the needle: the needle is found in x's first channel by the input projection
            put(t, p + "right.in", row(0, C_NEEDLE, 4.0))
            put(t, p + "right.x", lambda a: (a[:5].__setitem__((slice(None), slice(None)), 0.0), a.__setitem__((0, 0), 1.0)))
            put(t, p + "right.dt", lambda a: a.__setitem__((slice(None), 0), 0.6))
            put(t, p + "right.dt.b", lambda a: a.fill(-9.0))
            put(t, p + "right.A_log", lambda a: a.fill(-4.0))
        elif kind == "mlstm":
            for h in range(2):
                put(t, p + "i", lambda a: (a[h].fill(0.0), a.__setitem__((h, C_NEEDLE), 2.0)))
                put(t, p + "f", lambda a: a[h].fill(0.0))
            put(t, p + "i.b", lambda a: a.fill(-6.0))
            put(t, p + "f.b", lambda a: a.fill(9.0))
        else:
            for h in range(2):
                put(t, p + "b", lambda a: (a[h].fill(0.0), a.__setitem__((h, C_ONE), -3.5), a.__setitem__((h, C_NEEDLE), 2.0)))
            put(t, p + "dt_bias", lambda a: a.fill(-9.0))
            put(t, p + "A_log", lambda a: a.fill(-1.0))
    return cfg, make(lib, cfg, mode, seed=17, max_ctx=max_ctx, tweak=tweak)


def run_three_ways(m, t):
    """The last token's logits: whole prompt, decoded alone after the rest, and in portions of changing size."""
    n = len(t)
    whole = m.step([(0, t)], [n - 1])
    if n > 1:
        m.step([(1, t[:-1])])
    dec = m.step([(1, t[-1:])], [0])
    at, sizes = 0, [2, 37, 3, 64, 2, 90]
    while at < n - 1:
        s = min(sizes[0], n - 1 - at)
        sizes = sizes[1:] + sizes[:1]
        m.step([(2, t[at:at + s])])
        at += s
    por = m.step([(2, t[-1:])], [0])
    for s in range(3):
        m.reset(s)
    return whole, dec, por


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("kind", ["attention", "mlstm", "delta", "scan"])
def test_far_token_among_hundreds(lib, mode, kind):
    """One token hundreds of places back decides the answer; without it the answer moves far beyond the tolerance."""
    n = 640
    cfg, (m, W) = planted(lib, kind, mode)
    for at in (3, 63, 64, 500):
        t = toks(32, n, 60, lo=3)
        t[-1], t[at] = QUERY, NEEDLE
        book = {}
        want = R.forward(cfg, W, t, book=book)[-1:]
        if kind == "attention":
            assert book[0]["weights"][0][n - 1][at] > 0.5
        t2 = t.copy()
        t2[at] = 7
        moved = rel(R.forward(cfg, W, t2)[-1:], want)
        assert moved > 300 * TOL["float32"], moved
        if mode == "bfloat16" and moved < 3 * TOL[mode]:
            continue
        for got in run_three_ways(m, t):
            assert rel(got, want) < TOL[mode], at


@pytest.mark.parametrize("mode", MODES)
def test_the_denominator_of_the_matrix_memory(lib, mode):
    """An output norm whose eps matters lets the denominator's size show: max(|n . q|, exp(-m)) takes both sides, under running maxima of about
    -4, 0 and 17."""
    cfg = SI.make_config(vocab=60, width=48, layers=[ML(heads=3, gate_cap=25.0)], eps=0.05)

    def tweak(t):
        put(t, "l0.mix.i.b", lambda a: a.__setitem__(slice(None), [-4.0, 0.0, 20.0]))
        put(t, "l0.mix.f.b", lambda a: a.__setitem__(slice(None), [0.5, 2.0, 2.0]))
        put(t, "l0.norm1b", lambda a: a.__imul__(4.0))
    m, W = make(lib, cfg, mode, seed=25, tweak=tweak)
    t = toks(33, 150, 60)
    book = {}
    want = R.forward(cfg, W, t, book=book)
    nq, mx = (np.array([book[0][h][k] for h in range(3)]) for k in ("nq", "m"))
    floor = np.abs(nq) < np.exp(-mx)
    assert 0.2 < floor[:2].mean() < 0.98 and np.median(mx[2]) > 15.0
    assert rel(m.step([(0, t)], range(150)), want) < TOL[mode]
    got = np.concatenate([m.step([(1, t[i:i + 1])], [0]) for i in range(60)])
    assert rel(got, want[:60]) < TOL[mode]
    plain = R.mlstm_scan

    def no_floor(q, k, v, i, f, book=None):
        b = {}
        o = plain(q, k, v, i, f, b)
        n = np.abs(b["nq"])
        return o * ((np.maximum(n, np.exp(-np.array(b["m"]))) + 1e-6) / (n + 1e-6))[:, None]
    try:
        R.mlstm_scan = no_floor
        assert rel(R.forward(cfg, W, t), want) > 100 * TOL["float32"]
    finally:
        R.mlstm_scan = plain


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("how", ["forget_everything", "keep_everything", "mixed"])
def test_extreme_gates(lib, mode, how):
    """Log decays of about -12 a token (sums of hundreds inside a chunk), of about zero, and heads of both kinds side by side; input gates at the
    cap in both directions."""
    cfg = SI.make_config(vocab=60, width=48, layers=[ML(heads=4, dim=16, vdim=24, gate_cap=12.0), DE(heads=4, kv_heads=2), PA(inner=32, state=8)])

    def spread(lo, hi):
        return lambda a: a.__setitem__(slice(None), {"forget_everything": np.full(a.shape, lo), "keep_everything": np.full(a.shape, hi),
                                                     "mixed": np.resize([lo, hi], a.shape)}[how])

    def tweak(t):
        put(t, "l0.mix.f.b", spread(-20.0, 20.0))
        put(t, "l0.mix.i.b", lambda a: a.__setitem__(slice(None), [-30.0, 30.0, 30.0, 2.0]))
        put(t, "l1.mix.dt_bias", spread(4.0, -12.0))
        put(t, "l1.mix.A_log", spread(1.5, -3.0))
        put(t, "l2.mix.right.dt.b", spread(4.0, -9.0))
    m, W = make(lib, cfg, mode, seed=26, tweak=tweak)
    t = toks(34, 200, 60)
    want = R.forward(cfg, W, t)
    assert np.isfinite(want).all()
    assert close(m.step([(0, t)], range(200)), want, mode)
    got = np.concatenate([m.step([(1, t[:131])], range(131))] + [m.step([(1, t[i:i + 1])], [0]) for i in range(131, 160)])
    assert close(got, want[:160], mode)


def test_repeated_keys_under_the_delta_rule(lib):
    """Runs of one token: equal keys with large beta make the chunk's triangular system far from the identity."""
    cfg = SI.make_config(vocab=40, width=48, layers=[DE(heads=4, kv_heads=2, conv=1), DE(heads=2, kv_heads=2, conv=2)])

    def tweak(t):
        for i in (0, 1):
            put(t, f"l{i}.mix.b", lambda a: a.__imul__(6.0))
            put(t, f"l{i}.mix.dt_bias", lambda a: a.fill(-9.0))
    for mode in MODES:
        m, W = make(lib, cfg, mode, seed=27, tweak=tweak)
        t = np.repeat(toks(35, 10, 40), 19)[:180]
        want = R.forward(cfg, W, t)
        assert rel(m.step([(0, t)], range(180)), want) < TOL[mode]
        assert rel(np.concatenate([m.step([(1, t[i:i + 1])], [0]) for i in range(70)]), want[:70]) < TOL[mode]


def test_first_tokens(lib):
    """Positions 0 .. a few: convolutions that reach in front of the sequence, states and the running maximum at their start."""
    cfg = SI.make_config(vocab=50, width=64, layers=[DE(conv=4), PA(conv=8), ML(), DE(conv=7)])
    for mode in MODES:
        m, W = make(lib, cfg, mode, seed=23)
        t = toks(40, 11, 50)
        want = R.forward(cfg, W, t)
        assert rel(m.step([(0, t)], range(11)), want) < TOL[mode]
        got = np.concatenate([m.step([(1, t[i:i + 1])], [0]) for i in range(11)])
        assert rel(got, want) < TOL[mode]
        got = np.concatenate([m.step([(2, t[i:i + 2])], range(len(t[i:i + 2]))) for i in range(0, 11, 2)])
        assert rel(got, want) < TOL[mode]


def test_router_weights_are_the_softmax_over_the_chosen(lib):
    """Two experts with identical router rows tie at every token: the lower index is chosen.  A softmax over all experts would weigh differently."""
    cfg = SI.make_config(vocab=60, width=48, layers=[ML(mlp=E(ff=24, experts=6, top=2))])

    def tweak(t):
        put(t, "l0.mlp.router", lambda a: a.__setitem__(4, a[2]))
        put(t, "l0.norm2b", lambda a: a.__imul__(4.0))
    for mode, n in (("float32", 90), ("float32", 5)):
        m, W = make(lib, cfg, mode, seed=28, tweak=tweak)
        t = toks(36, n, 60)
        want = R.forward(cfg, W, t)
        assert rel(m.step([(0, t)], range(n)), want) < TOL[mode]
    swapped = dict(W)
    for n in ("gate", "up", "down"):
        swapped[f"l0.mlp.e2.{n}"], swapped[f"l0.mlp.e4.{n}"] = W[f"l0.mlp.e4.{n}"], W[f"l0.mlp.e2.{n}"]
    assert rel(R.forward(cfg, swapped, toks(36, 90, 60)), R.forward(cfg, W, toks(36, 90, 60))) > 50 * TOL["float32"]
    plain = R.route

    def all_experts(z, top):
        idx, _ = plain(z, top)
        s = np.exp(z - z.max(-1, keepdims=True))
        return idx, np.take_along_axis(s / s.sum(-1, keepdims=True), idx, -1)
    try:
        R.route = all_experts                         # (the norm behind the experts hides a common factor, not the eps beside it: compare the experts' own sum)
        h = np.random.default_rng(0).standard_normal((4, 48))
        a = R.experts(h, R.sub(W, "l0.mlp."), cfg["layers"][0]["mlp"])
    finally:
        R.route = plain
    assert not np.allclose(a, R.experts(h, R.sub(W, "l0.mlp."), cfg["layers"][0]["mlp"]), rtol=0.05)


# ------------------------------------------------------------------ long decoding, other sizes
@pytest.mark.parametrize("mode", MODES)
def test_long_decoding(lib, mode):
    cfg = SI.make_config(vocab=64, width=64, layers=NO_FF + [SI.again(NO_FF, 1)])
    m, W = make(lib, cfg, mode, seed=29)
    t = toks(50, 260, 64)
    want = R.forward(cfg, W, t)
    m.step([(0, t[:10])])
    got = np.concatenate([m.step([(0, t[i:i + 1])], [0]) for i in range(10, 260)])
    assert close(got, want[10:], mode)


@pytest.mark.parametrize("layers,vocab,width", [
    ([ML(heads=1, dim=40, vdim=40, gate_cap=3.0), DE(heads=5, kv_heads=5, dim=6, vdim=7, conv=2), PA(heads=7, kv_heads=7, dim=4, vdim=5, rot_dims=2, inner=9, state=3, dt_rank=2, conv=2)], 33, 40),
    ([PA(heads=6, kv_heads=2, dim=48, vdim=24, rot_dims=32, inner=136, state=24, dt_rank=72, conv=4), ML(heads=8, dim=24, vdim=40), DE(heads=8, kv_heads=2, dim=40, vdim=72, conv=5)], 130, 136),
    ([ML(heads=2, dim=136, vdim=200), PA(heads=2, kv_heads=1, dim=136, vdim=136, rot_dims=136), DE(heads=3, kv_heads=3, dim=256, vdim=80, conv=3)], 64, 64),      # heads beyond the tiled attention, chunks of 32 rows
    ([DE(heads=12, kv_heads=4, dim=16, vdim=16, conv=4), ML(heads=12, dim=16, vdim=16)], 64, 64),
    ([ML(heads=1, dim=520, vdim=8), DE(heads=1, kv_heads=1, dim=1000, vdim=6)], 37, 50),
])
def test_other_sizes(lib, layers, vocab, width):
    cfg = SI.make_config(vocab=vocab, width=width, layers=layers, eps=3e-4, embed_scale=2.5)
    for mode in MODES:
        m, W = make(lib, cfg, mode, seed=31)
        t = toks(60, 145, vocab)
        want = R.forward(cfg, W, t)
        got = np.concatenate([m.step([(0, t[:20])], range(20)), m.step([(0, t[20:22])], range(2)), m.step([(0, t[22:])], range(123))])
        assert close(got, want, mode), mode


@pytest.mark.parametrize("layers", [
    [ML(heads=4, dim=32, vdim=63), DE(heads=4, kv_heads=2, dim=64, vdim=64)],
    [ML(heads=2, dim=128, vdim=128), DE(heads=2, kv_heads=1, dim=128, vdim=128, conv=4), PA(inner=128, state=16, dt_rank=8)],
    [ML(heads=2, dim=200, vdim=100), DE(heads=4, kv_heads=4, dim=144, vdim=20), PA(heads=4, kv_heads=2, dim=64, vdim=64, rot_dims=64)],
])
def test_chunked_kernels_against_the_row_kernels(lib, layers):
    """bfloat16 prompt portions run the chunk kernels: portions that start in the middle of a sequence and end inside a chunk, passes of several
    segments -- against the restatement and against rows walked one by one (option fused_attn = 0)."""
    mode = "bfloat16"
    cfg = SI.make_config(vocab=64, width=64, layers=layers)
    m, W = make(lib, cfg, mode, seed=61, n_slots=4, max_ctx=400)
    a, b = toks(110, 300, 64), toks(111, 170, 64)
    wa, wb = R.forward(cfg, W, a), R.forward(cfg, W, b)
    outs = {}
    for fused in (1, 0):
        m.set_option("fused_attn", fused)
        sa, sb = (0, 1) if fused else (2, 3)
        g1 = m.step([(sa, a[:70])], range(70))
        g2 = m.step([(sa, a[70:199]), (sb, b[:33])], range(129 + 33))
        g3 = m.step([(sb, b[33:170]), (sa, a[199:300])], range(137 + 101))
        ga = np.concatenate([g1, g2[:129], g3[137:]])
        gb = np.concatenate([g2[129:], g3[:137]])
        assert close(ga, wa, mode) and close(gb, wb, mode), fused
        outs[fused] = (ga, gb)
    assert rel(outs[1][0], outs[0][0]) < TOL[mode] and rel(outs[1][1], outs[0][1]) < TOL[mode] and np.median(rows_rel(outs[1][0], outs[0][0])) < 0.1 * TOL[mode]
    m.set_option("fused_attn", 1)
    nxt = m.step([(0, [5])], [0])            # decoding continues from the states the chunk kernels left
    assert rel(nxt, R.forward(cfg, W, np.append(a, 5))[-1:]) < TOL[mode]


@pytest.mark.parametrize("mode", MODES)
def test_decode_rows_of_several_sequences(lib, mode):
    """Sequences at unequal positions decoded together (one to twelve rows)."""
    cfg = SI.make_config(vocab=64, width=64, layers=NO_FF)
    m, W = make(lib, cfg, mode, seed=63, n_slots=12, max_ctx=400)
    lens = (9, 150, 331, 1, 64, 65, 20, 21, 22, 23, 24, 25)
    seqs = [toks(140 + i, n + 4, 64) for i, n in enumerate(lens)]
    want = [R.forward(cfg, W, q) for q in seqs]
    for group in ((0, 1, 2), range(3, 12)):
        for i in group:
            m.step([(i, seqs[i][:-4])])
    for k in range(4):
        for group in ((0, 1, 2), range(12)) if k == 0 else (range(12),):
            rows = [i for i in group if k > 0 or m.position(i) == lens[i]]
            got = m.step([(i, seqs[i][lens[i] + k:lens[i] + k + 1]) for i in rows], range(len(rows)))
            for j, i in enumerate(rows):
                assert rel(got[j:j + 1], want[i][lens[i] + k:lens[i] + k + 1]) < 1.5 * TOL[mode], (mode, i)


def test_tensor_core_path_with_awkward_sizes(lib):
    """bfloat16 mode, portions of 64 rows and more: the tcgen05 products with sizes that are multiples of nothing, against the SIMT kernels."""
    cfg = SI.make_config(vocab=101, width=72, layers=[PA(heads=6, kv_heads=3, dim=12, vdim=14, inner=50, state=9, dt_rank=7), ML(heads=3, dim=21, vdim=13), DE(heads=3, kv_heads=1, dim=11, vdim=19)])
    m, W = make(lib, cfg, "bfloat16", seed=67)
    t = toks(120, 150, cfg["vocab"])
    want = R.forward(cfg, W, t)
    got = np.concatenate([m.step([(0, t[:70])], range(70)), m.step([(0, t[70:])], range(80))])
    assert close(got, want, "bfloat16")
    m.set_option("tensor", 0)
    simt = np.concatenate([m.step([(1, t[:70])], range(70)), m.step([(1, t[70:])], range(80))])
    assert close(got, simt, "bfloat16")


def test_new_parameters_combine_with_the_other_families_forms(lib):
    """A description of no family: layer-norm sandwich layers that sum (not join) a retention and a delta branch, an mLSTM beside attention with a
    window, a selective scan alone with a GELU feed-forward, and gated experts with logistic weights and a shared expert -- prefill against token by token."""
    s = lib
    Wd, H = 64, 2
    ret = {"kind": s.MIX_RETENTION, "name": "r", "heads": H, "dim": 16, "vdim": 16, "scale": 0.25, "decay": [0.9, 0.99]}
    dl = {"kind": s.MIX_DELTA, "name": "d", "heads": H, "kv_heads": 1, "dim": 16, "vdim": 12, "scale": 0.25, "conv": 3, "out_scale": 0.7}
    ml = {"kind": s.MIX_MLSTM, "name": "m", "heads": H, "dim": 16, "vdim": 12, "scale": 0.25, "gate_cap": 8.0, "out_scale": 1.2}
    at = {"kind": s.MIX_SOFTMAX_ATTN, "name": "a", "heads": H, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.25, "kv_from": -1, "window": 20}
    ss = {"kind": s.MIX_SSM, "name": "", "inner": 40, "state": 5, "dt_rank": 3, "conv": 2}
    lay = lambda br, **kw: {"style": s.BLOCK_SANDWICH, "norm_kind": s.NORM_LAYER_NB, "branches": br, "ff": 0, **kw}
    moe = dict(ff=32, ff_kind=s.FF_GATED_EXPERTS, experts=4, top=2, shared_ff=32)
    desc = {"vocab": 50, "width": Wd, "eps": 1e-5, "final_norm": 5, "layers": [lay([ret, dl]), lay([ml, at], **moe), lay([ss], ff=48, ff_kind=s.FF_GELU), lay([ret, dl], weights_of=0)]}
    shapes = {"embed": (50, Wd), "head": (50, Wd), "final.norm": (Wd,)}
    for i in range(3):
        shapes.update({f"l{i}.norm{q}": (Wd,) for q in (("1", "1b") if i == 0 else ("1", "1b", "2", "2b"))})
    p = "l0.mix."
    shapes.update({p + "r." + k: (32, Wd) for k in "qkv"} | {p + "r.o": (Wd, 32)})
    shapes.update({p + "d.q": (16, Wd), p + "d.k": (16, Wd), p + "d.v": (24, Wd), p + "d.g": (24, Wd), p + "d.a": (2, Wd), p + "d.b": (2, Wd), p + "d.A_log": (2,), p + "d.dt_bias": (2,), p + "d.norm": (12,),
                   p + "d.q.conv": (16, 3), p + "d.k.conv": (16, 3), p + "d.v.conv": (24, 3), p + "d.o": (Wd, 24)})
    p = "l1.mix."
    shapes.update({p + "m.q": (32, Wd), p + "m.k": (32, Wd), p + "m.v": (24, Wd), p + "m.g": (24, Wd), p + "m.i": (2, Wd), p + "m.f": (2, Wd), p + "m.i.b": (2,), p + "m.f.b": (2,), p + "m.norm": (24,),
                   p + "m.o": (Wd, 24), p + "a.q": (32, Wd), p + "a.k": (16, Wd), p + "a.v": (16, Wd), p + "a.o": (Wd, 32)})
    q = "l1.mlp."
    shapes.update({q + "router": (4, Wd), q + "shared.gate": (32, Wd), q + "shared.up": (32, Wd), q + "shared.down": (Wd, 32), q + "shared.sg": (1, Wd)})
    for e in range(4):
        shapes.update({q + f"e{e}.gate": (32, Wd), q + f"e{e}.up": (32, Wd), q + f"e{e}.down": (Wd, 32)})
    p = "l2.mix."
    shapes.update({p + "in": (80, Wd), p + "conv": (40, 2), p + "conv.b": (40,), p + "x": (13, 40), p + "dt": (40, 3), p + "dt.b": (40,), p + "A_log": (40, 5), p + "D": (40,), p + "o": (Wd, 40),
                   "l2.mlp.up": (48, Wd), "l2.mlp.down": (Wd, 48)})
    rng = np.random.default_rng(5)
    t = {k: st.f32_to_bf16_bits((rng.standard_normal(sh) / (np.sqrt(sh[-1]) if len(sh) == 2 and "conv" not in k and k != "embed" else 1.0)).astype(np.float32)) for k, sh in shapes.items()}
    x = toks(7, 90, 50)
    for mode in MODES:
        m = s.SeqModel(desc, s.MODE_BY_NAME[mode], 2, 128).load(t)
        whole = m.step([(0, x)], range(90))
        one = np.concatenate([m.step([(1, x[i:i + 1])], [0]) for i in range(90)])
        assert np.isfinite(whole).all()
        assert (rel(one, whole) if mode == "float32" else float(np.median(rows_rel(one, whole)))) < TOL[mode]


# ------------------------------------------------------------------ generation through the scheduler, command line
def oracle_greedy(cfg, W, prompt, n_new):
    t = list(prompt)
    margins = []
    for _ in range(n_new):
        lg = R.forward(cfg, W, t)[-1]
        o = np.argsort(lg)
        margins.append(lg[o[-1]] - lg[o[-2]])
        t.append(int(o[-1]))
    return np.asarray(t[len(prompt):]), np.asarray(margins)


def test_greedy_generation_through_the_scheduler(lib):
    from tinyllama_cpp_b200.scheduler import generate
    cfg = SI.make_config(vocab=64, width=64)
    m, W = make(lib, cfg, "float32", seed=41, n_slots=2, gain=2.0)
    prompts = [toks(80 + i, n, 64) for i, n in enumerate((19, 3, 40))]     # three requests, two slots: one waits
    outs = generate(m, prompts, 12, chunk=8, burst=5)
    for p, o in zip(prompts, outs):
        want, margin = oracle_greedy(cfg, W, p, 12)
        assert len(o) == 12
        k = int(np.argmax(o != want)) if np.any(o != want) else 12
        assert k == 12 or margin[k] < 1e-3, (o, want, margin)
        assert len(set(o.tolist())) > 2
    sampled = generate(m, prompts, 6, top_k=5, temperature=0.7, seed=3)
    assert all(len(o) == 6 for o in sampled)


def test_device_decode_loop_equals_host_fed_steps(lib):
    cfg = SI.make_config(vocab=64, width=64)
    for mode in MODES:
        m, _ = make(lib, cfg, mode, seed=43, n_slots=3, gain=2.0)
        p0, p1 = toks(90, 11, 64), toks(91, 30, 64)
        nxt = m.step_greedy([(0, p0), (1, p1)])
        dev = m.decode([0, 1], 20)
        m.set_option("graph", 0)
        m.reset(0), m.reset(1)
        assert np.array_equal(nxt, m.step_greedy([(0, p0), (1, p1)]))
        assert np.array_equal(dev, m.decode([0, 1], 20))
        m.set_option("graph", 1)
        m.reset(0), m.reset(1)
        m.step_greedy([(0, p0), (1, p1)])
        cur, host = [int(x) for x in nxt], [[], []]
        for _ in range(20):
            cur = [int(x) for x in m.step_greedy([(0, [cur[0]]), (1, [cur[1]])])]
            host[0].append(cur[0]), host[1].append(cur[1])
        assert host == dev.tolist() and m.position(1) == 30 + 20 and len(set(host[1])) > 2


def test_a_sequence_that_stops_beside_one_that_goes_on(lib):
    """Sequence 0 samples the end id in the device loop: it repeats that id, its position and states stay, sequence 1 is not disturbed, and the slot
    starts afresh after a reset."""
    cfg = SI.make_config(vocab=64, width=64)
    for seed in range(44, 60):                     # a model whose first sequence samples an id the second one does not
        m, W = make(lib, cfg, "float32", seed=seed, n_slots=2, gain=2.0)
        p0, p1 = toks(92, 11, 64), toks(93, 30, 64)
        nxt = m.step_greedy([(0, p0), (1, p1)])
        free = m.decode([0, 1], 12)
        ids = [int(e) for e in free[0] if e not in free[1] and e != nxt[0] and e != nxt[1]]
        if ids:
            break
    eos = ids[0]
    first = free[0].tolist().index(eos)
    m.reset(0), m.reset(1)
    m.step_greedy([(0, p0), (1, p1)])
    got = m.decode([0, 1], 12, eos)
    assert (got[0][first:] == eos).all() and got[0][:first].tolist() == free[0][:first].tolist() and np.array_equal(got[1], free[1])
    assert m.position(0) == 11 + 1 + first and m.position(1) == 30 + 12
    # the stopped slot's state is the one before the end id was fed: feeding it by hand continues as the free run did
    seq = np.concatenate([p0, nxt[:1], free[0][:first]])
    want = R.forward(cfg, W, np.append(seq, eos))[-1:]
    assert rel(m.step([(0, [eos])], [0]), want) < TOL["float32"]
    m.reset(0)
    assert rel(m.step([(0, p1[:9])], range(9)), R.forward(cfg, W, p1[:9])) < TOL["float32"]


def test_missing_and_misshapen_tensors_are_named(lib):
    cfg = SI.make_config(vocab=64, width=64)
    d = SI.describe(cfg)
    for gone in ("l0.mix.dt_bias", "l1.mix.right.A_log", "l1.mix.left.out", "l2.mix.f.b", "l1.mlp.e5.down"):
        t = SI.synth_tensors(d, 0)
        t.pop(gone)
        with pytest.raises(lib.SeqError, match=gone):
            lib.SeqModel(d, lib.F32, 1, 16).load(t)
    t = SI.synth_tensors(d, 0)
    t["l0.mix.v.conv"] = t["l0.mix.q.conv"][:5]
    with pytest.raises(lib.SeqError, match="l0.mix.v.conv"):
        lib.SeqModel(d, lib.F32, 1, 16).load(t)
    for extra, like in (("l3.norm1", "l1.norm1"), ("l0.mix.q.b", "l0.mix.norm"), ("l2.mix.conv", "l0.mix.q.conv"), ("l0.norm1.b", "l0.norm1")):
        t = SI.synth_tensors(d, 0)
        t[extra] = t[like]                             # tensors that this description does not have
        with pytest.raises(lib.SeqError, match=extra):
            lib.SeqModel(d, lib.F32, 1, 16).load(t)
    bad = SI.describe(cfg)
    bad["layers"][4]["weights_of"] = 3                 # a layer without tensors of its own
    with pytest.raises(lib.SeqError):
        lib.SeqModel(bad, lib.F32, 1, 16)


def test_command_line_generation_and_trace_replay(lib, tmp_path):
    """bin/generate and bin/trace_run on a checkpoint folder written by the family's own writer."""
    import subprocess
    import sys
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    base = [DE(), PA(), ML()]
    cfg = SI.make_config(vocab=64, width=64, layers=base + [SI.again(base, 1)])      # (no experts: bfloat16 is held to TOL below)
    t = SI.synth_tensors(SI.describe(cfg), 71, gain=2.0)
    SI.write_checkpoint(tmp_path / "m", cfg, t)
    W = {k: R.to_float(v) for k, v in t.items()}
    p = toks(130, 37, 64)
    out = subprocess.run([sys.executable, str(root / "bin" / "generate"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--prompt",
                          ",".join(map(str, p)), "--max-new", "6", "--chunk", "8"], capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr[-2000:]
    got = np.array([int(x) for x in out.stdout.strip().splitlines()[-1].split(",")])
    want, margin = oracle_greedy(cfg, W, p, 6)
    k = int(np.argmax(got != want)) if np.any(got != want) else 6
    assert k == 6 or margin[k] < 1e-3
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": p[:29].tolist(), "want": [28, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": p[29:].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [9], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": p[:3].tolist(), "want": [2]}], "end": ["b"]}]
    for dtype in MODES:
        o = tmp_path / ("o_" + dtype)
        tr = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(o), "--max-tokens", "64"],
                            input="\n".join(json.dumps(x) for x in steps) + "\n", capture_output=True, text=True, timeout=300)
        assert tr.returncode == 0, tr.stderr[-2000:]
        assert [l for l in tr.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
        lg = R.forward(cfg, W, np.append(p, 9))
        tol = TOL[dtype] if dtype == "float32" else 2.0 * TOL[dtype]
        assert rel(np.fromfile(o / "0.f32", "<f4").reshape(2, 64), lg[[28, 2]]) < tol      # in the order asked for
        assert not (o / "1.f32").exists()
        assert rel(np.fromfile(o / "2.f32", "<f4").reshape(1, 64), lg[37:38]) < tol
        assert rel(np.fromfile(o / "3.f32", "<f4").reshape(1, 64), lg[2:3]) < tol
