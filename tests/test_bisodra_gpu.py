"""The Bisodra family on the layer-list library (libgten_b200_seq.so) against the plain numpy restatement in oracle/bisodra_ref.py.

Every test makes its own small configuration and random weights.  float32 mode is held to rounding (1e-4 of the logits' spread);
bfloat16 mode to a loose bound that a wrong key, window edge, kept token or lost state still breaks by orders of magnitude.  Where
random weights would hide a fault (one far key among hundreds, a window's edge, the extra 1 in the denominator) the test plants a key:
one input channel marks the needle token and one the query token, a weight carries the first into one entry of a head's key and the
second into the same entry of that head's query, and the restatement confirms that this key takes the query's attention."""
import json

import numpy as np
import pytest

pytestmark = pytest.mark.gpu

from oracle import bisodra_ref as R  # noqa: E402
from tinyllama_cpp_b200 import bisodra as BI  # noqa: E402
from tinyllama_cpp_b200 import safetensors_io as st  # noqa: E402


@pytest.fixture(scope="module")
def lib():
    from tinyllama_cpp_b200 import build, seq
    build.build(target="seq")
    seq.init(0)
    return seq


def make(lib, cfg, mode="float32", seed=0, n_slots=3, max_ctx=512, max_rows=0, tweak=None, **synth):
    desc = BI.describe(cfg)
    t = BI.synth_tensors(desc, seed, **synth)
    if tweak:
        tweak(t)
    m = lib.SeqModel(desc, lib.MODE_BY_NAME[mode], n_slots, max_ctx, max_rows).load(t)
    return m, {k: R.to_float(v) for k, v in t.items()}


def rel(got, want):
    """Largest row: rms of the difference after removing each row's mean, over the rms spread of the expected rows."""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return float((np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())).max())


TOL = {"float32": 1e-4, "bfloat16": 6e-2}
MODES = ["float32", "bfloat16"]


def toks(seed, n, vocab, lo=0):
    return np.random.default_rng(2000 + seed).integers(lo, vocab, n).astype(np.int32)


WN, LA, D = BI.windowed_layer, BI.latent_layer, BI.dense_mlp


# ------------------------------------------------------------------ each mechanism alone
VARIANTS = {
    "windowed": [WN()],
    "windowed_no_mask": [WN(window=0)],
    "windowed_nothing_kept": [WN(window=9, keep_first=0)],
    "window_of_one_one_kept": [WN(window=1, keep_first=1)],
    "more_kept_than_the_window": [WN(window=3, keep_first=20)],
    "kept_everything": [WN(window=4, keep_first=100)],
    "conv_none": [WN(conv=0)],
    "conv_one_tap": [WN(conv=1)],
    "conv_two_taps": [WN(conv=2)],
    "conv_four_taps": [WN(conv=4, heads=6, kv_heads=2, dim=12)],
    "conv_seven_taps": [WN(conv=7, heads=3, kv_heads=1, dim=10)],
    "one_head": [WN(heads=1, kv_heads=1, dim=20)],
    "all_heads_own_keys": [WN(heads=5, kv_heads=5, dim=6, window=30)],
    "odd_head_size": [WN(heads=3, kv_heads=1, dim=7, conv=3)],
    "latent": [LA()],
    "latent_plain_rotation": [LA(yarn=None)],
    "latent_mostly_rotated": [LA(heads=2, dim=2, rot_dim=16, scale=0.9, yarn=(8.0, 64.0, 6.0, 1.5), rot_base=300.0)],
    "latent_all_frequencies_divided": [LA(rot_dim=8, yarn=(4.0, 6.0, 32.0, 2.0), scale=0.7)],
    "latent_no_frequency_divided": [LA(rot_dim=8, yarn=(4.0, 1e6, 2.0, 1.0), scale=0.7)],
    "latent_factor_one": [LA(yarn=(1.0, 32.0, 4.0, 1.0))],
    "latent_one_head": [LA(heads=1, dim=16, rot_dim=2, vdim=30, kv_rank=17, q_rank=9)],
    "latent_on_an_earlier_cache": [LA(heads=2), WN(), LA(heads=4, dim=6, vdim=9, q_rank=11, scale=0.5, kv_from=0), LA(heads=1, kv_from=0)],
    "two_shared_caches": [LA(), LA(kv_rank=16, rot_dim=8), LA(kv_from=0, mlp=D(24)), LA(kv_rank=16, rot_dim=8, kv_from=1)],
    "dense": [WN(mlp=D(40))],
    "dense_wide": [LA(mlp=D(150))],
    "all": None,
}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("variant", list(VARIANTS))
def test_mechanisms_one_at_a_time(lib, mode, variant):
    cfg = BI.make_config(vocab=101, width=72, layers=VARIANTS[variant])
    m, W = make(lib, cfg, mode, seed=3)
    m.set_option("capture", 1)
    t = toks(1, 75, cfg["vocab"])
    trace = []
    want = R.forward(cfg, W, t, trace)
    got = m.step([(0, t)], range(len(t)))
    assert m.n_runs == len(trace)
    for u in range(m.n_runs):                # the stream after every layer
        for r in (0, 20, len(t) - 1):
            assert rel(m.read_capture(u, r)[None], trace[u][r][None]) < TOL[mode], (u, r)
    assert rel(got, want) < TOL[mode]
    one = np.concatenate([m.step([(1, t[i:i + 1])], [0]) for i in range(40)])
    assert rel(one, want[:40]) < TOL[mode]


@pytest.mark.parametrize("embed_scale,logit_scale", [(1.0, 1.0), (0.25, 7.0), (12.0, 0.0625), (3.0, -1.5)])
def test_scales_of_the_embedding_and_the_logits(lib, embed_scale, logit_scale):
    """The table scales on the way in and is the plain output matrix: the logits' own size is compared, not only their pattern."""
    for width in (64, 56):                    # rows that are, and are not, the padded operand width (a copy of the table)
        cfg = BI.make_config(vocab=70, width=width, layers=[WN(), LA()], embed_scale=embed_scale, logit_scale=logit_scale)
        for mode in MODES:
            m, W = make(lib, cfg, mode, seed=4)
            t = toks(9, 70, 70)
            want = R.forward(cfg, W, t)
            got = m.step([(0, t)], range(70))
            assert np.abs(got - want).max() < 6 * TOL[mode] * want.std(), (mode, width)


def test_gelu_is_the_erf_form(lib):
    """Activations of size 0.1 .. 4, where the erf and the tanh form differ most: the tensor-core epilogue and the row kernel."""
    cfg = BI.make_config(vocab=60, width=64, layers=[WN(mlp=D(96))])

    def tweak(t):                         # the feed-forward's share of the stream made large
        put(t, "l0.norm2b", lambda a: a.__imul__(8.0))
    for mode, n in (("float32", 90), ("bfloat16", 90), ("bfloat16", 5)):
        m, W = make(lib, cfg, mode, seed=6, gain=1.5, tweak=tweak)
        t = toks(8, n, 60)
        assert rel(m.step([(0, t)], range(n)), R.forward(cfg, W, t)) < TOL[mode]
    erf = R.gelu
    try:
        R.gelu = lambda z: 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))
        tanh = R.forward(cfg, W, t)
    finally:
        R.gelu = erf
    m, _ = make(lib, cfg, "float32", seed=6, gain=1.5, tweak=tweak)
    got = m.step([(0, t)], range(n))
    assert rel(got, tanh) > 20 * rel(got, R.forward(cfg, W, t))        # the restatement with the other form is told apart


# ------------------------------------------------------------------ prefill = decode = portions
@pytest.mark.parametrize("mode", MODES)
def test_prefill_against_token_by_token(lib, mode):
    cfg = BI.make_config(vocab=90, width=64)
    m, W = make(lib, cfg, mode, seed=5)
    t = toks(2, 90, cfg["vocab"])
    whole = m.step([(0, t)], range(len(t)))
    one = np.concatenate([m.step([(1, t[i:i + 1])], [0]) for i in range(len(t))])
    want = R.forward(cfg, W, t)
    assert rel(whole, want) < TOL[mode] and rel(one, want) < TOL[mode] and rel(one, whole) < TOL[mode]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", [[2, 2, 2, 3, 50, 2, 7, 1, 1, 30], [33, 1, 64, 2], [97, 3], [1] * 5 + [95], [70, 30], [2] * 50])
def test_portions_of_any_size(lib, mode, sizes):
    layers = [LA(mlp=D(48)), WN(conv=4, window=13, keep_first=6), LA(heads=2, kv_from=0, mlp=D()), WN(conv=6, window=40, keep_first=1, heads=2, kv_heads=1, dim=24, mlp=D(64))]
    cfg = BI.make_config(vocab=77, width=48, layers=layers)
    m, W = make(lib, cfg, mode, seed=7)
    n = sum(sizes)
    t = toks(3, n, cfg["vocab"])
    want = R.forward(cfg, W, t)
    at, rows = 0, []
    for s in sizes:
        rows.append(m.step([(2, t[at:at + s])], range(s)))
        at += s
    assert m.position(2) == n
    assert rel(np.concatenate(rows), want) < TOL[mode]


def test_passes_inside_a_step_cut_anywhere(lib):
    """max_rows smaller than a step: the library cuts the step into passes; same logits."""
    cfg = BI.make_config(vocab=64, width=64)
    t = toks(4, 70, 64)
    m1, W = make(lib, cfg, "float32", seed=9, max_rows=16)
    m2, _ = make(lib, cfg, "float32", seed=9)
    a = m1.step([(0, t), (1, t[:23])], range(93))
    b = m2.step([(0, t), (1, t[:23])], range(93))
    assert rel(a[:70], R.forward(cfg, W, t)) < TOL["float32"] and rel(a, b) < 1e-5


def test_passes_of_the_tiled_path(lib):
    """bfloat16, passes of 64 rows inside longer steps: every pass continues the caches and the convolution's history."""
    cfg = BI.make_config(vocab=64, width=64, layers=[WN(window=50, keep_first=9, mlp=D(64)), LA(mlp=D(32)), WN(conv=5), LA(kv_from=1)])
    t = toks(5, 200, 64)
    m1, W = make(lib, cfg, "bfloat16", seed=10, max_rows=64)
    m2, _ = make(lib, cfg, "bfloat16", seed=10)
    a = m1.step([(0, t), (1, t[:70])], range(270))
    b = m2.step([(0, t), (1, t[:70])], range(270))
    want = R.forward(cfg, W, t)
    assert rel(a[:200], want) < TOL["bfloat16"] and rel(a[200:], want[:70]) < TOL["bfloat16"] and rel(a, b) < TOL["bfloat16"]


# ------------------------------------------------------------------ batches, slots
@pytest.mark.parametrize("mode", MODES)
def test_batch_of_unequal_requests_equals_each_alone(lib, mode):
    cfg = BI.make_config(vocab=80, width=64)
    m, W = make(lib, cfg, mode, seed=11, n_slots=4)
    seqs = [toks(10 + i, n, 80) for i, n in enumerate((67, 5, 94, 1))]
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
        assert rel(got, want) < TOL[mode], i


@pytest.mark.parametrize("mode", MODES)
def test_decoding_beside_a_prompt(lib, mode):
    """Steps that mix single decoded rows with prompt portions, short enough for the row kernels and long enough for the tiled ones."""
    cfg = BI.make_config(vocab=80, width=64, layers=[WN(conv=4, window=20, keep_first=3, mlp=D()), LA(mlp=D()), WN(conv=2), LA(kv_from=1)])
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
    from tinyllama_cpp_b200.scheduler import SlotManager
    def tweak(t):                         # a convolution that mostly reads the past: a history left behind would show at once
        for k in ("l0.mix.q.conv", "l0.mix.k.conv"):
            a = st.bf16_bits_to_f32(t[k]).copy()
            a[:, 0] = 1.5
            t[k] = st.f32_to_bf16_bits(a)
    cfg = BI.make_config(vocab=70, width=64, layers=[WN(conv=4, mlp=D()), LA(), LA(kv_from=1)])
    m, W = make(lib, cfg, mode, seed=13, n_slots=2, tweak=tweak)
    sm = SlotManager(m)
    a, b, c = toks(20, 60, 70), toks(21, 9, 70), toks(22, 45, 70)
    sa = sm.acquire("a")
    m.step([(sa, a)])
    sb = sm.acquire("b")
    m.step([(sb, b[:4])])
    sm.release("a")
    sc = sm.acquire("c")                 # takes a's slot: neither a's cached keys nor its convolution history may show
    assert sc == sa
    got_c = m.step([(sc, c[:2]), (sb, b[4:])], range(2 + len(b) - 4))
    assert rel(got_c[:2], R.forward(cfg, W, c)[:2]) < TOL[mode]
    assert rel(got_c[2:], R.forward(cfg, W, b)[4:]) < TOL[mode]
    assert rel(m.step([(sc, c[2:])], range(len(c) - 2)), R.forward(cfg, W, c)[2:]) < TOL[mode]
    with pytest.raises(RuntimeError):
        sm.acquire("d")


# ------------------------------------------------------------------ planted keys: window edges, kept tokens, far keys
NEEDLE, QUERY, C_NEEDLE, C_QUERY = 1, 2, 5, 9


def put(t, name, fn):
    a = st.bf16_bits_to_f32(t[name]).astype(np.float64)
    fn(a)
    t[name] = st.f32_to_bf16_bits(a.astype(np.float32))


def planted(lib, kind, mode="float32", max_ctx=700, window=0, keep=0, heads=2, n_slots=3, dim=8):
    """One layer without a feed-forward.  Channel C_NEEDLE of the embedding is non-zero for token NEEDLE only and C_QUERY for token QUERY
    only (large: after the layer norm that channel stands out).  Filler tokens are 3 .. vocab-1.  "windowed": the first row of the last
    head's key projection reads C_NEEDLE only and that of its query projection C_QUERY only, through a convolution that passes
    the present (the last head's distance slope is the smallest).  "latent" / "shared": row 0 of the key latent reads C_NEEDLE and row 0 of
    the query latent C_QUERY, and head 0's first plain entries read only those; "shared" does it in a second layer that reads the first
    one's latents, whose own output is made small."""
    if kind == "windowed":
        layers = [WN(heads=heads, kv_heads=1, dim=dim, conv=3, window=window, keep_first=keep, scale=0.09)]
    else:
        layers = [LA(heads=heads, dim=dim, rot_dim=4, vdim=12, kv_rank=20, q_rank=16, scale=0.3)]
        if kind == "shared":
            layers.append(LA(heads=heads, dim=dim, rot_dim=4, vdim=12, kv_rank=20, q_rank=16, scale=0.3, kv_from=0))
    cfg = BI.make_config(vocab=60, width=40, layers=layers, embed_scale=4.0)

    def only(row, col, value, whole_column=True):
        def fn(a):
            a[row, :] = 0.0
            if whole_column:
                a[:, col] = 0.0
            a[row, col] = value
        return fn

    def tweak(t):
        def emb(a):
            a[:, C_NEEDLE] = 0.0
            a[:, C_QUERY] = 0.0
            a[NEEDLE, C_NEEDLE] = 10.0
            a[QUERY, C_QUERY] = 10.0
        put(t, "embed", emb)
        last = len(layers) - 1
        for i in range(len(layers)):
            put(t, f"l{i}.norm1", lambda a: a.__setitem__([C_NEEDLE, C_QUERY], 1.0))
        if kind == "windowed":
            row = (heads - 1) * dim
            put(t, "l0.mix.q", only(row, C_QUERY, 3.0))
            put(t, "l0.mix.k", only(0, C_NEEDLE, 3.0))
            for nm, r in (("q", row), ("k", 0)):
                put(t, f"l0.mix.{nm}.b", lambda a: a.__setitem__(r, 0.0))
                put(t, f"l0.mix.{nm}.conv", lambda a: a.__setitem__(r, [0.0, 0.0, 1.0]))
        else:
            put(t, "l0.mix.dkv", only(0, C_NEEDLE, 3.0))
            put(t, "l0.mix.dkv.norm", lambda a: a.__setitem__(0, 1.0))
            if last:
                put(t, "l0.norm1b", lambda a: a.__imul__(0.05))
            p = f"l{last}.mix."
            put(t, p + "dq", only(0, C_QUERY, 3.0))
            put(t, p + "dq.norm", lambda a: a.__setitem__(0, 1.0))
            put(t, p + "uq", only(0, 0, 4.0))
            put(t, p + "uk", only(0, 0, 4.0))
    return cfg, make(lib, cfg, mode, seed=17, max_ctx=max_ctx, n_slots=n_slots, tweak=tweak)


def needle_weight(cfg, W, t, kind):
    """Share of the last query's attention in the planted head that lands on needle tokens, by the restatement."""
    book = {}
    R.forward(cfg, W, t, book=book)
    lay = len(cfg["layers"]) - 1
    head = cfg["layers"][0]["mixer"]["heads"] - 1 if kind == "windowed" else 0
    w = book[lay]["weights"][head][len(t) - 1]
    return float(sum(w[j] for j in range(len(t)) if t[j] == NEEDLE))


def run_three_ways(m, t):
    """The last token's logits: whole prompt, decoded alone after the rest, and in portions of changing size."""
    n = len(t)
    whole = m.step([(0, t)], [n - 1])
    if n > 1:
        m.step([(1, t[:-1])])
    dec = m.step([(1, t[-1:])], [0])
    at, sizes = 0, [2, 37, 3, 64, 2, 5]
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
@pytest.mark.parametrize("window,keep,n", [(21, 5, 90), (64, 64, 200), (64, 10, 193), (1, 1, 40), (2, 70, 150), (130, 3, 300), (100, 0, 260), (33, 65, 99)])
def test_window_edge_and_kept_tokens(lib, mode, window, keep, n):
    """Seen: the window's oldest token and the last kept one.  Not seen: the token before the window and the first one that is not kept."""
    cfg, (m, W) = planted(lib, "windowed", mode, window=window, keep=keep)
    last = n - 1
    places = {last - window + 1: True, keep - 1: True, last - window: last - window < keep, keep: last - keep < window}
    for at, seen in places.items():
        if not 0 <= at < last:
            continue
        t = toks(30, n, 60, lo=3)
        t[-1], t[at] = QUERY, NEEDLE
        share = needle_weight(cfg, W, t, "windowed")
        assert share > 0.5 if seen else share == 0.0, (at, share)
        want = R.forward(cfg, W, t)[-1:]
        for got in run_three_ways(m, t):
            assert rel(got, want) < TOL[mode], at


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("kind", ["windowed", "latent", "shared"])
def test_far_key_among_hundreds(lib, mode, kind):
    """One needle hundreds of tokens back carries the last query (in the windowed form as a kept token); without it the answer moves."""
    n = 640
    cfg, (m, W) = planted(lib, kind, mode, window=50, keep=12)
    t = toks(32, n, 60, lo=3)
    t[-1], t[7] = QUERY, NEEDLE
    assert needle_weight(cfg, W, t, kind) > 0.5
    want = R.forward(cfg, W, t)[-1:]
    for got in run_three_ways(m, t):
        assert rel(got, want) < TOL[mode]
    t2 = t.copy()
    t2[7] = 7
    assert rel(R.forward(cfg, W, t2)[-1:], want) > 50 * TOL["float32"]


def test_slope_follows_true_distances(lib):
    """Two needles, one near and one a kept token far back: their shares differ by about exp(slope times the true distance between them)."""
    cfg, (m, W) = planted(lib, "windowed", "float32", window=30, keep=4, heads=4)
    t = toks(36, 400, 60, lo=3)
    t[-1], t[2], t[390] = QUERY, NEEDLE, NEEDLE
    book = {}
    want = R.forward(cfg, W, t, book=book)[-1:]
    w = book[0]["weights"][3][399]
    assert abs(np.log(w[390] / w[2]) - 2.0 ** -8 * 388) < 0.5 and w[2] > 0.05
    for got in run_three_ways(m, t):
        assert rel(got, want) < TOL["float32"]


def test_one_more_in_the_denominator(lib):
    """Random weights give small scores, so the extra 1 matters most at the first tokens: the restatement without it is told apart."""
    cfg = BI.make_config(vocab=60, width=40, layers=[WN(window=9, keep_first=2)])
    m, W = make(lib, cfg, "float32", seed=18)
    t = toks(37, 70, 60)
    got = m.step([(0, t)], range(70))
    assert rel(got, R.forward(cfg, W, t)) < TOL["float32"]
    plain = R.masked_softmax
    try:
        R.masked_softmax = lambda s, mask, extra: plain(s, mask, 0.0)
        assert rel(got, R.forward(cfg, W, t)) > 100 * TOL["float32"]
    finally:
        R.masked_softmax = plain


@pytest.mark.parametrize("n", [63, 64, 65, 127, 128, 129, 257])
def test_key_tile_borders_in_prompt_and_decode(lib, n):
    cfg = BI.make_config(vocab=64, width=64, layers=[WN(window=0), WN(window=150, keep_first=64, mlp=D(32)), LA(), WN(window=64, keep_first=65), LA(kv_from=2)])
    for mode in MODES:
        m, W = make(lib, cfg, mode, seed=19)
        t = toks(30, n + 2, 64)
        want = R.forward(cfg, W, t)
        got = m.step([(0, t[:n])], [n - 2, n - 1])
        got = np.concatenate([got, m.step([(0, t[n:n + 1])], [0]), m.step([(0, t[n + 1:])], [0])])
        assert rel(got, want[n - 2:]) < TOL[mode]


def test_first_tokens(lib):
    """Positions 0 .. a few: one key beside the extra 1, a convolution that reaches in front of the sequence."""
    cfg = BI.make_config(vocab=50, width=64, layers=[WN(conv=4, window=4, keep_first=2), LA(mlp=D()), WN(conv=8, window=3, keep_first=0), LA(kv_from=1)])
    for mode in MODES:
        m, W = make(lib, cfg, mode, seed=23)
        t = toks(40, 11, 50)
        want = R.forward(cfg, W, t)
        assert rel(m.step([(0, t)], range(11)), want) < TOL[mode]
        got = np.concatenate([m.step([(1, t[i:i + 1])], [0]) for i in range(11)])
        assert rel(got, want) < TOL[mode]
        got = np.concatenate([m.step([(2, t[i:i + 2])], range(len(t[i:i + 2]))) for i in range(0, 11, 2)])
        assert rel(got, want) < TOL[mode]


# ------------------------------------------------------------------ long decoding, other sizes
@pytest.mark.parametrize("mode", MODES)
def test_long_decoding(lib, mode):
    """Windows pass over decoded tokens for 250 steps; the latent layers keep every key."""
    cfg = BI.make_config(vocab=64, width=64, layers=[WN(window=40, keep_first=15, mlp=D()), LA(mlp=D()), WN(conv=4, window=17, keep_first=3), LA(kv_from=1)])
    m, W = make(lib, cfg, mode, seed=29)
    t = toks(50, 260, 64)
    want = R.forward(cfg, W, t)
    m.step([(0, t[:10])])
    got = np.concatenate([m.step([(0, t[i:i + 1])], [0]) for i in range(10, 260)])
    assert rel(got, want[10:]) < TOL[mode]


@pytest.mark.parametrize("layers,vocab,width", [
    ([WN(heads=1, kv_heads=1, dim=40, conv=2, window=7, keep_first=3, mlp=D(24)), LA(heads=5, dim=6, rot_dim=2, vdim=7, kv_rank=9, q_rank=5, mlp=D(33))], 33, 40),
    ([LA(heads=8, dim=24, rot_dim=8, vdim=40, kv_rank=72, q_rank=136, mlp=D(200)), WN(heads=6, kv_heads=2, dim=48, conv=5, window=6, keep_first=1), LA(heads=3, dim=8, rot_dim=8, vdim=16, kv_rank=72, q_rank=40, kv_from=0)], 130, 136),
    ([WN(heads=2, kv_heads=1, dim=136, conv=3, window=20, mlp=D(32)), LA(heads=2, dim=120, rot_dim=16, vdim=136, kv_rank=200, q_rank=64, mlp=D(64))], 64, 64),      # heads beyond the tiled kernels
    ([WN(heads=4, kv_heads=4, dim=20, conv=4, window=1, keep_first=1), WN(heads=12, kv_heads=3, dim=16, conv=1, window=64), LA(heads=20, dim=4, rot_dim=4, vdim=4, kv_rank=8, q_rank=8)], 64, 64),
    ([LA(heads=3, dim=10, rot_dim=10, vdim=10, kv_rank=10, q_rank=10, yarn=(3.0, 20.0, 3.0, 0.5), mlp=D(10)), WN(heads=3, kv_heads=3, dim=10, conv=3, mlp=D(30))], 37, 50),
])
def test_other_sizes(lib, layers, vocab, width):
    cfg = BI.make_config(vocab=vocab, width=width, layers=layers, eps=3e-4, embed_scale=2.5, logit_scale=1.25)
    for mode in MODES:
        m, W = make(lib, cfg, mode, seed=31)
        t = toks(60, 105, vocab)
        want = R.forward(cfg, W, t)
        got = np.concatenate([m.step([(0, t[:20])], range(20)), m.step([(0, t[20:22])], range(2)), m.step([(0, t[22:])], range(83))])
        assert rel(got, want) < TOL[mode], mode


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("layers", [
    [WN(heads=4, kv_heads=2, dim=16, conv=4, window=100, keep_first=70, mlp=D(96)), LA(heads=2, dim=24, rot_dim=8, vdim=48, kv_rank=64, q_rank=64, mlp=D(64))],
    [LA(heads=4, dim=48, rot_dim=16, vdim=80, kv_rank=128, q_rank=64), WN(heads=4, kv_heads=1, dim=64, conv=2, window=33, keep_first=5), LA(heads=2, dim=40, rot_dim=16, vdim=24, kv_rank=128, q_rank=24, kv_from=0)],
    [WN(heads=3, kv_heads=3, dim=96, conv=3, window=64, keep_first=64, mlp=D(80)), WN(heads=2, kv_heads=2, dim=20, window=0), LA(heads=1, dim=100, rot_dim=20, vdim=128, kv_rank=40, q_rank=40)],
])
def test_tiled_kernels_on_portions(lib, mode, layers):
    """Prompt portions run the tiled path (tensor-core attention with kept tokens, slopes and one tile for keys and values; expanded
    latents): portions that start in the middle of a sequence and end inside a tile, passes of several segments -- against the restatement
    and against the row kernels (option fused_attn = 0)."""
    cfg = BI.make_config(vocab=64, width=64, layers=layers)
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
        assert rel(ga, wa) < TOL[mode] and rel(gb, wb) < TOL[mode], fused
        outs[fused] = (ga, gb)
    assert rel(outs[1][0], outs[0][0]) < TOL[mode] and rel(outs[1][1], outs[0][1]) < TOL[mode]
    m.set_option("fused_attn", 1)
    nxt = m.step([(0, [5])], [0])            # decoding continues from the caches the tiled path left
    assert rel(nxt, R.forward(cfg, W, np.append(a, 5))[-1:]) < TOL[mode]


def test_decode_rows_of_several_sequences(lib):
    """Sequences at unequal positions (inside the first key tile, across several, past the windows) decoded together, with the keys of a
    row split over several CTAs (more than 128 keys)."""
    cfg = BI.make_config(vocab=64, width=64, layers=[WN(window=200, keep_first=40), LA(), WN(window=0), LA(heads=17, kv_from=1)])
    for mode in MODES:
        m, W = make(lib, cfg, mode, seed=63, n_slots=3, max_ctx=400)
        seqs = [toks(140 + i, n, 64) for i, n in enumerate((9, 150, 331))]
        want = [R.forward(cfg, W, q) for q in seqs]
        for i, q in enumerate(seqs):
            m.step([(i, q[:-4])])
        rows = [m.step([(i, q[len(q) - 4 + k:len(q) - 3 + k]) for i, q in enumerate(seqs)], range(3)) for k in range(4)]
        got = np.stack(rows, 1)                          # [sequence, step, vocab]
        for i in range(3):
            assert rel(got[i], want[i][-4:]) < TOL[mode], (mode, i)


def test_tensor_core_path_with_awkward_sizes(lib):
    """bfloat16 mode, portions of 64 rows and more: the tcgen05 products (bias and GELU epilogues) and the tiled attention with sizes that
    are multiples of nothing, against the SIMT kernels."""
    cfg = BI.make_config(vocab=101, width=72, layers=[WN(heads=6, kv_heads=3, dim=12, conv=3, window=37, keep_first=11, mlp=D(85)), LA(heads=3, dim=20, rot_dim=6, vdim=10, kv_rank=36, q_rank=28, mlp=D(97))])
    m, W = make(lib, cfg, "bfloat16", seed=67)
    t = toks(120, 150, cfg["vocab"])
    want = R.forward(cfg, W, t)
    got = np.concatenate([m.step([(0, t[:70])], range(70)), m.step([(0, t[70:])], range(80))])
    assert rel(got, want) < TOL["bfloat16"]
    m.set_option("tensor", 0)
    simt = np.concatenate([m.step([(1, t[:70])], range(70)), m.step([(1, t[70:])], range(80))])
    assert rel(got, simt) < TOL["bfloat16"]


# ------------------------------------------------------------------ the new parameters beside the older ones
def test_new_parameters_combine_with_the_other_families_forms(lib):
    """A description of no family: bias-free RMS sandwich layers whose attention convolves q and k but keeps values of its own, and whose
    keys-as-values attention has a learned sink and one gate per head -- prefill against token by token."""
    s = lib
    H, G, Dm, V, Wd = 4, 2, 16, 24, 64
    a = {"kind": s.MIX_SOFTMAX_ATTN, "name": "", "heads": H, "kv_heads": G, "dim": Dm, "vdim": V, "scale": 0.25, "kv_from": -1, "conv": 3, "window": 20, "keep_first": 4,
         "slopes": 1, "bias": 1}
    b = {"kind": s.MIX_SOFTMAX_ATTN, "name": "", "heads": H, "kv_heads": G, "dim": Dm, "vdim": Dm, "scale": 0.25, "kv_from": -1, "v_from_k": 1, "sink": 1, "gated": 3,
         "chunk": 30, "keep_first": 6, "rot_dims": 8, "rot_base": 100.0, "rot_scaling": s.ROT_SCALE_YARN, "rot_factor": 4.0, "rot_low": 1.0, "rot_high": 4.0, "rot_original": 32.0}
    desc = {"vocab": 50, "width": Wd, "eps": 1e-5, "final_norm": 1, "logit_scale": 2.0, "tied_head": 0,
            "layers": [{"style": s.BLOCK_SANDWICH, "norm_kind": s.NORM_RMS, "branches": [x], "ff": 48, "ff_kind": s.FF_GELU} for x in (a, b)]}
    rng = np.random.default_rng(5)
    shapes = {"embed": (50, Wd), "head": (50, Wd), "final.norm": (Wd,)}
    for i in range(2):
        p = f"l{i}."
        vd = V if i == 0 else Dm
        shapes.update({p + "mix.q": (H * Dm, Wd), p + "mix.k": (G * Dm, Wd), p + "mix.o": (Wd, H * vd), p + "mlp.up": (48, Wd), p + "mlp.down": (Wd, 48)})
        shapes.update({p + "norm" + q: (Wd,) for q in ("1", "1b", "2", "2b")})
    shapes.update({"l0.mix.v": (G * V, Wd), "l0.mix.q.b": (H * Dm,), "l0.mix.k.b": (G * Dm,), "l0.mix.v.b": (G * V,), "l0.mix.q.conv": (H * Dm, 3), "l0.mix.k.conv": (G * Dm, 3),
                   "l1.mix.sink": (H,), "l1.mix.g": (H, Wd)})
    t = {k: st.f32_to_bf16_bits((rng.standard_normal(sh) / (np.sqrt(sh[-1]) if len(sh) == 2 and "conv" not in k and k != "embed" else 1.0)).astype(np.float32)) for k, sh in shapes.items()}
    x = toks(7, 90, 50)
    for mode in MODES:
        m = s.SeqModel(desc, s.MODE_BY_NAME[mode], 2, 128).load(t)
        whole = m.step([(0, x)], range(90))
        one = np.concatenate([m.step([(1, x[i:i + 1])], [0]) for i in range(90)])
        assert np.isfinite(whole).all() and rel(one, whole) < TOL[mode]
        first = whole
    desc["logit_scale"] = 1.0
    m = s.SeqModel(desc, s.BF16, 2, 128).load(t)
    assert np.allclose(m.step([(0, x)], range(90)) * 2.0, first, rtol=1e-5, atol=1e-5)


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
    cfg = BI.make_config(vocab=64, width=64, logit_scale=-0.5)      # (a tied head with a positive scale mostly repeats its last token)
    m, W = make(lib, cfg, "float32", seed=41, n_slots=2, gain=2.0)
    prompts = [toks(80 + i, n, 64) for i, n in enumerate((19, 3, 40))]     # three requests, two slots: one waits
    outs = generate(m, prompts, 12, chunk=8, burst=5)
    for p, o in zip(prompts, outs):
        want, margin = oracle_greedy(cfg, W, p, 12)
        assert len(o) == 12
        k = int(np.argmax(o != want)) if np.any(o != want) else 12
        assert k == 12 or margin[k] < 1e-3, (o, want, margin)
        assert len(set(o.tolist())) > 2


def test_device_decode_loop_equals_host_fed_steps(lib):
    """The graph-replayed loop, across a window's edge."""
    cfg = BI.make_config(vocab=64, width=64, logit_scale=-0.5)
    m, _ = make(lib, cfg, "float32", seed=43, n_slots=3, gain=2.0)
    p0, p1 = toks(90, 11, 64), toks(91, 30, 64)
    nxt = m.step_greedy([(0, p0), (1, p1)])
    dev = m.decode([0, 1], 20)
    m.set_option("graph", 0)
    m.reset(0), m.reset(1)
    assert np.array_equal(nxt, m.step_greedy([(0, p0), (1, p1)]))
    assert np.array_equal(dev, m.decode([0, 1], 20))
    m.reset(2)
    cur, host = int(m.step_greedy([(2, p1)])[0]), []
    for _ in range(20):
        cur = int(m.step_greedy([(2, [cur])])[0])
        host.append(cur)
    assert host == dev[1].tolist()
    assert m.position(1) == 30 + 20 and len(set(host)) > 2


def test_a_sequence_that_stops_beside_one_that_goes_on(lib):
    """Sequence 0 samples the end id in the device loop: it repeats that id and its position stays, sequence 1 is not disturbed, and the slot
    starts afresh after a reset (its cache and convolution history were written until it stopped)."""
    cfg = BI.make_config(vocab=64, width=64, logit_scale=-0.5)
    m, W = make(lib, cfg, "float32", seed=44, n_slots=2, gain=2.0)
    p0, p1 = toks(92, 11, 64), toks(93, 30, 64)
    nxt = m.step_greedy([(0, p0), (1, p1)])
    free = m.decode([0, 1], 12)
    eos = next(int(e) for e in free[0] if e not in free[1] and e != nxt[0] and e != nxt[1])
    first = free[0].tolist().index(eos)
    m.reset(0), m.reset(1)
    m.step_greedy([(0, p0), (1, p1)])
    got = m.decode([0, 1], 12, eos)
    assert (got[0][first:] == eos).all() and got[0][:first].tolist() == free[0][:first].tolist() and np.array_equal(got[1], free[1])
    assert m.position(0) == 11 + 1 + first and m.position(1) == 30 + 12
    m.reset(0)
    assert rel(m.step([(0, p1[:9])], range(9)), R.forward(cfg, W, p1[:9])) < TOL["float32"]


def test_missing_and_misshapen_tensors_are_named(lib):
    cfg = BI.make_config(vocab=64, width=64)
    d = BI.describe(cfg)
    t = BI.synth_tensors(d, 0)
    t.pop("l0.mix.o.b")
    with pytest.raises(lib.SeqError, match="l0.mix.o.b"):
        lib.SeqModel(d, lib.F32, 1, 16).load(t)
    t = BI.synth_tensors(d, 0)
    t["l2.mix.k.conv"] = t["l0.mix.k.conv"]            # three taps where the layer has two
    with pytest.raises(lib.SeqError, match="l2.mix.k.conv"):
        lib.SeqModel(d, lib.F32, 1, 16).load(t)
    for extra, like in (("l3.mix.dkv", "l1.mix.dkv"), ("l0.mix.v", "l0.mix.k"), ("head", "embed"), ("l0.norm1.b", "l0.norm1")):
        t = BI.synth_tensors(d, 0)
        t[extra] = t[like]                             # tensors that this design does not have
        with pytest.raises(lib.SeqError, match=extra):
            lib.SeqModel(d, lib.F32, 1, 16).load(t)


def test_command_line_generation_and_trace_replay(lib, tmp_path):
    """bin/generate and bin/trace_run on a checkpoint folder written by the family's own writer."""
    import subprocess
    import sys
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    cfg = BI.make_config(vocab=64, width=64, logit_scale=-0.5)
    t = BI.synth_tensors(BI.describe(cfg), 71, gain=2.0)
    BI.write_checkpoint(tmp_path / "m", cfg, t)
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
    for dtype in ("bfloat16", "float32"):
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
