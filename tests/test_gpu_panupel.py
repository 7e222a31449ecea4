"""GPU tests of the Panupel family: the CUDA engine (through runtime.Model, i.e. the C ABI's infer / state / sampling entry
points and its own step packing) against the plain NumPy restatement in oracle/panupel_numpy.py, on small random models made
here.  precision 1 (every product in f32) is held to a tight bound, precision 0 (bf16 tensor-core products) to the
restatement's own bf16 operand-rounding error.
"""
import json

import numpy as np
import pytest

from ai00_server_b200 import capi, runtime, synth
from oracle import panupel_numpy as P

pytestmark = pytest.mark.gpu

# f32 engine vs float64 oracle, relative to the logits' spread.  Rounding noise of one part in 2^24 on the projections' outputs moves a
# typical row of the restatement by 2e-6 and a rare row (a head whose read-out is nearly zero before it is normalised) by 7e-5.
TIGHT, TYPICAL = 2e-4, 1e-5
L = synth.panupel_layer
A, D = "parallel", "delta"


def row_errs(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt(((want - want.mean(-1, keepdims=True)) ** 2).mean())


def exact(got, want):
    e = row_errs(got, want)
    assert len(e) == len(want) and e.max() <= TIGHT, (e.argmax(), e.max())
    assert len(e) < 20 or np.median(e) <= TYPICAL, np.median(e)


class Bundle:
    def __init__(self, layers, precision=1, slots=3, kv_tokens=2048, kv_page=16, seed=0, chunk=128, tweak=None, **kw):
        self.cfg_bytes, self.st, self.w = synth.make_panupel(layers, seed=seed, **kw)
        self.cfg = json.loads(self.cfg_bytes)
        if tweak:                                   # planted weights: edit the rounded arrays, write them again
            tweak(self.cfg, self.w)
            self.cfg_bytes = json.dumps(self.cfg).encode()
            self.st = synth.pack_st_bf16({k: np.asarray(v, np.float32) for k, v in self.w.items()})
            self.w = {k: v.astype(np.float64) for k, v in P.read_safetensors(bytes(self.st)).items()}
        self.m = runtime.Model(self.st, max_batch=slots, token_chunk_size=chunk, precision=precision, config=self.cfg_bytes,
                               kv_tokens=kv_tokens, kv_page=kv_page)
        self.vocab = self.cfg["vocab"]
        self.runs = len(P.layer_runs(self.cfg))

    def tokens(self, n, seed=0):
        return [int(t) for t in np.random.default_rng(seed).integers(0, self.vocab, n)]

    def oracle(self, toks, layers=False):
        return P.run(self.cfg, self.w, toks, layers=layers)

    def feed(self, slot, toks, opt=capi.OPTION_FULL):
        return self.m.infer_raw([slot], [len(toks)], list(toks), [opt])[0].copy()

    def close(self):
        self.m.close()


def bf16_floor(b, toks, want):
    """How far the restatement itself moves when every projection's activation operand is rounded to bfloat16: the yardstick
    for precision 0, whose tensor-core steps round exactly those operands."""
    P.ROUND_OPERANDS = True
    try:
        return row_errs(b.oracle(toks), want)
    finally:
        P.ROUND_OPERANDS = False


def assert_serving(got, want, floor):
    e = row_errs(got, want)
    assert np.median(e) <= 2.0 * np.median(floor)
    assert (e > 3.0 * floor.max()).sum() <= max(1, 0.02 * len(e))


STACK = [L(D, kv_heads=2, conv=4),
         L(A, kv_heads=2, rot_dims=12, scaling=(8.0, 1.0, 4.0, 64), mm_heads=3),
         L(D, heads=6, kv_heads=3, dim=8, vdim=20, conv=2, ff=None),
         L(A, heads=6, kv_heads=1, dim=20, vdim=12, base=500.0, scaling=(3.0, 0.5, 6.0, 100), mm_heads=1, mm_dim=20, mm_vdim=36, gate_cap=4.0,
           left_scale=0.7, right_scale=-1.3, ff=40)]
STACK_KW = dict(loop=(1, 3, 3))


@pytest.fixture(scope="module")
def stack():
    b = Bundle(STACK, **STACK_KW)
    yield b
    b.close()


@pytest.fixture(scope="module")
def stack_ref(stack):
    toks = stack.tokens(150, 5)
    return toks, stack.oracle(toks)


# ---- each mechanism alone: small models, residual stream after every layer run and logits ----
ATT = dict(right_scale=0.0, ff=None)          # the matrix memory runs, its output counts for nothing
MEM = dict(left_scale=0.0, ff=None)


@pytest.mark.parametrize("layers,kw", [
    ([L(A, kv_heads=2, **ATT)], {"loop": None}),
    ([L(A, kv_heads=1, rot_dims=0, **ATT)], {"loop": None}),
    ([L(A, rot_dims=6, vdim=9, base=30.0, **ATT)], {"loop": None}),
    ([L(A, dim=32, base=2000.0, scaling=(4.0, 1.0, 4.0, 32), **ATT)], {"loop": None}),
    ([L(A, dim=32, base=500000.0, scaling=(16.0, 2.0, 5.0, 300), **ATT)], {"loop": None}),
    ([L(A, **MEM)], {"loop": None}),
    ([L(A, mm_heads=1, mm_dim=5, mm_vdim=30, gate_cap=2.0, **MEM)], {"loop": None}),
    ([L(A, mm_heads=4, mm_dim=33, mm_vdim=7, gate_cap=30.0, **MEM)], {"loop": None}),
    ([L(A, left_scale=-0.4, right_scale=2.0, ff=None)], {"loop": None, "residual_mult": 1.0}),
    ([L(D, ff=None)], {"loop": None}),
    ([L(D, kv_heads=1, conv=1, vdim=5, ff=None)], {"loop": None, "residual_mult": 1.0}),
    ([L(D, kv_heads=2, conv=5, dim=7, vdim=24, ff=None)], {"loop": None}),
    ([L(D, heads=1, dim=40, conv=2, ff=None)], {"loop": None}),
    ([L(D, ff=33)], {"loop": None, "residual_mult": 0.25}),
    ([L(A, ff=20)], {"loop": None, "residual_mult": 1.5, "eps": 1e-3}),
    ([L(D, ff=None), L(A, ff=None)], {"loop": (0, 2, 3)}),
    ([L(D), L(A), L(D)], {"loop": (1, 2, 2)}),
    ([L(A), L(D)], {"loop": (1, 2, 1)}),
    ([L(D), L(A)], {"loop": (0, 1, 4)}),
], ids=["attention", "attention-no-rotation", "attention-partial-rotation", "bands-short-context", "bands-long-context", "memory", "memory-tight-cap",
        "memory-two-parts-per-column", "both-sides", "delta", "delta-one-tap", "delta-five-taps", "delta-one-head", "delta-dense", "parallel-dense",
        "loop-whole-stack", "loop-in-the-middle", "loop-once-at-the-end", "loop-first-layer"])
def test_single_mechanisms(layers, kw):
    b = Bundle(layers, seed=3, **kw)
    try:
        toks = b.tokens(61, 1)
        b.m.debug_read("layers_on", 1)
        got = b.feed(0, toks)
        want, lay = b.oracle(toks, layers=True)
        buf = np.empty(b.runs * 128 * b.cfg["width"], np.float32)
        capi.check(capi.lib().b200rwkv_debug_read(b.m._h, b"layers", capi.ptr(buf), buf.size), b.m._h)
        buf = buf.reshape(b.runs, 128, -1)[:, :len(toks)]
        assert lay.shape[0] == b.runs
        for i in range(b.runs):
            assert np.abs(buf[i] - lay[i]).max() <= 1e-4 * max(1.0, np.abs(lay[i]).max()), i
        exact(got, want)
    finally:
        b.close()


def test_whole_prompt_and_first_tokens(stack, stack_ref):
    toks, want = stack_ref
    stack.m.state.reset(0)
    exact(stack.feed(0, toks), want)
    for n in (1, 2, 3, 4):                                     # sequences shorter than any convolution
        stack.m.state.reset(1)
        exact(stack.feed(1, toks[:n]), want[:n])


def test_prefill_against_token_by_token(stack, stack_ref):
    toks, want = stack_ref
    stack.m.state.reset(0)
    rows = np.concatenate([stack.feed(0, [t], capi.OPTION_LAST) for t in toks])
    exact(rows, want)


@pytest.mark.parametrize("cuts", [[2, 2, 3, 64, 5, 2, 31, 17, 16, 8], [15, 1, 1, 16, 17, 2, 98], [128, 22], [7] * 21 + [3], [1, 2] * 50, [2] * 75])
def test_portions(stack, stack_ref, cuts):
    toks, want = stack_ref
    assert sum(cuts) == len(toks)
    stack.m.state.reset(0)
    out, at = [], 0
    for c in cuts:
        out.append(stack.feed(0, toks[at:at + c]))
        at += c
    exact(np.concatenate(out), want)


def test_unequal_batch_against_each_alone(stack):
    reqs = [stack.tokens(n, 10 + n) for n in (41, 1, 19)]
    want = [stack.oracle(r) for r in reqs]
    for s in range(3):
        stack.m.state.reset(s)
    rows = stack.m.infer_raw([0, 1, 2], [len(r) for r in reqs], [t for r in reqs for t in r], [capi.OPTION_FULL] * 3)
    for r, w in zip(rows, want):
        exact(r, w)
    nxt = [3, 4, 5]                                            # decode all three together: the rows do not depend on the company
    together = stack.m.infer_raw([0, 1, 2], [1, 1, 1], nxt, [capi.OPTION_LAST] * 3)
    for s in range(3):
        exact(together[s], stack.oracle(reqs[s] + [nxt[s]])[-1:])
    # a prompt portion of one sequence beside single tokens of two others
    more = [stack.tokens(9, 77), [6], [7]]
    mixed = stack.m.infer_raw([1, 0, 2], [9, 1, 1], more[0] + more[1] + more[2], [capi.OPTION_FULL, capi.OPTION_LAST, capi.OPTION_LAST])
    exact(mixed[0], stack.oracle(reqs[1] + [nxt[1]] + more[0])[-9:])
    exact(mixed[1], stack.oracle(reqs[0] + [nxt[0]] + more[1])[-1:])
    exact(mixed[2], stack.oracle(reqs[2] + [nxt[2]] + more[2])[-1:])


def test_pages_and_slots_reused():
    b = Bundle(STACK[:3], slots=2, kv_tokens=64, kv_page=8, seed=4, loop=(0, 2, 2))
    try:
        a, c = b.tokens(60, 1), b.tokens(50, 2)
        wa, wc = b.oracle(a), b.oracle(c)
        exact(b.feed(0, a), wa)
        with pytest.raises(capi.B200Error):                    # the pool is for 64 tokens (+ one partly filled page per slot)
            b.feed(1, c)
        b.m.state.reset(1)
        b.m.state.reset(0)                                     # pages go back ...
        exact(b.feed(1, c), wc)                  # ... and are used again by another slot, in another order:
        b.m.state.reset(1)                                     # stale rows, states, maxima and convolution tails must not show
        exact(b.feed(0, c[:9]), wc[:9])
        exact(b.feed(1, a[:33]), wa[:33])        # two live sequences share the pool
        exact(b.feed(0, c[9:40]), wc[9:40])
    finally:
        b.close()


# ---- page borders with peaked softmaxes: one key seen too much, too little or in the wrong place changes the row ----
def sharpen(cfg, w):
    for l in cfg["layers"]:
        if l["type"] == A:
            l["mixer"]["left"]["scale"] *= 8.0
    for k in w:
        if k.endswith("left.sink"):
            w[k] = w[k] * 0.0 + 12.0                            # a sink that counts: about as large as a good score


EDGE_MODELS = [([L(A, heads=2, kv_heads=1, ff=None, right_scale=0.2)], 8),
               ([L(A, heads=4, kv_heads=4, rot_dims=8, scaling=(4.0, 1.0, 4.0, 48), ff=None), L(D)], 16),
               ([L(A, heads=3, kv_heads=1, dim=18, vdim=6, ff=None)], 4)]


@pytest.mark.parametrize("which", range(len(EDGE_MODELS)))
def test_page_borders(which):
    layers, page = EDGE_MODELS[which]
    b = Bundle(layers, kv_page=page, seed=6, loop=(0, len(layers), 2), tweak=sharpen)
    try:
        toks = b.tokens(130, 3)
        want = b.oracle(toks)
        exact(b.feed(0, toks), want)
        out = [b.feed(1, toks[:5])]
        for i in range(5, 100):                                # decoded alone across many page borders
            out.append(b.feed(1, [toks[i]], capi.OPTION_LAST))
        out += [b.feed(1, toks[100:103]), b.feed(1, toks[103:105]), b.feed(1, toks[105:])]
        exact(np.concatenate(out), want)
    finally:
        b.close()


def test_the_sharpened_inputs_matter():
    # the inputs do what the test above needs: a lost key, a key one place off or a lost sink gives other rows altogether
    layers, _ = EDGE_MODELS[0]
    cfgb, st, w = synth.make_panupel(layers, seed=6, loop=(0, 1, 2))
    cfg = json.loads(cfgb)
    sharpen(cfg, w)
    toks = [int(t) for t in np.random.default_rng(3).integers(0, 96, 60)]
    a = P.run(cfg, w, toks)
    ss, rh = P.sink_softmax, P.rotate_half
    try:
        P.sink_softmax = lambda s, sink: ss(s, -1e30)
        nosink = P.run(cfg, w, toks)
        P.sink_softmax = lambda s, sink: np.concatenate([[0.0], ss(s[1:], sink)]) if len(s) > 1 else ss(s, sink)
        lost = P.run(cfg, w, toks)                              # the first key is not seen
        P.sink_softmax = ss
        P.rotate_half = lambda x, pos, f: rh(x, pos + (pos >= 8), f)
        shifted = P.run(cfg, w, toks)                           # positions jump at a page border
    finally:
        P.sink_softmax, P.rotate_half = ss, rh
    assert np.median(row_errs(nosink[8:], a[8:])) > 100 * TIGHT
    assert np.median(row_errs(lost[1:8], a[1:8])) > 100 * TIGHT
    assert np.median(row_errs(shifted[8:], a[8:])) > 100 * TIGHT


def plant_far_key(cfg, w):
    """Every query of layer 0 points along the key of token 1, which stands at position 1 only and outscores every other key,
    near or hundreds of tokens away.  (Entry 0 of every embedding row is the same number, so it can carry a fixed query.)"""
    dk = cfg["layers"][0]["mixer"]["left"]["dim"]
    w["embed"][:, 0] = 2.0
    w["embed"][:, 1] = 0.0
    w["embed"][1, 1] = 8.0
    d = np.zeros(dk)
    d[:3] = (1.0, -2.0, 1.5)
    w["l0.mix.left.q"] *= 0.05
    w["l0.mix.left.q"][:, 0] = d
    w["l0.mix.left.k"] *= 0.2
    w["l0.mix.left.k"][:, 1] = d
    w["l0.mix.left.sink"] *= 0.0


def test_a_far_key_carries_the_row():
    b = Bundle([L(A, heads=1, kv_heads=1, dim=16, rot_dims=0, scale=2.0, right_scale=0.1, ff=None)], seed=11, vocab=8, loop=None, tweak=plant_far_key)
    try:
        toks = [0, 1] + [int(t) for t in np.random.default_rng(1).integers(2, 8, 500)]
        want = b.oracle(toks)
        blind = b.oracle([0, 0] + toks[2:])                    # the inputs do what the test needs: without that key the rows change
        assert (row_errs(blind[10:], want[10:]) > 1000 * TIGHT).mean() > 0.95
        exact(b.feed(0, toks), want)
        b.feed(1, toks[:250], capi.OPTION_NONE)
        rows = np.concatenate([b.feed(1, [t], capi.OPTION_LAST) for t in toks[250:]])
        exact(rows, want[250:])
    finally:
        b.close()


def slow_decay(cfg, w):
    for k in w:
        if k.endswith("mix.A_log"):
            w[k] = w[k] * 0.0 - 9.0
        if k.endswith("right.f.b"):
            w[k] = w[k] * 0.0 + 12.0                            # forget gates within 1e-5 of one
        if k.endswith("right.i.b"):
            w[k] = w[k] * 0.0 - 4.0
        if k.endswith("mix.b"):
            w[k] = w[k] * 0.25
    w["embed"][1] *= 6.0                                        # the token that matters: at position 1 only


@pytest.mark.parametrize("kind", [D, A])
def test_states_carry_the_first_tokens_far(kind):
    layer = L(D, dim=24, vdim=16, ff=None) if kind == D else L(A, left_scale=0.0, mm_dim=24, mm_vdim=16, ff=None)
    b = Bundle([layer], seed=12, vocab=12, loop=None, tweak=slow_decay, residual_mult=1.0)
    try:
        toks = [0, 1] + [int(t) for t in np.random.default_rng(1).integers(2, 12, 400)]
        want = b.oracle(toks)
        blind = b.oracle([0, 2] + toks[2:])
        assert np.median(row_errs(blind[300:], want[300:])) > 10 * TIGHT       # the first tokens still show after 300
        exact(b.feed(0, toks), want)
        b.feed(1, toks[:99], capi.OPTION_NONE)
        rows = np.concatenate([b.feed(1, [t], capi.OPTION_LAST) for t in toks[99:]])
        exact(rows, want[99:])
    finally:
        b.close()


@pytest.mark.parametrize("i_bias,f_bias,cap", [(40.0, 40.0, 15.0), (-40.0, 40.0, 15.0), (40.0, -40.0, 15.0), (-40.0, -40.0, 15.0), (3.0, 0.0, 0.5), (30.0, 3.0, 60.0)])
def test_extreme_gates(i_bias, f_bias, cap):
    # gates at both ends of their range: the running maximum moves, rests at its start, or follows the input gate alone
    def tweak(cfg, w):
        w["l0.mix.right.i.b"] = w["l0.mix.right.i.b"] * 0.0 + i_bias
        w["l0.mix.right.f.b"] = w["l0.mix.right.f.b"] * 0.0 + f_bias

    b = Bundle([L(A, left_scale=0.0, mm_heads=2, gate_cap=cap, ff=None)], seed=13, loop=None, tweak=tweak)
    try:
        toks = b.tokens(120, 2)
        want = b.oracle(toks)
        exact(b.feed(0, toks), want)
        out = [b.feed(1, toks[:40])] + [b.feed(1, [t], capi.OPTION_LAST) for t in toks[40:80]] + [b.feed(1, toks[80:])]
        exact(np.concatenate(out), want)
    finally:
        b.close()


def test_long_decoding(stack):
    toks = stack.tokens(260, 9)
    want = stack.oracle(toks)
    stack.m.state.reset(0)
    out = [stack.feed(0, toks[:60])] + [stack.feed(0, [t], capi.OPTION_LAST) for t in toks[60:]]
    exact(np.concatenate(out), want)


ODD = [L(D, heads=3, kv_heads=3, dim=10, vdim=7, conv=5, ff=10),
       L(A, heads=5, dim=6, vdim=9, rot_dims=4, scaling=(2.0, 1.0, 2.0, 10), mm_heads=3, mm_dim=7, mm_vdim=11, ff=7),
       L(D, heads=1, dim=34, vdim=3, conv=1, ff=None),
       L(A, heads=1, dim=7, vdim=3, rot_dims=2, mm_heads=1, mm_dim=1, mm_vdim=1, ff=9),
       L(A, heads=6, kv_heads=2, dim=6, mm_heads=5, mm_dim=9, mm_vdim=2, left_scale=1.0, right_scale=1.0, ff=None),
       L(D, heads=10, kv_heads=5, dim=9, vdim=5, conv=2, ff=3)]


@pytest.mark.parametrize("precision", [1, 0])
def test_other_sizes(precision):
    b = Bundle(ODD, precision=precision, width=50, vocab=61, seed=7, loop=(2, 5, 2), eps=1e-6, residual_mult=1.0)
    try:
        toks = b.tokens(90, 4)
        want = b.oracle(toks)
        got = np.concatenate([b.feed(0, toks[:70]), b.feed(0, toks[70:72])] + [b.feed(0, [t], capi.OPTION_LAST) for t in toks[72:]])
        if precision == 1:
            exact(got, want)
        else:
            assert_serving(got, want, bf16_floor(b, toks, want))
    finally:
        b.close()


WIDE = [L(D, heads=8, kv_heads=2, dim=64, vdim=64, conv=4, ff=320),
        L(A, heads=8, kv_heads=2, dim=64, scaling=(8.0, 1.0, 4.0, 50), mm_heads=4, mm_dim=64, mm_vdim=128, ff=320),
        L(D, heads=4, kv_heads=4, dim=128, vdim=128, ff=None),
        L(A, heads=4, kv_heads=1, dim=128, mm_heads=2, mm_dim=128, ff=256)]


@pytest.mark.parametrize("precision", [1, 0])
def test_wider_layers(precision):
    b = Bundle(WIDE, precision=precision, width=256, vocab=300, seed=5, loop=(0, 2, 2))
    try:
        toks = b.tokens(140, 6)
        want = b.oracle(toks)
        got = np.concatenate([b.feed(0, toks[:100])] + [b.feed(0, [t], capi.OPTION_LAST) for t in toks[100:120]] + [b.feed(0, toks[120:])])
        if precision == 1:
            exact(got, want)
        else:
            assert_serving(got, want, bf16_floor(b, toks, want))
    finally:
        b.close()


# state sizes around the scan kernels' launch shapes: lanes per column, columns per CTA, one or several CTAs per head (in prompts, in
# decoding, in both), padded key parts, groups of fewer tokens where many lanes share a column
@pytest.mark.parametrize("dk,dv", [(1, 1), (3, 70), (32, 128), (33, 64), (64, 64), (68, 33), (96, 48), (100, 100), (128, 130), (128, 260), (250, 40), (256, 256),
                                   (500, 12), (1024, 5)])
def test_state_shapes(dk, dv):
    layers = [L(D, heads=2, kv_heads=1, dim=dk, vdim=dv, ff=None), L(A, heads=1, dim=4, left_scale=0.1, mm_heads=2, mm_dim=dk, mm_vdim=dv, ff=None)]
    b = Bundle(layers, seed=dk + dv, width=40, vocab=50, kv_page=8, loop=(1, 2, 2))
    try:
        toks = b.tokens(70, 2)
        want = b.oracle(toks)
        exact(b.feed(0, toks), want)
        out = [b.feed(1, toks[:37])] + [b.feed(1, [t], capi.OPTION_LAST) for t in toks[37:50]] + [b.feed(1, toks[50:53]), b.feed(1, toks[53:])]
        exact(np.concatenate(out), want)
    finally:
        b.close()


def test_states_too_tall_are_refused():
    with pytest.raises(capi.B200Error):
        Bundle([L(D, heads=1, dim=1025, vdim=4, ff=None)], width=16, vocab=20, loop=None)


# head counts, head ratios and head sizes around the attention kernel's launch shapes
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(1, 1, 4, 4), (2, 2, 128, 128), (3, 1, 12, 20), (12, 4, 20, 8), (7, 7, 9, 5), (32, 32, 8, 8), (40, 20, 4, 4),
                                                     (24, 1, 16, 12), (16, 16, 64, 32), (2, 1, 136, 72), (4, 2, 32, 160), (2, 1, 256, 256)])
def test_head_shapes(heads, kv_heads, dim, vdim):
    hd = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim)
    layers = [L(A, rot_dims=dim // 2 * 2, ff=None, **hd), L(A, rot_dims=2, **hd)]
    b = Bundle(layers, seed=heads + dim, width=40, vocab=50, kv_page=8, loop=(1, 2, 2))
    try:
        toks = b.tokens(100, 2)
        want = b.oracle(toks)
        exact(b.feed(0, toks), want)
        out = [b.feed(1, toks[:41])] + [b.feed(1, [t], capi.OPTION_LAST) for t in toks[41:80]] + [b.feed(1, toks[80:83]), b.feed(1, toks[83:])]
        exact(np.concatenate(out), want)
    finally:
        b.close()


def random_model(seed):
    """A configuration drawn at random: every size, count and constant of the family varies, layers differ from one another."""
    rng = np.random.default_rng(3000 + seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        ff = pick(None, 8, 24, 33)
        kv = pick(1, 2, 4)
        heads = kv * pick(1, 2, 3, 4)
        if rng.integers(2):
            dim = pick(4, 8, 12, 18, 32, 40)
            layers.append(L(A, heads=heads, kv_heads=kv, dim=dim, vdim=pick(4, 6, 16, dim), rot_dims=pick(0, 2, dim), base=pick(100.0, 10000.0, 5e5),
                            scaling=pick(None, (8.0, 1.0, 4.0, 64), (2.0, 0.5, 8.0, 500)), scale=float(rng.uniform(0.1, 0.6)),
                            mm_heads=pick(1, 2, 3, 8), mm_dim=pick(2, 8, 20, 48), mm_vdim=pick(3, 8, 24, 50), gate_cap=pick(1.0, 5.0, 15.0, 40.0),
                            left_scale=float(rng.uniform(-2, 2)), right_scale=float(rng.uniform(-2, 2)), ff=ff))
        else:
            layers.append(L(D, heads=heads, kv_heads=kv, dim=pick(3, 8, 16, 36, 48), vdim=pick(4, 10, 16, 40), conv=pick(1, 2, 3, 4, 6), ff=ff))
    n = len(layers)
    start = int(rng.integers(0, n))
    loop = pick(None, (start, int(rng.integers(start + 1, n + 1)), pick(1, 2, 3)))
    kw = dict(width=pick(24, 40, 56, 100), vocab=pick(31, 64, 150), loop=loop, residual_mult=float(rng.uniform(0.2, 1.2)), eps=pick(1e-5, 1e-6, 1e-3))
    return layers, kw


@pytest.mark.parametrize("seed", range(10))
def test_random_configurations(seed):
    layers, kw = random_model(seed)
    b = Bundle(layers, seed=seed, kv_page=int(np.random.default_rng(seed).choice([4, 8, 16, 64])), **kw)
    try:
        toks = b.tokens(150, seed)
        want = b.oracle(toks)
        exact(b.feed(0, toks), want)                                        # a prompt of two steps
        out = [b.feed(1, toks[:57]), b.feed(1, toks[57:59])] + [b.feed(1, [t], capi.OPTION_LAST) for t in toks[59:110]] + [b.feed(1, toks[110:])]
        exact(np.concatenate(out), want)                                    # portions, then decoding, then a portion
    finally:
        b.close()


def test_serving_precision(stack_ref):
    toks, want = stack_ref
    b = Bundle(STACK, precision=0, **STACK_KW)
    try:
        floor = bf16_floor(b, toks, want)
        assert_serving(b.feed(0, toks), want, floor)
        b.m.state.reset(0)
        out = [b.feed(0, toks[:50])] + [b.feed(0, [t], capi.OPTION_LAST) for t in toks[50:90]] + [b.feed(0, toks[90:])]
        assert_serving(np.concatenate(out), want, floor)
    finally:
        b.close()


def test_steps_of_up_to_512_tokens_and_long_contexts(stack_ref):
    toks, want = stack_ref
    b = Bundle(STACK, chunk=512, **STACK_KW)
    try:
        long = toks + b.tokens(550, 8)                         # several key tiles per cluster rank, many staged groups, two steps
        ref = b.oracle(long)
        exact(b.feed(0, long), ref)
        b.m.state.reset(0)
        b.feed(0, long[:660], capi.OPTION_NONE)
        rows = np.concatenate([b.feed(0, [t], capi.OPTION_LAST) for t in long[660:]])     # decoding with the keys split over a cluster
        exact(rows, ref[660:])
    finally:
        b.close()


def test_greedy_generation_through_the_runtime(stack):
    # the framework's own entry point: Runtime.infer (its token budget and slot batching) + the GPU sampling front half
    prompt = stack.tokens(21, 12)
    mem = P.new_memory(stack.cfg)
    row = P.run(stack.cfg, stack.w, prompt, mem=mem)[-1]
    want = []
    for _ in range(12):
        want.append(int(row.argmax()))
        row = P.run(stack.cfg, stack.w, [want[-1]], mem=mem)[-1]
    stack.m.state.reset(0)
    inp = runtime.RnnInput([runtime.RnnInputBatch(list(prompt), runtime.RnnOption.Last)], token_chunk_size=8)
    got = []
    while len(got) < 12:
        inp, out = stack.m.runtime.infer(inp)
        if out[0].is_empty():
            continue
        ids, probs = stack.m.sample_topk([0], top_k=4)
        assert int(ids[0, 0]) == int(out[0].data[0].argmax())
        got.append(int(ids[0, 0]))
        inp = runtime.RnnInput([runtime.RnnInputBatch([got[-1]], runtime.RnnOption.Last)], token_chunk_size=8)
    assert got == want


def test_state_snapshots_and_host_round_trip(stack, stack_ref):
    toks, want = stack_ref
    m = stack.m
    m.state.reset(0)
    stack.feed(0, toks[:50], capi.OPTION_LAST)
    snap = m.state.read(0)
    host = m.state.back(0)
    assert int(host.reshape(-1)[0]) == 50
    a = stack.feed(0, toks[50:90])
    m.state.write(snap, 1)                                     # device snapshot into another slot
    b_ = stack.feed(1, toks[50:90])
    m.state.load(host, 2)                                      # host tensor into a third
    c = stack.feed(2, toks[50:90])
    exact(a, want[50:90])
    assert np.array_equal(a, b_) and np.array_equal(a, c)
    snap.free()
