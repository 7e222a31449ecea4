"""GPU tests of the Fufipel family: the CUDA engine (through runtime.Model, i.e. the C ABI's infer / state / sampling entry
points and its own step packing) against the plain NumPy restatement in oracle/fufipel_numpy.py, on small random models made
here.  precision 1 (every product in f32) is held to a tight bound, precision 0 (bf16 tensor-core products) to the
restatement's own bf16 operand-rounding error.
"""
import json

import numpy as np
import pytest

from ai00_server_b200 import capi, runtime, synth
from oracle import fufipel_numpy as F

pytestmark = pytest.mark.gpu

# f32 engine vs float64 oracle, relative to the logits' spread: any row / the median row
TIGHT, TYPICAL = 2e-4, 1e-5
L = synth.fufipel_layer
A, P = "attention", "parallel"


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
        self.cfg_bytes, self.st, self.w = synth.make_fufipel(layers, seed=seed, **kw)
        self.cfg = json.loads(self.cfg_bytes)
        if tweak:                                   # planted weights: edit the rounded arrays, write them again
            tweak(self.cfg, self.w)
            self.cfg_bytes = json.dumps(self.cfg).encode()
            self.st = synth.pack_st_bf16({k: np.asarray(v, np.float32) for k, v in self.w.items()})
            self.w = {k: v.astype(np.float64) for k, v in F.read_safetensors(bytes(self.st)).items()}
        self.m = runtime.Model(self.st, max_batch=slots, token_chunk_size=chunk, precision=precision, config=self.cfg_bytes,
                               kv_tokens=kv_tokens, kv_page=kv_page)
        self.vocab = self.cfg["vocab"]

    def tokens(self, n, seed=0):
        return [int(t) for t in np.random.default_rng(seed).integers(0, self.vocab, n)]

    def oracle(self, toks, layers=False):
        return F.run(self.cfg, self.w, toks, layers=layers)

    def feed(self, slot, toks, opt=capi.OPTION_FULL):
        return self.m.infer_raw([slot], [len(toks)], list(toks), [opt])[0].copy()

    def decode(self, slot, toks):
        return [self.feed(slot, [t], capi.OPTION_LAST) for t in toks]

    def close(self):
        self.m.close()


def bf16_floor(b, toks, want):
    """How far the restatement itself moves when every projection's activation operand is rounded to bfloat16: the yardstick
    for precision 0, whose tensor-core steps round exactly those operands."""
    F.ROUND_OPERANDS = True
    try:
        return row_errs(b.oracle(toks), want)
    finally:
        F.ROUND_OPERANDS = False


def assert_serving(got, want, floor):
    e = row_errs(got, want)
    assert np.median(e) <= 2.0 * np.median(floor)
    assert (e > 3.0 * floor.max()).sum() <= max(1, 0.02 * len(e))


RAMP = (8.0, 16.0, 1.0, 300)
STACK = [L(A, kv_heads=2, window=9, keep_first=3),
         L(P, kv_heads=2, rot_dims=12, scaling=RAMP, gla_heads=3, chunk=13),
         L(A, heads=6, kv_heads=3, dim=8, vdim=20, window=21, keep_first=0, bias_max=17.5, ff=None),
         L(P, heads=6, kv_heads=1, dim=20, vdim=12, base=500.0, scaling=(3.0, 6.0, 0.5, 100), chunk=40, gla_heads=1, gla_dim=20, gla_vdim=36, tau=3.0, ff=40),
         L(A, kv_heads=2, window=30, keep_first=5, bias_max=90, kv_from=0, ff=33)]


@pytest.fixture(scope="module")
def stack():
    b = Bundle(STACK)
    yield b
    b.close()


@pytest.fixture(scope="module")
def stack_ref(stack):
    toks = stack.tokens(150, 5)
    return toks, stack.oracle(toks)


def half_off(side):
    """One half of every parallel layer runs, its output counts for nothing."""
    def tweak(cfg, w):
        for k in w:
            if k.endswith("mix.%s.out" % side):
                w[k] = w[k] * 0.0
    return tweak


# ---- each mechanism alone: small models, residual stream after every layer and logits ----
@pytest.mark.parametrize("layers,kw", [
    ([L(A, ff=None)], {}),
    ([L(A, kv_heads=1, window=1, keep_first=0, ff=None)], {}),
    ([L(A, kv_heads=2, window=5, keep_first=9, vdim=9, ff=None)], {"rel_rows": 2, "residual_mult": 1.0}),
    ([L(A, window=100, keep_first=1, bias_max=11, ff=None)], {"rel_rows": 20}),
    ([L(A, window=12, keep_first=4, bias_max=1000, ff=None), L(A, window=3, keep_first=0, kv_from=0, ff=None)], {"rel_rows": 7}),
    ([L(P, rot_dims=0, ff=None)], {"tweak": half_off("right")}),
    ([L(P, kv_heads=2, rot_dims=6, vdim=9, base=30.0, chunk=1, ff=None)], {"tweak": half_off("right")}),
    ([L(P, kv_heads=1, dim=32, base=2000.0, scaling=(4.0, 8.0, 1.0, 64), chunk=200, ff=None)], {"tweak": half_off("right")}),
    ([L(P, dim=32, base=500000.0, scaling=(16.0, 32.0, 1.0, 4096), chunk=16, scale=1.3, ff=None)], {"tweak": half_off("right")}),
    ([L(P, ff=None)], {"tweak": half_off("left"), "low_rank": 1}),
    ([L(P, gla_heads=1, gla_dim=5, gla_vdim=30, tau=1.0, ff=None)], {"tweak": half_off("left"), "low_rank": 5}),
    ([L(P, gla_heads=4, gla_dim=33, gla_vdim=7, tau=40.0, ff=None)], {"tweak": half_off("left")}),
    ([L(P, ff=None)], {"residual_mult": 1.0, "eps": 1e-3}),
    ([L(A, ff=33)], {"residual_mult": 0.25}),
    ([L(P, ff=20)], {"residual_mult": 1.5, "logit_scale": -0.3}),
    ([L(P, ff=20), L(P, ff=None), L(A, ff=8)], {"bigram": None, "embed_scale": 1.0, "logit_scale": 1.0}),
    ([L(A, ff=20)], {"bigram": (1, 1, 1), "vocab": 50}),
    ([L(A, ff=20)], {"bigram": (1009, 999999937, 999999893), "vocab": 50, "embed_scale": 20.0}),
], ids=["attention", "window-of-one", "more-kept-than-window", "window-beyond-the-prompt", "borrowed-keys", "chunks-no-rotation", "chunks-of-one",
        "ramp-short-context", "ramp-long-context", "gla", "gla-fast-decay", "gla-two-parts-per-column", "both-halves", "attention-ff", "parallel-ff",
        "no-pair-rows", "one-bucket", "large-multipliers"])
def test_single_mechanisms(layers, kw):
    b = Bundle(layers, seed=3, **kw)
    try:
        toks = b.tokens(61, 1)
        b.m.debug_read("layers_on", 1)
        got = b.feed(0, toks)
        want, lay = b.oracle(toks, layers=True)
        n = len(layers)
        buf = np.empty(n * 128 * b.cfg["width"], np.float32)
        capi.check(capi.lib().b200rwkv_debug_read(b.m._h, b"layers", capi.ptr(buf), buf.size), b.m._h)
        buf = buf.reshape(n, 128, -1)[:, :len(toks)]
        for i in range(n):
            assert np.abs(buf[i] - lay[i]).max() <= 1e-4 * max(1.0, np.abs(lay[i]).max()), i
        exact(got, want)
    finally:
        b.close()


def test_whole_prompt_and_first_tokens(stack, stack_ref):
    toks, want = stack_ref
    stack.m.state.reset(0)
    exact(stack.feed(0, toks), want)
    for n in (1, 2, 3, 4):
        stack.m.state.reset(1)
        exact(stack.feed(1, toks[:n]), want[:n])


def test_prefill_against_token_by_token(stack, stack_ref):
    toks, want = stack_ref
    stack.m.state.reset(0)
    exact(np.concatenate(stack.decode(0, toks)), want)


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
    # every sequence's last token is remembered by a mixed step, too
    last = stack.m.infer_raw([2, 0], [1, 2], [8, 9, 10], [capi.OPTION_LAST, capi.OPTION_FULL])
    exact(last[0], stack.oracle(reqs[2] + [nxt[2]] + more[2] + [8])[-1:])
    exact(last[1], stack.oracle(reqs[0] + [nxt[0]] + more[1] + [9, 10])[-2:])


def test_pages_and_slots_reused():
    b = Bundle(STACK, slots=2, kv_tokens=64, kv_page=8, seed=4)
    try:
        a, c = b.tokens(60, 1), b.tokens(50, 2)
        wa, wc = b.oracle(a), b.oracle(c)
        exact(b.feed(0, a), wa)
        with pytest.raises(capi.B200Error):                    # the pool is for 64 tokens (+ one partly filled page per slot)
            b.feed(1, c)
        b.m.state.reset(1)
        b.m.state.reset(0)                                     # pages go back ...
        exact(b.feed(1, c), wc)                  # ... and are used again by another slot, in another order:
        b.m.state.reset(1)                                     # stale rows, states and last tokens must not show
        exact(b.feed(0, c[:9]), wc[:9])
        exact(b.feed(1, a[:33]), wa[:33])        # two live sequences share the pool
        exact(b.feed(0, c[9:40]), wc[9:40])
    finally:
        b.close()


# ---- edges: with peaked softmaxes one key seen too much, too little or in the wrong place changes the row ----
def sharpen(cfg, w):
    for l in cfg["layers"]:
        (l["mixer"] if l["type"] == A else l["mixer"]["left"])["scale"] *= 8.0
    for k in w:
        if k.endswith("mix.rel"):
            w[k] = w[k] * 4.0
            w[k][-2:] += 4.0                                    # far keys count as much as near ones


EDGE_MODELS = [([L(A, heads=2, kv_heads=1, window=24, keep_first=5, bias_max=40, ff=None)], 8),
               ([L(A, heads=4, kv_heads=2, window=33, keep_first=2, bias_max=30), L(P, heads=4, rot_dims=8, scaling=RAMP, chunk=20, ff=None),
                 L(A, heads=4, kv_heads=2, window=7, keep_first=11, kv_from=0)], 16),
               ([L(P, heads=2, kv_heads=1, chunk=32, ff=None), L(P, heads=2, chunk=5)], 8),
               ([L(A, heads=3, kv_heads=1, dim=18, vdim=6, window=10, keep_first=1, ff=None), L(P, heads=3, dim=10, vdim=6, chunk=9)], 4),
               ([L(A, heads=2, kv_heads=1, window=64, keep_first=40, bias_max=200, ff=None), L(A, heads=2, kv_heads=1, window=1, keep_first=1, kv_from=0)], 16)]


@pytest.mark.parametrize("which", range(len(EDGE_MODELS)))
def test_window_chunk_and_page_borders(which):
    layers, page = EDGE_MODELS[which]
    b = Bundle(layers, kv_page=page, seed=6, tweak=sharpen)
    try:
        toks = b.tokens(130, 3)
        want = b.oracle(toks)
        exact(b.feed(0, toks), want)
        out = [b.feed(1, toks[:5])] + b.decode(1, toks[5:100])               # decoded alone across every kind of border
        out += [b.feed(1, toks[100:103]), b.feed(1, toks[103:105]), b.feed(1, toks[105:])]
        exact(np.concatenate(out), want)
    finally:
        b.close()


def test_the_sharpened_inputs_matter():
    # the inputs do what the test above needs: a border one key off, a lost kept token, a bias or a rotation one place off, a wrong
    # previous token, a lost state give other rows altogether
    layers, _ = EDGE_MODELS[1]
    cfgb, st, w = synth.make_fufipel(layers, seed=6)
    cfg = json.loads(cfgb)
    sharpen(cfg, w)
    toks = [int(t) for t in np.random.default_rng(3).integers(0, 96, 90)]
    ref = F.run(cfg, w, toks)
    names = ("window_keys", "chunk_keys", "bucket", "rotate_half", "pair_row", "gla_step")
    orig = {n: getattr(F, n) for n in names}
    wk, ck, bu, rh, pr, gl = (orig[n] for n in names)
    faults = [("window_keys", lambda i, s, k: wk(i, s - 1, k), 40), ("window_keys", lambda i, s, k: wk(i, s + 1, k), 40),
              ("window_keys", lambda i, s, k: wk(i, s, k - 1), 50), ("window_keys", lambda i, s, k: wk(i, s, k + 1), 50),
              ("chunk_keys", lambda i, s: ck(i, s + 1), 25), ("chunk_keys", lambda i, s: ck(i, s)[-5:], 25),
              ("bucket", lambda n, rows, far: bu(max(n - 1, 0), rows, far), 8), ("rotate_half", lambda x, pos, f, m: rh(x, pos + (pos % 20 >= 7), f, m), 20),
              ("rotate_half", lambda x, pos, f, m: rh(x, pos, f, 1.0), 8), ("pair_row", lambda b, p, t: pr(b, (p or 0) + 1, t), 8),
              ("gla_step", lambda S, q, k, v, a: gl(S * 0.0, q, k, v, a), 8)]
    for name, fault, start in faults:
        try:
            setattr(F, name, fault)
            e = row_errs(F.run(cfg, w, toks), ref)
        finally:
            setattr(F, name, orig[name])
        assert (e[start:] > 10 * TIGHT).mean() > 0.25, (name, start, np.median(e[start:]))


def plant_far_key(cfg, w):
    """Every query of layer 0 points along the key of token 1, which stands at position 1 only and outscores every other key
    wherever it is visible.  (Entry 0 of every embedding row is the same number, so it can carry a fixed query.)"""
    m = cfg["layers"][0]["mixer"]
    m, p = (m, "l0.mix.") if cfg["layers"][0]["type"] == A else (m["left"], "l0.mix.left.")
    dk = m["dim"]
    w["embed"][:, 0] = 2.0
    w["embed"][:, 1] = 0.0
    w["embed"][1, 1] = 8.0
    d = np.zeros(dk)
    d[:3] = (1.0, -2.0, 1.5)
    w[p + "q"] *= 0.05
    w[p + "q"][:, 0] = d
    w[p + "k"] *= 0.2
    w[p + "k"][:, 1] = d
    if p + "rel" in w:
        w[p + "rel"] *= 0.3


FAR = [(L(A, heads=1, dim=16, scale=8.0, window=40, keep_first=2, bias_max=300, ff=None), 2, 10 ** 9),        # kept for good
       (L(A, heads=1, dim=16, scale=8.0, window=300, keep_first=1, bias_max=200, ff=None), 2, 301),           # until the window has passed it
       (L(P, heads=1, dim=16, rot_dims=0, scale=2.0, chunk=280, ff=None), 2, 280)]                            # until its chunk ends


@pytest.mark.parametrize("which", range(len(FAR)))
def test_a_far_key_carries_the_row(which):
    layer, lo, hi = FAR[which]
    b = Bundle([layer], seed=11, vocab=8, bigram=None, embed_scale=1.0, tweak=plant_far_key)
    try:
        toks = [0, 1] + [int(t) for t in np.random.default_rng(1).integers(2, 8, 400)]
        want = b.oracle(toks)
        wk, ck = F.window_keys, F.chunk_keys
        try:                                                   # the inputs do what the test needs: that key shows where, and only where, it is seen
            F.window_keys = lambda i, s, k: [j for j in wk(i, s, k) if j != 1 or i == 1]
            F.chunk_keys = lambda i, s: [j for j in ck(i, s) if j != 1 or i == 1]
            blind = b.oracle(toks)
        finally:
            F.window_keys, F.chunk_keys = wk, ck
        far = row_errs(blind, want)
        hi = min(hi, len(toks))
        assert (far[lo:hi] > 50 * TIGHT).mean() > 0.9
        if hi < len(toks):
            assert far[hi:].max() == 0.0
        exact(b.feed(0, toks), want)
        b.feed(1, toks[:250], capi.OPTION_NONE)
        exact(np.concatenate(b.decode(1, toks[250:])), want[250:])
    finally:
        b.close()


def slow_decay(cfg, w):
    for k in w:
        if k.endswith("a2.b"):
            w[k] = w[k] * 0.0 + 9.0                             # decays within 1e-4 of one
        if k.endswith("left.out"):
            w[k] = w[k] * 0.0
    w["embed"][1] *= 6.0                                        # the token that matters: at position 1 only


def test_the_state_carries_the_first_tokens_far():
    b = Bundle([L(P, gla_dim=24, gla_vdim=16, tau=1.0, ff=None)], seed=12, vocab=12, bigram=None, residual_mult=1.0, tweak=slow_decay)
    try:
        toks = [0, 1] + [int(t) for t in np.random.default_rng(1).integers(2, 12, 400)]
        want = b.oracle(toks)
        blind = b.oracle([0, 2] + toks[2:])
        assert np.median(row_errs(blind[300:], want[300:])) > 10 * TIGHT       # the first tokens still show after 300
        exact(b.feed(0, toks), want)
        b.feed(1, toks[:99], capi.OPTION_NONE)
        exact(np.concatenate(b.decode(1, toks[99:])), want[99:])
    finally:
        b.close()


@pytest.mark.parametrize("bias,tau", [(40.0, 16.0), (-40.0, 16.0), (-40.0, 1.0), (0.0, 0.3), (-300.0, 1.0)])
def test_extreme_decays(bias, tau):
    def tweak(cfg, w):
        w["l0.mix.right.a2.b"] = w["l0.mix.right.a2.b"] * 0.0 + bias

    b = Bundle([L(P, tau=tau, ff=None)], seed=13, tweak=tweak)
    try:
        toks = b.tokens(120, 2)
        want = b.oracle(toks)
        exact(b.feed(0, toks), want)
        exact(np.concatenate([b.feed(1, toks[:40])] + b.decode(1, toks[40:80]) + [b.feed(1, toks[80:])]), want)
    finally:
        b.close()


def test_long_decoding(stack):
    toks = stack.tokens(260, 9)
    want = stack.oracle(toks)
    stack.m.state.reset(0)
    exact(np.concatenate([stack.feed(0, toks[:60])] + stack.decode(0, toks[60:])), want)


ODD = [L(P, heads=5, dim=6, vdim=9, rot_dims=4, scaling=(2.0, 4.0, 1.0, 40), chunk=7, gla_heads=3, gla_dim=7, gla_vdim=11, tau=5.0, ff=7),
       L(A, heads=3, kv_heads=3, dim=10, vdim=7, window=11, keep_first=1, bias_max=9, ff=10),
       L(P, heads=1, dim=7, vdim=3, rot_dims=2, chunk=50, gla_heads=1, gla_dim=1, gla_vdim=1, ff=9),
       L(A, heads=1, dim=34, vdim=3, window=2, keep_first=0, ff=None),
       L(P, heads=6, kv_heads=2, dim=6, chunk=3, gla_heads=5, gla_dim=9, gla_vdim=2, ff=None),
       L(A, heads=9, kv_heads=3, dim=10, vdim=7, window=40, keep_first=6, kv_from=1, ff=3)]


@pytest.mark.parametrize("precision", [1, 0])
def test_other_sizes(precision):
    b = Bundle(ODD, precision=precision, width=50, vocab=61, seed=7, eps=1e-6, residual_mult=1.0, rel_rows=6, low_rank=3)
    try:
        toks = b.tokens(90, 4)
        want = b.oracle(toks)
        got = np.concatenate([b.feed(0, toks[:70]), b.feed(0, toks[70:72])] + b.decode(0, toks[72:]))
        if precision == 1:
            exact(got, want)
        else:
            assert_serving(got, want, bf16_floor(b, toks, want))
    finally:
        b.close()


WIDE = [L(A, heads=8, kv_heads=2, dim=64, window=50, keep_first=4, bias_max=60, ff=320),
        L(P, heads=8, kv_heads=2, dim=64, rot_dims=32, scaling=RAMP, chunk=70, gla_heads=4, gla_dim=64, gla_vdim=128, ff=320),
        L(P, heads=4, kv_heads=1, dim=128, chunk=33, gla_heads=2, gla_dim=128, ff=None),
        L(A, heads=8, kv_heads=2, dim=64, window=90, keep_first=0, kv_from=0, ff=256)]


@pytest.mark.parametrize("precision", [1, 0])
def test_wider_layers(precision):
    b = Bundle(WIDE, precision=precision, width=192, vocab=300, seed=5, low_rank=24)
    try:
        toks = b.tokens(140, 6)
        want = b.oracle(toks)
        got = np.concatenate([b.feed(0, toks[:100])] + b.decode(0, toks[100:120]) + [b.feed(0, toks[120:])])
        if precision == 1:
            exact(got, want)
        else:
            assert_serving(got, want, bf16_floor(b, toks, want))
    finally:
        b.close()


# state sizes around the scan kernel's launch shapes: lanes per column, columns per CTA, one or several CTAs per head (in prompts, in
# decoding, in both), padded key parts, groups of fewer tokens where many lanes share a column
@pytest.mark.parametrize("dk,dv", [(1, 1), (3, 70), (32, 128), (33, 64), (64, 64), (68, 33), (96, 48), (100, 100), (128, 130), (128, 260), (250, 40), (256, 256),
                                   (500, 12), (1024, 5)])
def test_state_shapes(dk, dv):
    b = Bundle([L(P, heads=1, dim=4, gla_heads=2, gla_dim=dk, gla_vdim=dv, ff=None)] * 2, seed=dk + dv, width=40, vocab=50, kv_page=8)
    try:
        toks = b.tokens(70, 2)
        want = b.oracle(toks)
        exact(b.feed(0, toks), want)
        exact(np.concatenate([b.feed(1, toks[:37])] + b.decode(1, toks[37:50]) + [b.feed(1, toks[50:53]), b.feed(1, toks[53:])]), want)
    finally:
        b.close()


def test_bad_configurations_are_refused():
    for layers, tweak in [([L(P, heads=1, gla_heads=1, gla_dim=1025, gla_vdim=4, ff=None)], None),
                          ([L(A, ff=None), L(A, dim=8, kv_from=0, ff=None)], None),             # the lender has other sizes
                          ([L(P, ff=None), L(A, kv_from=0, ff=None)], None),                    # the lender is no attention layer
                          ([L(A, ff=None), L(A, kv_from=0, ff=None), L(A, kv_from=1, ff=None)], None),
                          ([L(A, kv_from=0, ff=None)], None),
                          ([L(A, bias_max=3, ff=None)], None),                                  # inside the buckets of their own
                          ([L(A, heads=4, kv_heads=3, ff=None)], None)]:
        with pytest.raises(capi.B200Error):
            Bundle(layers, width=16, vocab=20, tweak=tweak)


# head counts, head ratios and head sizes around the attention kernel's launch shapes
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(1, 1, 4, 4), (2, 2, 128, 128), (3, 1, 12, 20), (12, 4, 20, 8), (7, 7, 9, 5), (32, 32, 8, 8), (40, 20, 4, 4),
                                                     (24, 1, 16, 12), (16, 16, 64, 32), (2, 1, 136, 72), (4, 2, 32, 160), (2, 1, 256, 256)])
def test_head_shapes(heads, kv_heads, dim, vdim):
    hd = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim)
    layers = [L(A, window=37, keep_first=6, bias_max=50, ff=None, **hd), L(P, rot_dims=dim // 2 * 2, chunk=45, **hd), L(A, window=60, keep_first=0, kv_from=0, **hd)]
    b = Bundle(layers, seed=heads + dim, width=40, vocab=50, kv_page=8)
    try:
        toks = b.tokens(100, 2)
        want = b.oracle(toks)
        exact(b.feed(0, toks), want)
        exact(np.concatenate([b.feed(1, toks[:41])] + b.decode(1, toks[41:80]) + [b.feed(1, toks[80:83]), b.feed(1, toks[83:])]), want)
    finally:
        b.close()


def random_model(seed):
    """A configuration drawn at random: every size, count and constant of the family varies, layers differ from one another."""
    rng = np.random.default_rng(4000 + seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    rel_rows = pick(2, 6, 9, 16, 32)
    layers = []
    for _ in range(int(rng.integers(1, 7))):
        ff = pick(None, 8, 24, 33)
        kv = pick(1, 2, 4)
        heads = kv * pick(1, 2, 3, 4)
        dim = pick(4, 8, 12, 18, 32, 40)
        vdim = pick(4, 6, 16, dim)
        scale = float(rng.uniform(0.1, 0.9))
        if rng.integers(2):
            lenders = [i for i, l in enumerate(layers) if l["type"] == A and l["mixer"].get("kv_from") is None]
            kw = dict(window=pick(1, 5, 16, 31, 64, 500), keep_first=pick(0, 1, 4, 33), bias_max=pick(17, 40, 128, 333.0), scale=scale, ff=ff)
            if lenders and rng.integers(2):
                j = pick(*lenders)
                m = layers[j]["mixer"]
                layers.append(L(A, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], kv_from=j, **kw))
            else:
                layers.append(L(A, heads=heads, kv_heads=kv, dim=dim, vdim=vdim, **kw))
        else:
            layers.append(L(P, heads=heads, kv_heads=kv, dim=dim, vdim=vdim, rot_dims=pick(0, 2, dim), base=pick(100.0, 10000.0, 5e5), scale=scale,
                            scaling=pick(None, (8.0, 32.0, 1.0, 512), (2.0, 4.0, 0.5, 60)), chunk=pick(1, 6, 16, 50, 64, 400), gla_heads=pick(1, 2, 3, 8),
                            gla_dim=pick(2, 8, 20, 48), gla_vdim=pick(3, 8, 24, 50), tau=pick(1.0, 4.0, 16.0), ff=ff))
    kw = dict(width=pick(24, 40, 56, 100), vocab=pick(31, 64, 150), residual_mult=float(rng.uniform(0.2, 1.2)), eps=pick(1e-5, 1e-6, 1e-3), rel_rows=rel_rows,
              low_rank=pick(1, 4, 7, 16), embed_scale=pick(1.0, 4.0, 11.5), logit_scale=pick(1.0, 0.25, 3.0), bigram=pick(None, (37, 5, 3), (1000, 31, 77)))
    return layers, kw


@pytest.mark.parametrize("seed", range(12))
def test_random_configurations(seed):
    layers, kw = random_model(seed)
    b = Bundle(layers, seed=seed, kv_page=int(np.random.default_rng(seed).choice([4, 8, 16, 64])), **kw)
    try:
        toks = b.tokens(150, seed)
        want = b.oracle(toks)
        exact(b.feed(0, toks), want)                                        # a prompt of two steps
        out = [b.feed(1, toks[:57]), b.feed(1, toks[57:59])] + b.decode(1, toks[59:110]) + [b.feed(1, toks[110:])]
        exact(np.concatenate(out), want)                                    # portions, then decoding, then a portion
    finally:
        b.close()


def test_serving_precision(stack_ref):
    toks, want = stack_ref
    b = Bundle(STACK, precision=0)
    try:
        floor = bf16_floor(b, toks, want)
        assert_serving(b.feed(0, toks), want, floor)
        b.m.state.reset(0)
        assert_serving(np.concatenate([b.feed(0, toks[:50])] + b.decode(0, toks[50:90]) + [b.feed(0, toks[90:])]), want, floor)
    finally:
        b.close()


def test_steps_of_up_to_512_tokens_and_long_contexts():
    layers = [L(A, kv_heads=2, window=300, keep_first=40, bias_max=400), L(P, kv_heads=2, chunk=350), L(A, kv_heads=2, window=600, keep_first=1, kv_from=0, ff=None)]
    b = Bundle(layers, chunk=512, seed=14)
    try:
        long = b.tokens(700, 8)                                # several key tiles per cluster rank, many staged groups, two steps
        ref = b.oracle(long)
        exact(b.feed(0, long), ref)
        b.m.state.reset(0)
        b.feed(0, long[:660], capi.OPTION_NONE)
        exact(np.concatenate(b.decode(0, long[660:])), ref[660:])            # decoding with the keys split over a cluster
    finally:
        b.close()


def test_greedy_generation_through_the_runtime(stack):
    # the framework's own entry point: Runtime.infer (its token budget and slot batching) + the GPU sampling front half
    prompt = stack.tokens(21, 12)
    mem = F.new_memory(stack.cfg)
    row = F.run(stack.cfg, stack.w, prompt, mem=mem)[-1]
    want = []
    for _ in range(12):
        want.append(int(row.argmax()))
        row = F.run(stack.cfg, stack.w, [want[-1]], mem=mem)[-1]
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
    m.state.write(snap, 1)                                     # device snapshot into another slot (the last token travels along)
    b_ = stack.feed(1, toks[50:90])
    m.state.load(host, 2)                                      # host tensor into a third
    c = stack.feed(2, toks[50:90])
    exact(a, want[50:90])
    assert np.array_equal(a, b_) and np.array_equal(a, c)
    snap.free()
