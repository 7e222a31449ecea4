"""CPU tests of the Panupel pieces that need no GPU: the NumPy restatement against independent formulations of the same
mechanisms (batched masked attention over materialised keys / values, the matrix memory as an explicit sum over past tokens, the
delta rule as a product of matrices, a direct convolution, the frequency bands by their defining properties, the loop written out
by hand), invariance of the restatement to how a sequence is cut, the synthetic-model writer, and the host-only model detection
of the C ABI."""
import json

import numpy as np

from ai00_server_b200 import capi, synth
from oracle import panupel_numpy as P

L = synth.panupel_layer


def model(layers, **kw):
    cfgb, st, w = synth.make_panupel(layers, **kw)
    return json.loads(cfgb), st, w


def test_writer_round_trips():
    cfg, st, w = model([L("delta", kv_heads=2), L("parallel", kv_heads=1, ff=None), L("delta")], seed=2, loop=(1, 3, 2))
    back = P.read_safetensors(bytes(st))
    assert set(back) == set(w)
    for k in w:
        assert np.array_equal(back[k], w[k]), k
    assert "l1.norm2" not in w and "l1.norm2b" not in w and "l1.norm1b" in w and "head" in w
    assert w["loop.in"].shape == (64, 128) and w["l1.mix.left.k.norm"].shape == (16,) and w["l1.mix.left.q.norm"].shape == (64,)


def test_frequency_bands():
    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}}
    plain = P.frequencies({"base": 10000.0, "dims": 32})
    assert np.allclose(plain, 10000.0 ** (-np.arange(16) / 16.0))
    f = P.frequencies(rot)
    wave = 2 * np.pi / plain
    short, long = wave < 16.0, wave > 64.0
    mid = ~short & ~long
    assert short.any() and long.any() and mid.any()             # all three bands are there
    assert np.array_equal(f[short], plain[short]) and np.allclose(f[long], plain[long] / 8.0)
    assert np.all(f[mid] < plain[mid]) and np.all(f[mid] > plain[mid] / 8.0)
    assert np.all(np.diff(f) < 0)                               # the blend keeps the order
    # continuous at both ends: a wavelength just inside a band is (nearly) treated as one just outside
    for edge, ratio in ((16.0, 1.0), (64.0, 8.0)):
        base = (edge * (1.0 + 1e-9 * (1 if edge == 16.0 else -1)) / (2 * np.pi)) ** 2      # dims = 4: pair 1 has wavelength 2 pi sqrt(base)
        g = P.frequencies(dict(rot, base=base, dims=4))
        assert abs(g[1] * np.sqrt(base) * ratio - 1.0) < 1e-6


def test_rotation_pairs_halves_and_depends_on_distances_only():
    x = np.arange(1.0, 9.0)
    f = np.array([0.7, 0.05, 0.3])
    y = P.rotate_half(x, 5, f)
    assert np.array_equal(y[6:], x[6:])
    for i in range(3):
        z = complex(x[i], x[i + 3]) * np.exp(1j * 5 * f[i])
        assert abs(y[i] - z.real) < 1e-12 and abs(y[i + 3] - z.imag) < 1e-12
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal(8), rng.standard_normal(8)
    assert abs(P.rotate_half(q, 17, f) @ P.rotate_half(k, 11, f) - P.rotate_half(q, 906, f) @ P.rotate_half(k, 900, f)) < 1e-9


def test_sink_softmax():
    s = np.array([0.3, -1.0, 2.0])
    w = P.sink_softmax(s, 0.5)
    e = np.exp(s)
    assert np.allclose(w, e / (e.sum() + np.exp(0.5))) and w.sum() < 1.0
    assert np.allclose(P.sink_softmax(s, -1e9), e / e.sum())
    assert P.sink_softmax(s, 80.0).sum() < 1e-30


def test_attention_equals_a_batched_form():
    H, G, dk, dv, n, W = 6, 2, 8, 5, 23, 24
    cfg, st, w = model([L("parallel", heads=H, kv_heads=G, dim=dk, vdim=dv, rot_dims=6, base=50.0, scaling=(4.0, 1.0, 3.0, 20), scale=0.9, ff=None)],
                       width=W, seed=1, loop=None)
    c, p = cfg["layers"][0]["mixer"]["left"], "l0.mix.left."
    hs = np.random.default_rng(3).standard_normal((n, W))
    mem = {"k": [], "v": []}
    got = np.array([P.attention(w, p, c, 1e-5, h, mem, t) for t, h in enumerate(hs)])
    rms = lambda u, g: u / np.sqrt((u ** 2).mean(-1, keepdims=True) + 1e-5) * g
    q = rms(hs @ w[p + "q"].T, w[p + "q.norm"]).reshape(n, H, dk)          # over all heads together
    k = rms(hs @ w[p + "k"].T, w[p + "k.norm"]).reshape(n, G, dk)
    v = (hs @ w[p + "v"].T).reshape(n, G, dv)
    ang = np.arange(n)[:, None] * P.frequencies(c["rot"])[None]
    turn = lambda u: np.concatenate([u[..., :3] * np.cos(ang)[:, None] - u[..., 3:6] * np.sin(ang)[:, None],
                                     u[..., 3:6] * np.cos(ang)[:, None] + u[..., :3] * np.sin(ang)[:, None], u[..., 6:]], -1)
    q, k = turn(q), turn(k)
    out = np.zeros((n, H, dv))
    for h in range(H):
        s = np.where(np.tril(np.ones((n, n), bool)), q[:, h] @ k[:, h // 3].T * 0.9, -np.inf)
        e = np.exp(s)
        out[:, h] = e / (e.sum(1, keepdims=True) + np.exp(w[p + "sink"][h])) @ v[:, h // 3]
    gate = 1 / (1 + np.exp(-(hs @ w[p + "g"].T)))                          # one number per head
    want = (out * gate[:, :, None]).reshape(n, -1) @ w[p + "o"].T
    assert np.abs(got - want).max() < 1e-10


def test_matrix_memory_equals_an_explicit_sum():
    H, dk, dv, n, W, cap = 3, 6, 4, 19, 20, 3.0
    cfg, st, w = model([L("parallel", mm_heads=H, mm_dim=dk, mm_vdim=dv, gate_cap=cap, ff=None)], width=W, seed=4, loop=None)
    layer, p = cfg["layers"][0], "l0.mix.right."
    hs = np.random.default_rng(5).standard_normal((n, W)) * 2.0
    mem = P.new_layer_memory(layer)["right"]
    got = np.array([P.matrix_memory(w, p, layer["mixer"]["right"], 1e-5, h, mem, t) for t, h in enumerate(hs)])
    q = (hs @ w[p + "q"].T).reshape(n, H, dk) / np.sqrt(dk)
    k, v = (hs @ w[p + "k"].T).reshape(n, H, dk), (hs @ w[p + "v"].T).reshape(n, H, dv)
    i = cap * np.tanh((hs @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = -np.log1p(np.exp(-cap * np.tanh((hs @ w[p + "f"].T + w[p + "f.b"]) / cap)))
    out, floored = np.zeros((n, H, dv)), 0
    for h in range(H):
        for t in range(n):
            # gate products as plain exponentials of sums; the running maximum only scales numerator and denominator alike, and
            # the state before the first token (zero) carries the sum of all forget gates with a maximum of zero
            a = np.array([np.exp(i[s, h] + f[s + 1:t + 1, h].sum()) for s in range(t + 1)])
            m = max([f[:t + 1, h].sum()] + [i[s, h] + f[s + 1:t + 1, h].sum() for s in range(t + 1)])
            num = (a * (k[:t + 1, h] @ q[t, h])) @ v[:t + 1, h]
            nq = a @ (k[:t + 1, h] @ q[t, h])
            floored += abs(nq) < 1.0
            out[t, h] = num * np.exp(-m) / (max(abs(nq) * np.exp(-m), np.exp(-m)) + 1e-6)
    assert 0 < floored < n * H                                  # both arms of the denominator occur
    y = out / np.sqrt((out ** 2).mean(-1, keepdims=True) + 1e-5)
    want = (y.reshape(n, -1) * w[p + "norm"] / (1 + np.exp(-(hs @ w[p + "g"].T)))) @ w[p + "o"].T
    assert np.abs(got - want).max() < 1e-9


def test_both_sides_are_added_with_their_factors():
    cfg, st, w = model([L("parallel", left_scale=0.7, right_scale=-1.6, ff=None)], seed=5, loop=None)
    layer, h = cfg["layers"][0], np.random.default_rng(0).standard_normal(64)
    m1, m2, m3 = (P.new_layer_memory(layer) for _ in range(3))
    both = P.parallel(w, "l0.mix.", layer["mixer"], 1e-5, h, m1, 0)
    a = P.attention(w, "l0.mix.left.", layer["mixer"]["left"], 1e-5, h, m2["left"], 0)
    b = P.matrix_memory(w, "l0.mix.right.", layer["mixer"]["right"], 1e-5, h, m3["right"], 0)
    assert np.allclose(both, 0.7 * a - 1.6 * b)


def test_delta_rule_equals_a_matrix_product_form():
    H, G, dk, dv, taps, n, W = 4, 2, 5, 3, 3, 17, 20
    cfg, st, w = model([L("delta", heads=H, kv_heads=G, dim=dk, vdim=dv, conv=taps, ff=None)], width=W, seed=6, loop=None)
    layer, p = cfg["layers"][0], "l0.mix."
    hs = np.random.default_rng(7).standard_normal((n, W))
    mem = P.new_layer_memory(layer)
    got = np.array([P.delta(w, p, layer["mixer"], 1e-5, h, mem, t) for t, h in enumerate(hs)])
    silu = lambda z: z / (1 + np.exp(-z))

    def conv(name):
        u, cw = hs @ w[p + name].T, w[p + name + ".conv"]
        return silu(np.stack([sum(cw[:, j] * (u[t - taps + 1 + j] if t - taps + 1 + j >= 0 else 0.0) for j in range(taps)) for t in range(n)]))

    unit = lambda u: u / np.sqrt((u ** 2).sum(-1, keepdims=True) + 1e-6)
    q, k, v = unit(conv("q").reshape(n, G, dk)) / np.sqrt(dk), unit(conv("k").reshape(n, G, dk)), conv("v").reshape(n, H, dv)
    beta = 1 / (1 + np.exp(-(hs @ w[p + "b"].T)))
    g = np.exp(-np.exp(w[p + "A_log"]) * np.log1p(np.exp(hs @ w[p + "a"].T + w[p + "dt_bias"])))
    out = np.zeros((n, H, dv))
    for h in range(H):
        S = np.zeros((dk, dv))
        for t in range(n):
            kk = k[t, h // 2]
            S = (np.eye(dk) - beta[t, h] * np.outer(kk, kk)) @ (g[t, h] * S) + beta[t, h] * np.outer(kk, v[t, h])
            out[t, h] = S.T @ q[t, h // 2]
    y = out / np.sqrt((out ** 2).mean(-1, keepdims=True) + 1e-5) * w[p + "norm"]
    want = (y * silu(hs @ w[p + "g"].T).reshape(n, H, dv)).reshape(n, -1) @ w[p + "o"].T
    assert np.abs(got - want).max() < 1e-10


def test_layer_runs_and_the_loop_written_out():
    cfg, st, w = model([L("delta", ff=None), L("parallel"), L("delta")], seed=8, loop=(1, 3, 2), residual_mult=0.3)
    assert P.layer_runs(cfg) == [(0, False), (1, True), (2, False), (1, True), (2, False)]
    cfg0 = dict(cfg)
    del cfg0["loop"]
    assert P.layer_runs(cfg0) == [(0, False), (1, False), (2, False)]
    assert P.layer_runs(dict(cfg, loop={"start": 0, "stop": 3, "times": 1})) == [(0, True), (1, False), (2, False)]
    eps, x0 = cfg["norm"]["eps"], w["embed"][5]
    mems = [P.new_layer_memory(cfg["layers"][i]) for i in (0, 1, 2, 1, 2)]
    rms = lambda u, g: u / np.sqrt((u * u).mean() + eps) * g

    def lay(x, i, mem):
        c, q = cfg["layers"][i], "l%d." % i
        x = x + 0.3 * rms(P.MIXERS[c["type"]](w, q + "mix.", c["mixer"], eps, rms(x, w[q + "norm1"]), mem, 0), w[q + "norm1b"])
        if c["mlp"]:
            h = rms(x, w[q + "norm2"])
            a = w[q + "mlp.gate"] @ h
            x = x + 0.3 * rms(w[q + "mlp.down"] @ (a / (1 + np.exp(-a)) * (w[q + "mlp.up"] @ h)), w[q + "norm2b"])
        return x

    opens = lambda x: w["loop.in"][:, :64] @ x + w["loop.in"][:, 64:] @ x0       # the residual's half of the matrix comes first
    x = lay(x0, 0, mems[0])
    x = lay(lay(opens(x), 1, mems[1]), 2, mems[2])
    x = lay(lay(opens(x), 1, mems[3]), 2, mems[4])
    assert np.abs(P.run(cfg, w, [5])[0] - w["head"] @ rms(x, w["final.norm"])).max() < 1e-10


def test_sequence_memory_makes_the_cut_irrelevant():
    cfg, st, w = model([L("delta", kv_heads=2), L("parallel", kv_heads=2)], seed=9, loop=(0, 2, 2))
    toks = [int(t) for t in np.random.default_rng(0).integers(0, 96, 30)]
    whole = P.run(cfg, w, toks)
    mem = P.new_memory(cfg)
    parts = [P.run(cfg, w, toks[a:b], mem=mem) for a, b in ((0, 7), (7, 8), (8, 30))]
    assert np.array_equal(np.concatenate(parts), whole)


def test_model_detection_and_info_without_a_gpu():
    for layers in ([L("delta"), L("parallel")], [L("parallel", ff=None)]):
        cfg, st, w = model(layers, width=40, vocab=77)
        info = capi.info_from_st(st)
        assert info["version"] == capi.ARCH_PANUPEL and info["num_layer"] == len(layers) and info["num_emb"] == 40 and info["num_vocab"] == 77
