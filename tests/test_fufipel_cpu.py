"""CPU tests of the Fufipel pieces that need no GPU: the NumPy restatement against independent formulations of the same
mechanisms (batched masked attention over materialised keys / values with a bias matrix, gated linear attention as an explicit
sum over past tokens, the frequency ramp by its defining properties, buckets by a search, the embedding hash by hand), invariance
of the restatement to how a sequence is cut, the synthetic-model writer, and the host-only model detection of the C ABI."""
import json

import numpy as np

from ai00_server_b200 import capi, synth
from oracle import fufipel_numpy as F

L = synth.fufipel_layer


def model(layers, **kw):
    cfgb, st, w = synth.make_fufipel(layers, **kw)
    return json.loads(cfgb), st, w


def test_writer_round_trips():
    cfg, st, w = model([L("attention", kv_heads=2), L("parallel", kv_heads=1, ff=None), L("attention", kv_heads=2, kv_from=0)], seed=2)
    back = F.read_safetensors(bytes(st))
    assert set(back) == set(w)
    for k in w:
        assert np.array_equal(back[k], w[k]), k
    assert "head" not in w and "l1.mlp.gate" not in w and "l2.mix.k" not in w and "l2.mix.k.norm" not in w and "l2.mix.q.norm" in w
    assert w["bigram"].shape == (62, 64) and w["l0.mix.k.norm"].shape == (32,) and w["l0.mix.rel"].shape == (12, 4)


def test_pair_rows():
    b = {"buckets": 7, "mul_prev": 3, "mul_cur": 5}
    assert F.pair_row(b, None, 4) == 7                          # the last row is the first token's alone
    assert F.pair_row(b, 0, 0) == 0 and F.pair_row(b, 2, 3) == 0 and F.pair_row(b, 3, 2) == 5
    assert {F.pair_row(b, p, t) for p in range(20) for t in range(20)} == set(range(7))
    cfg, st, w = model([L("attention")], seed=1, embed_scale=2.5)
    assert np.allclose(F.embedding(cfg, w, None, 9), 2.5 * w["embed"][9] + w["bigram"][61])
    assert np.allclose(F.embedding(cfg, w, 30, 9), 2.5 * w["embed"][9] + w["bigram"][(30 * 17 + 9 * 5) % 61])
    cfg0, st0, w0 = model([L("attention")], seed=1, embed_scale=2.5, bigram=None)
    assert np.allclose(F.embedding(cfg0, w0, 30, 9), 2.5 * w0["embed"][9])


def test_visible_keys():
    assert F.window_keys(0, 1, 0) == [0] and F.window_keys(9, 1, 0) == [9]
    assert F.window_keys(9, 3, 2) == [0, 1, 7, 8, 9]
    assert F.window_keys(4, 3, 2) == [0, 1, 2, 3, 4]            # kept tokens and window touch
    assert F.window_keys(5, 3, 7) == list(range(6))             # more kept tokens than there are
    assert F.chunk_keys(9, 5) == [5, 6, 7, 8, 9] and F.chunk_keys(10, 5) == [10] and F.chunk_keys(3, 1) == [3]


def test_frequency_ramp():
    plain, one = F.frequencies({"base": 20000.0, "dims": 32})
    assert one == 1.0 and np.allclose(plain, 20000.0 ** (-np.arange(16) / 16.0))
    f, mag = F.frequencies({"base": 20000.0, "dims": 32, "scaling": {"factor": 4.0, "fast": 8.0, "slow": 1.0, "original": 256}})
    assert abs(mag - (1.0 + np.log(4.0) / 10.0)) < 1e-12
    turns = 256 * plain / (2 * np.pi)                           # turns of every pair over the original context
    keep = (f - plain / 4.0) / (plain - plain / 4.0)            # 1: unchanged, 0: slowed down by the whole factor
    assert np.all(keep[turns > 8.0] == 1.0)
    assert np.allclose(keep[np.nonzero(turns < 1.0)[0][1:]], 0.0)          # the ramp ends on the next whole dimension
    mid = keep[(keep > 1e-9) & (keep < 1 - 1e-9)]
    assert len(mid) >= 2 and np.all(np.diff(mid) < 0)
    assert np.allclose(np.diff(mid), mid[1] - mid[0])           # linear in the pair index
    q, k = np.random.default_rng(0).standard_normal((2, 40))
    a = F.rotate_half(q, 17, f, mag) @ F.rotate_half(k, 11, f, mag)
    assert abs(a - F.rotate_half(q, 906, f, mag) @ F.rotate_half(k, 900, f, mag)) < 1e-9
    assert np.array_equal(F.rotate_half(q, 5, f, mag)[32:], q[32:])        # the rest passes without the factor too


def test_buckets():
    for rows, far in ((12, 40), (16, 200.0), (2, 3), (32, 128), (6, 3.5)):
        half = rows // 2
        edges = [half * (far / half) ** (i / (rows - half)) for i in range(rows - half)]
        got = [F.bucket(n, rows, far) for n in range(500)]
        assert got[:half] == list(range(half)) and got[-1] == rows - 1 and all(b >= a for a, b in zip(got, got[1:]))
        for n in range(half, 500):
            if min(abs(n - e) for e in edges) > 1e-9:
                assert got[n] == half - 1 + sum(n >= e for e in edges), (rows, far, n)


def rms(u, g):
    return u / np.sqrt((u ** 2).mean(-1, keepdims=True) + 1e-5) * g


def test_attention_equals_a_batched_form():
    H, G, dk, dv, n, W, win, keep = 6, 2, 8, 5, 33, 24, 7, 3
    hd = dict(heads=H, kv_heads=G, dim=dk, vdim=dv, ff=None)
    cfg, st, w = model([L("attention", window=4, **hd), L("attention", window=win, keep_first=keep, bias_max=15, scale=0.9, kv_from=0, **hd)], width=W, seed=1)
    hs = np.random.default_rng(3).standard_normal((2, n, W))
    mem = {"k": [], "v": []}
    for t in range(n):                                          # the lender's keys and values, made from its own input
        F.attention(w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5, hs[0, t], mem, t, None)
    c, p = cfg["layers"][1]["mixer"], "l1.mix."
    got = np.array([F.attention(w, p, c, 1e-5, h, {}, t, mem) for t, h in enumerate(hs[1])])
    q = rms(hs[1] @ w[p + "q"].T, w[p + "q.norm"]).reshape(n, H, dk)       # over all heads together
    k = rms(hs[0] @ w["l0.mix.k"].T, w["l0.mix.k.norm"]).reshape(n, G, dk)
    v = (hs[0] @ w["l0.mix.v"].T).reshape(n, G, dv)
    i, j = np.arange(n)[:, None], np.arange(n)[None]
    vis = (j <= i) & ((i - j < win) | (j < keep))
    row = np.array([[F.bucket(max(a - b, 0), 12, 15) for b in range(n)] for a in range(n)])
    out = np.zeros((n, H, dv))
    for h in range(H):
        e = np.where(vis, np.exp(q[:, h] @ k[:, h // 3].T * 0.9 + w[p + "rel"][row, h]), 0.0)
        out[:, h] = e / e.sum(1, keepdims=True) @ v[:, h // 3]
    gate = 1 / (1 + np.exp(-(hs[1] @ w[p + "g"].T)))
    assert np.abs(got - (out.reshape(n, -1) * gate) @ w[p + "o"].T).max() < 1e-10


def test_chunk_attention_equals_a_batched_form():
    H, G, dk, dv, n, W, chunk = 6, 3, 8, 5, 29, 24, 6
    cfg, st, w = model([L("parallel", heads=H, kv_heads=G, dim=dk, vdim=dv, rot_dims=6, base=50.0, scaling=(4.0, 3.0, 1.0, 20), scale=0.9, chunk=chunk, ff=None)],
                       width=W, seed=1)
    c, p = cfg["layers"][0]["mixer"]["left"], "l0.mix.left."
    hs = np.random.default_rng(3).standard_normal((n, W))
    mem = {"k": [], "v": []}
    got = np.array([F.chunk_attention(w, p, c, h, mem, t) for t, h in enumerate(hs)])
    f, mag = F.frequencies(c["rot"])
    z = mag * np.exp(1j * np.arange(n)[:, None] * f)[:, None]              # the rotation as a complex product
    def turn(u):
        r = (u[..., :3] + 1j * u[..., 3:6]) * z
        return np.concatenate([r.real, r.imag, u[..., 6:]], -1)
    q, k = turn((hs @ w[p + "q"].T).reshape(n, H, dk)), turn((hs @ w[p + "k"].T).reshape(n, G, dk))
    v = (hs @ w[p + "v"].T).reshape(n, G, dv)
    i, j = np.arange(n)[:, None], np.arange(n)[None]
    out = np.zeros((n, H, dv))
    for h in range(H):
        e = np.where((j <= i) & (i // chunk == j // chunk), np.exp(q[:, h] @ k[:, h // 2].T * 0.9), 0.0)
        out[:, h] = e / e.sum(1, keepdims=True) @ v[:, h // 2]
    assert np.abs(got - out.reshape(n, -1) @ w[p + "o"].T).max() < 1e-10


def test_gated_linear_attention_equals_an_explicit_sum():
    H, dk, dv, n, W, tau = 3, 6, 4, 19, 20, 2.5
    cfg, st, w = model([L("parallel", gla_heads=H, gla_dim=dk, gla_vdim=dv, tau=tau, ff=None)], width=W, seed=4)
    layer, p = cfg["layers"][0], "l0.mix.right."
    hs = np.random.default_rng(5).standard_normal((n, W))
    mem = F.new_layer_memory(layer)["right"]
    got = np.array([F.gated_linear(w, p, layer["mixer"]["right"], 1e-5, h, mem) for h in hs])
    q, k = (hs @ w[p + "q"].T).reshape(n, H, dk) / np.sqrt(dk), (hs @ w[p + "k"].T).reshape(n, H, dk)
    v = (hs @ w[p + "v"].T).reshape(n, H, dv)
    alpha = (1 / (1 + np.exp(-((hs @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"])))) ** (1 / tau)
    alpha = alpha.reshape(n, H, dk)
    out = np.zeros((n, H, dv))
    for t in range(n):
        for s in range(t + 1):
            out[t] += np.einsum("hk,hk,hk,hv->hv", q[t], np.prod(alpha[s + 1:t + 1], 0), k[s], v[s])
    g = hs @ w[p + "g"].T
    want = (rms(out, w[p + "norm"]).reshape(n, -1) * g / (1 + np.exp(-g))) @ w[p + "o"].T
    assert np.abs(got - want).max() < 1e-10


def test_a_stack_written_out():
    cfg, st, w = model([L("parallel", ff=30), L("attention", ff=None)], seed=8, residual_mult=0.3, logit_scale=-2.0, embed_scale=1.7)
    x = 1.7 * w["embed"][5] + w["bigram"][61]
    one = lambda u, name: rms(u, 1 + w[name])
    h = one(x, "l0.norm1")
    m, c = F.new_layer_memory(cfg["layers"][0]), cfg["layers"][0]["mixer"]
    a = F.chunk_attention(w, "l0.mix.left.", c["left"], h, m["left"], 0)
    b = F.gated_linear(w, "l0.mix.right.", c["right"], 1e-5, h, m["right"])
    ff = w["l0.mlp.down"] @ (np.maximum(w["l0.mlp.gate"] @ h, 0) * (w["l0.mlp.up"] @ h))
    x = x + 0.3 * ((rms(a, w["l0.mix.left.out"]) + rms(b, w["l0.mix.right.out"])) / 2 + ff)
    x = x + 0.3 * F.attention(w, "l1.mix.", cfg["layers"][1]["mixer"], 1e-5, one(x, "l1.norm1"), {"k": [], "v": []}, 0, None)
    assert np.abs(F.run(cfg, w, [5])[0] - -2.0 * (w["embed"] @ one(x, "final.norm"))).max() < 1e-10


def test_sequence_memory_makes_the_cut_irrelevant():
    cfg, st, w = model([L("attention", kv_heads=2), L("parallel", kv_heads=2), L("attention", kv_heads=2, kv_from=0)], seed=9)
    toks = [int(t) for t in np.random.default_rng(0).integers(0, 96, 30)]
    whole = F.run(cfg, w, toks)
    mem = F.new_memory(cfg)
    parts = [F.run(cfg, w, toks[a:b], mem=mem) for a, b in ((0, 7), (7, 8), (8, 30))]
    assert np.array_equal(np.concatenate(parts), whole)


def test_model_detection_and_info_without_a_gpu():
    for layers in ([L("attention"), L("parallel")], [L("parallel", ff=None)]):
        cfg, st, w = model(layers, width=40, vocab=77)
        info = capi.info_from_st(st)
        assert info["version"] == capi.ARCH_FUFIPEL and info["num_layer"] == len(layers) and info["num_emb"] == 40 and info["num_vocab"] == 77
