"""Plain NumPy restatement of the Fufipel decoder: one function per mechanism, token by token, written for clarity.  It
shares no code with the CUDA engine and is test infrastructure only.

Notation: W[out, in] applied as W @ x; `cfg` is the parsed config.json; weights are a dict name -> float64 array.
The embedding row of a token is scaled and a second row, looked up by a hash of (previous token, token), is added.  A layer has one
norm and two sublayers that both read its output,
    h = N1(x);   x <- x + r (Mixer(h) + FF(h))          (r: `residual_mult`; FF may be absent)
Two mixers:
  * attention: norm over the whole query / key projection, no rotation, a learned bias per (distance bucket, head), a sliding window
    that keeps the first tokens, an output gate per entry; a layer may read an earlier layer's keys and values;
  * parallel: rotary softmax attention inside fixed chunks of the sequence beside gated linear attention, each output normed over
    the width, the two averaged.
Feed-forward: W_down (relu(W_gate h) * (W_up h)).  The embedding table is the output matrix.
"""
from __future__ import annotations

import numpy as np

from .kemirax_numpy import bf16_round, read_safetensors  # noqa: F401  (file helpers only)

ROUND_OPERANDS = False      # True: the activation operand of every projection is rounded to bfloat16 first (noise-floor runs)


def lin(W, x):
    return W @ (bf16_round(x) if ROUND_OPERANDS else x)


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softmax(s):
    e = np.exp(s - np.max(s))
    return e / e.sum()


# ----------------------------------------------------------------------------------------------------------------------
# embedding
# ----------------------------------------------------------------------------------------------------------------------
def pair_row(b, prev, token):
    """Row of the pair table; prev None: the sequence's first token."""
    if prev is None:
        return b["buckets"]
    return (prev * b["mul_prev"] + token * b["mul_cur"]) % b["buckets"]


def embedding(cfg, w, prev, token):
    e = cfg["embedding"]
    x = w["embed"][token] * e["scale"]
    if e.get("bigram"):
        x = x + w["bigram"][pair_row(e["bigram"], prev, token)]
    return x


# ----------------------------------------------------------------------------------------------------------------------
# masks: the visible positions of query position i
# ----------------------------------------------------------------------------------------------------------------------
def window_keys(i, size, keep_first):
    return [j for j in range(i + 1) if i - j < size or j < keep_first]


def chunk_keys(i, size):
    return list(range(i // size * size, i + 1))


# ----------------------------------------------------------------------------------------------------------------------
# attention with a distance bias
# ----------------------------------------------------------------------------------------------------------------------
def bucket(n, rows, far):
    """Distances below half the rows have a bucket each; larger ones share buckets evenly spaced in the logarithm up to `far`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(np.floor(np.log(n / half) / np.log(far / half) * (rows - half))))


def attention(w, p, c, eps, h, mem, pos, source):
    """mem: {'k': [[G, dim] per token], 'v': [[G, vdim] per token]}; source: the memory of the layer named by kv_from, or None."""
    H, G, dk, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = rms_norm(lin(w[p + "q"], h), w[p + "q.norm"], eps).reshape(H, dk)       # one norm over all heads together
    if source is None:
        mem["k"].append(rms_norm(lin(w[p + "k"], h), w[p + "k.norm"], eps).reshape(G, dk))
        mem["v"].append(lin(w[p + "v"], h).reshape(G, dv))
        source = mem
    seen = window_keys(pos, c["mask"]["size"], c["mask"].get("keep_first", 0))
    rel = w[p + "rel"]
    row = [bucket(pos - j, rel.shape[0], c["bias_max"]) for j in seen]
    out = np.zeros((H, dv))
    for hd in range(H):
        g = hd // (H // G)
        s = np.array([q[hd] @ source["k"][j][g] for j in seen]) * c["scale"] + rel[row, hd]
        out[hd] = softmax(s) @ np.array([source["v"][j][g] for j in seen])
    return lin(w[p + "o"], out.reshape(-1) * sigmoid(lin(w[p + "g"], h)))


# ----------------------------------------------------------------------------------------------------------------------
# rotary attention inside chunks
# ----------------------------------------------------------------------------------------------------------------------
def frequencies(rot):
    """(angle per token of the dims / 2 pairs, factor on cosine and sine).  With `scaling`, pairs that turn more than `fast` times
    over the original context keep their frequency, those that turn fewer than `slow` times are slowed down by `factor`, with a
    linear ramp over the pair index in between."""
    d = rot["dims"]
    i = np.arange(d // 2, dtype=np.float64)
    f = rot["base"] ** (-2.0 * i / max(d, 1))
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def turning(t):
        return d * np.log(s["original"] / (2.0 * np.pi * t)) / (2.0 * np.log(rot["base"]))

    lo, hi = max(np.floor(turning(s["fast"])), 0.0), min(np.ceil(turning(s["slow"])), d - 1.0)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * np.log(s["factor"]) + 1.0


def rotate_half(x, pos, freq, mag):
    """Entry i turns with entry i + n (n = len(freq)) by pos * freq[i] and is scaled by mag; entries from 2 n on stay."""
    n = len(freq)
    y = np.array(x, np.float64)
    c, s = np.cos(pos * freq) * mag, np.sin(pos * freq) * mag
    y[:n] = x[:n] * c - x[n:2 * n] * s
    y[n:2 * n] = x[n:2 * n] * c + x[:n] * s
    return y


def chunk_attention(w, p, c, h, mem, pos):
    H, G, dk, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    freq, mag = frequencies(c["rot"])
    q = lin(w[p + "q"], h).reshape(H, dk)
    k = lin(w[p + "k"], h).reshape(G, dk)
    mem["k"].append(np.stack([rotate_half(k[g], pos, freq, mag) for g in range(G)]))
    mem["v"].append(lin(w[p + "v"], h).reshape(G, dv))
    seen = chunk_keys(pos, c["mask"]["size"])
    out = np.zeros((H, dv))
    for hd in range(H):
        g = hd // (H // G)
        qr = rotate_half(q[hd], pos, freq, mag)
        s = np.array([qr @ mem["k"][j][g] for j in seen]) * c["scale"]
        out[hd] = softmax(s) @ np.array([mem["v"][j][g] for j in seen])
    return lin(w[p + "o"], out.reshape(-1))


# ----------------------------------------------------------------------------------------------------------------------
# gated linear attention
# ----------------------------------------------------------------------------------------------------------------------
def gla_step(S, q, k, v, alpha):
    """One token of one head: the decay acts on the rows of S (key channels); the read-out sees this token's write."""
    S = alpha[:, None] * S + np.outer(k, v)
    return S, S.T @ q


def gated_linear(w, p, c, eps, h, mem):
    """mem: {'S': [H, dk, dv]}."""
    H, dk, dv = c["heads"], c["dim"], c["vdim"]
    q = lin(w[p + "q"], h).reshape(H, dk) * dk ** -0.5
    k = lin(w[p + "k"], h).reshape(H, dk)
    v = lin(w[p + "v"], h).reshape(H, dv)
    z = lin(w[p + "a2"], lin(w[p + "a1"], h)) + w[p + "a2.b"]
    alpha = np.exp(-np.logaddexp(0.0, -z) / c["tau"]).reshape(H, dk)
    out = np.zeros((H, dv))
    for hd in range(H):
        mem["S"][hd], out[hd] = gla_step(mem["S"][hd], q[hd], k[hd], v[hd], alpha[hd])
    return lin(w[p + "o"], rms_norm(out, w[p + "norm"], eps).reshape(-1) * silu(lin(w[p + "g"], h)))


def parallel(w, p, c, eps, h, mem, pos, source=None):
    a = chunk_attention(w, p + "left.", c["left"], h, mem["left"], pos)
    b = gated_linear(w, p + "right.", c["right"], eps, h, mem["right"])
    return 0.5 * (rms_norm(a, w[p + "left.out"], eps) + rms_norm(b, w[p + "right.out"], eps))


MIXERS = {"attention": attention, "parallel": parallel}


def feed_forward(w, p, h):
    return lin(w[p + "down"], np.maximum(lin(w[p + "gate"], h), 0.0) * lin(w[p + "up"], h))


# ----------------------------------------------------------------------------------------------------------------------
# model
# ----------------------------------------------------------------------------------------------------------------------
def new_layer_memory(layer):
    if layer["type"] == "attention":
        return {"k": [], "v": []}
    r = layer["mixer"]["right"]
    return {"left": {"k": [], "v": []}, "right": {"S": np.zeros((r["heads"], r["dim"], r["vdim"]))}}


def new_memory(cfg):
    return {"pos": 0, "prev": None, "layers": [new_layer_memory(l) for l in cfg["layers"]]}


def step(cfg, w, mem, token, residuals=None):
    """One token through the stack; returns the logits row and advances `mem`."""
    eps, r = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embedding(cfg, w, mem["prev"], token)
    for i, layer in enumerate(cfg["layers"]):
        p, c = "l%d." % i, layer["mixer"]
        h = rms_norm(x, 1.0 + w[p + "norm1"], eps)
        source = mem["layers"][c["kv_from"]] if c.get("kv_from") is not None else None
        y = MIXERS[layer["type"]](w, p + "mix.", c, eps, h, mem["layers"][i], mem["pos"], source)
        if layer.get("mlp"):
            y = y + feed_forward(w, p + "mlp.", h)
        x = x + r * y
        if residuals is not None:
            residuals.append(x.copy())
    mem["pos"] += 1
    mem["prev"] = token
    return lin(w["embed"], rms_norm(x, 1.0 + w["final.norm"], eps)) * cfg["logit_scale"]


def run(cfg, w, toks, layers=False, mem=None):
    """Logits rows [len(toks), vocab] (and, with layers, the residual after every layer [layers, len(toks), width])."""
    mem = mem if mem is not None else new_memory(cfg)
    rows, res = [], []
    for t in toks:
        r = []
        rows.append(step(cfg, w, mem, int(t), r))
        res.append(np.stack(r))
    if layers:
        return np.stack(rows), np.stack(res, 1)
    return np.stack(rows)
