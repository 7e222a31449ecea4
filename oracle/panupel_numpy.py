"""Plain NumPy restatement of the Panupel decoder: one function per mechanism, token by token, written for clarity.  It
shares no code with the CUDA engine and is test infrastructure only.

Notation: W[out, in] applied as W @ x; `cfg` is the parsed config.json; weights are a dict name -> float64 array.
A model is a stack of blocks with a norm on both sides of every sublayer,
    x <- x + r N1b(Mixer(N1(x)));   x <- x + r N2b(FF(N2(x)))          (r: `residual_mult`)
A run of consecutive layers (`loop`) is executed several times with the same tensors and a memory of its own per pass; every
pass begins by replacing the residual with a projection of the residual and the token's embedding row.  Two mixers:
  * parallel: softmax attention (query / key norm over the whole projection, rotation with stretched low frequencies, a sink term
    per head, one output gate per head) beside a matrix memory with exponential gates kept in range by a running maximum; both
    read the same input and their outputs are added with two constants;
  * delta: the gated delta rule with one decay per head, behind short causal convolutions.
Feed-forward: W_down (silu(W_gate h) * (W_up h)), or none.
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


def softplus(z):
    return np.logaddexp(0.0, z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


# ----------------------------------------------------------------------------------------------------------------------
# attention side
# ----------------------------------------------------------------------------------------------------------------------
def frequencies(rot):
    """Angles per token of the dims / 2 pairs.  With `scaling`: wavelengths up to original / high keep their frequency, those
    beyond original / low are stretched by `factor`, in between the two are blended linearly in original / wavelength."""
    n = rot["dims"] // 2
    f = np.array([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(n)])
    s = rot.get("scaling")
    if not s:
        return f
    out = np.empty(n)
    for i in range(n):
        wave = 2.0 * np.pi / f[i]
        if wave < s["original"] / s["high"]:
            out[i] = f[i]
        elif wave > s["original"] / s["low"]:
            out[i] = f[i] / s["factor"]
        else:
            keep = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out[i] = (1.0 - keep) * f[i] / s["factor"] + keep * f[i]
    return out


def rotate_half(x, pos, freq):
    """Entry i turns with entry i + n (n = len(freq)) by pos * freq[i]; entries from 2 n on stay."""
    n = len(freq)
    y = np.array(x, np.float64)
    c, s = np.cos(pos * freq), np.sin(pos * freq)
    y[:n] = x[:n] * c - x[n:2 * n] * s
    y[n:2 * n] = x[n:2 * n] * c + x[:n] * s
    return y


def sink_softmax(scores, sink):
    """Weights of the keys when the denominator holds one more term exp(sink) that belongs to no key."""
    m = max(float(np.max(scores)), float(sink))
    e = np.exp(scores - m)
    return e / (e.sum() + np.exp(sink - m))


def attention(w, p, c, eps, h, mem, pos):
    """mem: {'k': [[G, dim] per token], 'v': [[G, vdim] per token]}."""
    H, G, dk, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    freq = frequencies(c["rot"])
    q = rms_norm(lin(w[p + "q"], h), w[p + "q.norm"], eps).reshape(H, dk)      # one norm over all heads together
    k = rms_norm(lin(w[p + "k"], h), w[p + "k.norm"], eps).reshape(G, dk)
    mem["k"].append(np.stack([rotate_half(k[g], pos, freq) for g in range(G)]))
    mem["v"].append(lin(w[p + "v"], h).reshape(G, dv))
    gate = sigmoid(lin(w[p + "g"], h))
    out = np.zeros((H, dv))
    for hd in range(H):
        g = hd // (H // G)
        qr = rotate_half(q[hd], pos, freq)
        s = np.array([qr @ kk[g] for kk in mem["k"]]) * c["scale"]
        out[hd] = sink_softmax(s, w[p + "sink"][hd]) @ np.array([v[g] for v in mem["v"]]) * gate[hd]
    return lin(w[p + "o"], out.reshape(-1))


# ----------------------------------------------------------------------------------------------------------------------
# matrix memory side
# ----------------------------------------------------------------------------------------------------------------------
def matrix_memory_step(S, n, m, q, k, v, i_log, f_log):
    """One token of one head: S [dk, dv], n [dk], running maximum m -> (S, n, m, read-out [dv])."""
    m_new = max(f_log + m, i_log)
    keep, add = np.exp(f_log + m - m_new), np.exp(i_log - m_new)
    S = keep * S + add * np.outer(k, v)
    n = keep * n + add * k
    return S, n, m_new, S.T @ q / (max(abs(n @ q), np.exp(-m_new)) + 1e-6)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def matrix_memory(w, p, c, eps, h, mem, pos):
    """mem: {'S': [H, dk, dv], 'n': [H, dk], 'm': [H]}; everything starts at zero, the running maximum too."""
    H, dk, dv = c["heads"], c["dim"], c["vdim"]
    q = lin(w[p + "q"], h).reshape(H, dk) * dk ** -0.5
    k = lin(w[p + "k"], h).reshape(H, dk)
    v = lin(w[p + "v"], h).reshape(H, dv)
    i_log = soft_cap(lin(w[p + "i"], h) + w[p + "i.b"], c["gate_cap"])
    f_log = log_sigmoid(soft_cap(lin(w[p + "f"], h) + w[p + "f.b"], c["gate_cap"]))
    out = np.zeros((H, dv))
    for hd in range(H):
        mem["S"][hd], mem["n"][hd], mem["m"][hd], out[hd] = matrix_memory_step(
            mem["S"][hd], mem["n"][hd], mem["m"][hd], q[hd], k[hd], v[hd], i_log[hd], f_log[hd])
    y = unit_rms(out, eps).reshape(-1) * w[p + "norm"] * sigmoid(lin(w[p + "g"], h))
    return lin(w[p + "o"], y)


def parallel(w, p, c, eps, h, mem, pos):
    return (c["left_scale"] * attention(w, p + "left.", c["left"], eps, h, mem["left"], pos)
            + c["right_scale"] * matrix_memory(w, p + "right.", c["right"], eps, h, mem["right"], pos))


# ----------------------------------------------------------------------------------------------------------------------
# gated delta rule
# ----------------------------------------------------------------------------------------------------------------------
def short_conv(taps_w, history):
    """taps_w [C, taps]; history: the last `taps` inputs, oldest first (zeros before the start of the sequence)."""
    return sum(taps_w[:, j] * history[j] for j in range(taps_w.shape[1]))


def unit_length(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_step(S, q, k, v, g, beta):
    """One token of one head: decay, write what the memory does not yet say about k, read (the read sees the write)."""
    S = g * S
    S = S + np.outer(k, beta * (v - S.T @ k))
    return S, S.T @ q


def delta(w, p, c, eps, h, mem, pos):
    """mem: {'S': [H, dk, dv], 'q' / 'k' / 'v': lists of the last inputs of the three convolutions}."""
    H, G, dk, dv, taps = c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["conv"]
    u = {}
    for name in "qkv":
        mem[name].append(lin(w[p + name], h))
        del mem[name][:-taps]
        pad = [np.zeros_like(mem[name][-1])] * (taps - len(mem[name]))
        u[name] = silu(short_conv(w[p + name + ".conv"], pad + mem[name]))
    q = unit_length(u["q"].reshape(G, dk)) * dk ** -0.5
    k = unit_length(u["k"].reshape(G, dk))
    v = u["v"].reshape(H, dv)
    beta = sigmoid(lin(w[p + "b"], h))
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(lin(w[p + "a"], h) + w[p + "dt_bias"]))
    out = np.zeros((H, dv))
    for hd in range(H):
        r = hd // (H // G)
        mem["S"][hd], out[hd] = delta_step(mem["S"][hd], q[r], k[r], v[hd], g[hd], beta[hd])
    y = rms_norm(out, w[p + "norm"], eps) * silu(lin(w[p + "g"], h)).reshape(H, dv)
    return lin(w[p + "o"], y.reshape(-1))


MIXERS = {"parallel": parallel, "delta": delta}


def new_layer_memory(layer):
    c = layer["mixer"]
    if layer["type"] == "delta":
        return {"S": np.zeros((c["heads"], c["dim"], c["vdim"])), "q": [], "k": [], "v": []}
    r = c["right"]
    return {"left": {"k": [], "v": []},
            "right": {"S": np.zeros((r["heads"], r["dim"], r["vdim"])), "n": np.zeros((r["heads"], r["dim"])), "m": np.zeros(r["heads"])}}


def feed_forward(w, p, h):
    return lin(w[p + "down"], silu(lin(w[p + "gate"], h)) * lin(w[p + "up"], h))


# ----------------------------------------------------------------------------------------------------------------------
# model
# ----------------------------------------------------------------------------------------------------------------------
def layer_runs(cfg):
    """[(layer index, does this run open a pass of the looped layers)] in execution order."""
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp or lp["stop"] <= lp["start"]:
        return [(i, False) for i in range(n)]
    runs = [(i, False) for i in range(lp["start"])]
    for _ in range(lp["times"]):
        runs += [(i, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return runs + [(i, False) for i in range(lp["stop"], n)]


def new_memory(cfg):
    return {"pos": 0, "runs": [new_layer_memory(cfg["layers"][i]) for i, _ in layer_runs(cfg)]}


def pass_input(w, x, x0):
    return lin(w["loop.in"], np.concatenate([x, x0]))


def block(w, i, layer, eps, mult, x, mem, pos):
    p = "l%d." % i
    y = MIXERS[layer["type"]](w, p + "mix.", layer["mixer"], eps, rms_norm(x, w[p + "norm1"], eps), mem, pos)
    x = x + mult * rms_norm(y, w[p + "norm1b"], eps)
    if layer.get("mlp"):
        y = feed_forward(w, p + "mlp.", rms_norm(x, w[p + "norm2"], eps))
        x = x + mult * rms_norm(y, w[p + "norm2b"], eps)
    return x


def step(cfg, w, mem, token, residuals=None):
    """One token through the stack; returns the logits row and advances `mem`."""
    eps = cfg["norm"]["eps"]
    x0 = np.array(w["embed"][token], np.float64)
    x = x0.copy()
    for r, (i, opens) in enumerate(layer_runs(cfg)):
        if opens:
            x = pass_input(w, x, x0)
        x = block(w, i, cfg["layers"][i], eps, cfg["residual_mult"], x, mem["runs"][r], mem["pos"])
        if residuals is not None:
            residuals.append(x.copy())
    mem["pos"] += 1
    return lin(w["head"], rms_norm(x, w["final.norm"], eps))


def run(cfg, w, toks, layers=False, mem=None):
    """Logits rows [len(toks), vocab] (and, with layers, the residual after every layer run [runs, len(toks), width])."""
    mem = mem if mem is not None else new_memory(cfg)
    rows, res = [], []
    for t in toks:
        r = []
        rows.append(step(cfg, w, mem, int(t), r))
        res.append(np.stack(r))
    if layers:
        return np.stack(rows), np.stack(res, 1)
    return np.stack(rows)
