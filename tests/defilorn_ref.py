"""Plain float64 restatement of the Defilorn design, one function per mechanism, numpy only.

It shares no code with the product path: whole sequences, loops over tokens and heads, no cache,
no state slots.  `forward(cfg_json, weights, tokens)` returns the logits of every position.

Notation: x [T, W] is the residual stream, h what a sublayer reads, names of `weights` are the
checkpoint's ("l<i>.mix.q", ...), linears are [out, in]."""
import math

import numpy as np


# ------------------------------------------------------------------ small pieces
def over_rms(z, eps):
    """z / sqrt(mean(z^2) + eps) along the last axis."""
    return z / np.sqrt((z * z).mean(axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


# ------------------------------------------------------------------ rotation
def frequencies(rot):
    """(one frequency per pair, what cos and sin are multiplied by)."""
    n, b = rot["dims"], float(rot["base"])
    f = [b ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def entry(turns):  # the (fractional) pair that turns this often over the original length
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(b))

    first, last = max(math.floor(entry(sc["fast"])), 0), min(math.ceil(entry(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        t = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(t * fi / sc["factor"] + (1.0 - t) * fi)
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_pairs(x, rot, positions):
    """Entries (2i, 2i + 1) of the first rot.dims entries turn together; the rest stays.  x [T, heads, n]."""
    y = x.copy()
    f, mult = frequencies(rot)
    for i, fi in enumerate(f):
        c, s = mult * np.cos(positions * fi)[:, None], mult * np.sin(positions * fi)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = u * c - v * s
        y[:, :, 2 * i + 1] = v * c + u * s
    return y


# ------------------------------------------------------------------ softmax
def softmax_rows(scores, window=0, sink=None):
    """Row i over the keys j with 0 <= i - j < window (window 0: every j <= i); with a sink the
    denominator holds exp(sink) too, which goes to no key."""
    T = scores.shape[0]
    out = np.zeros((T, T))
    for i in range(T):
        lo = max(0, i - window + 1) if window else 0
        s = scores[i, lo:i + 1]
        top = s.max() if sink is None else max(s.max(), sink)
        e = np.exp(s - top)
        out[i, lo:i + 1] = e / (e.sum() + (0.0 if sink is None else math.exp(sink - top)))
    return out


# ------------------------------------------------------------------ mixers
def latent_attention(h, mx, w, pre, eps):
    """Keys and values are expanded per head from one normed latent per token; a rotated key part
    is shared by the heads; a sink per head, an output gate per entry."""
    T = h.shape[0]
    H, d, r, m, R = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    pos = np.arange(T, dtype=np.float64)
    q = ((over_rms(h @ w[pre + "dq"].T, eps) * w[pre + "dq.norm"]) @ w[pre + "uq"].T).reshape(T, H, d + r)
    q_rot = rotate_pairs(q[:, :, d:], mx["rot"], pos)
    u = h @ w[pre + "dkv"].T
    c = over_rms(u[:, :R], eps) * w[pre + "dkv.norm"]
    k_rot = rotate_pairs(u[:, None, R:], mx["rot"], pos)[:, 0]
    k = (c @ w[pre + "uk"].T).reshape(T, H, d)
    v = (c @ w[pre + "uv"].T).reshape(T, H, m)
    out = np.zeros((T, H, m))
    for a in range(H):
        s = (q[:, a, :d] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * mx["scale"]
        out[:, a] = softmax_rows(s, sink=float(w[pre + "sink"][a])) @ v[:, a]
    return (out.reshape(T, H * m) * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def difference_weight(w, pre, diff):
    """What the second map is multiplied by."""
    return math.exp(float(w[pre + "lq1"] @ w[pre + "lk1"])) - math.exp(float(w[pre + "lq2"] @ w[pre + "lk2"])) + diff


def differential_attention(h, mx, w, pre, eps):
    """Two softmax maps per head over the same values, the second subtracted from the first."""
    T = h.shape[0]
    H, G, d, m = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = over_rms((h @ w[pre + "q"].T).reshape(T, H, 2, d), eps) * w[pre + "q.norm"]
    k = over_rms((h @ w[pre + "k"].T).reshape(T, G, 2, d), eps) * w[pre + "k.norm"]
    v = (h @ w[pre + "v"].T).reshape(T, G, m)
    lam = difference_weight(w, pre, mx["diff"])
    size = (mx.get("mask") or {}).get("size", 0)
    out = np.zeros((T, H, m))
    for a in range(H):
        g = a // (H // G)
        o = [softmax_rows(q[:, a, i] @ k[:, g, i].T * mx["scale"], size) @ v[:, g] for i in range(2)]
        out[:, a] = over_rms(o[0] - lam * o[1], eps) * (1.0 - mx["diff"])
    return out.reshape(T, H * m) @ w[pre + "o"].T


def matrix_memory(q, k, v, gi, gf):
    """One head: a matrix S and a vector n, both decaying by the forget gate, kept relative to a
    running maximum of the log gates (which starts at 0).  q, k [T, n], v [T, m], gi, gf [T] logarithms."""
    T, n = q.shape
    S, z, top = np.zeros((n, v.shape[1])), np.zeros(n), 0.0
    o = np.zeros((T, v.shape[1]))
    for t in range(T):
        new = max(gf[t] + top, gi[t])
        keep, write = math.exp(gf[t] + top - new), math.exp(gi[t] - new)
        S = keep * S + write * np.outer(k[t], v[t])
        z = keep * z + write * k[t]
        top = new
        o[t] = S.T @ q[t] / (max(abs(z @ q[t]), math.exp(-top)) + 1e-6)
    return o


def mlstm(h, mx, w, pre, eps):
    T = h.shape[0]
    H, n, m, cap = mx["heads"], mx["dim"], mx["vdim"], mx["gate_cap"]
    q = (h @ w[pre + "q"].T).reshape(T, H, n) / math.sqrt(n)
    k = (h @ w[pre + "k"].T).reshape(T, H, n)
    v = (h @ w[pre + "v"].T).reshape(T, H, m)
    gi = cap * np.tanh((h @ w[pre + "i"].T + w[pre + "i.b"]) / cap)
    gf = log_sigmoid(cap * np.tanh((h @ w[pre + "f"].T + w[pre + "f.b"]) / cap))
    o = np.stack([matrix_memory(q[:, a], k[:, a], v[:, a], gi[:, a], gf[:, a]) for a in range(H)], axis=1)
    o = over_rms(o, eps).reshape(T, H * m) * w[pre + "norm"]
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ------------------------------------------------------------------ feed-forward
def glu(h, w, pre, act):
    return (act(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(z, correction, top):
    """One token's logits: softmax over all, the choice by corrected scores, the weights uncorrected."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    idx = sorted(range(len(z)), key=lambda e: (-(s[e] + correction[e]), e))[:top]
    return idx, s[idx]


def experts(h, m, w, pre):
    z = h @ w[pre + "router"].T
    real = m["router"]["experts"]
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(*route(z[t], w[pre + "correction"], m["router"]["top"])):
            out[t] += p * (glu(h[t:t + 1], w, f"{pre}e{e}.", silu)[0] if e < real else h[t])
    if m.get("shared"):
        out += glu(h, w, pre + "shared.", silu) * sigmoid(h @ w[pre + "shared.sg"].T)
    return out


# ------------------------------------------------------------------ the model
def schedule(j):
    """(layer, is it the first of a pass other than the first pass?) in order of execution."""
    n, lp = len(j["layers"]), j.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    run = [(i, False) for i in range(a)]
    for t in range(lp["times"]):
        run += [(i, i == a and t > 0) for i in range(a, b)]
    return run + [(i, False) for i in range(b, n)]


def forward(j, weights, tokens, stream=None):
    """Logits [T, vocab].  `stream`: a list that receives x after every layer execution."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = j["norm"]["eps"]
    x0 = w["embed"][np.asarray(tokens)]
    x = x0
    mixers = {"latent_attention": latent_attention, "attention": differential_attention, "mlstm": mlstm}
    for i, again in schedule(j):
        lc, p = j["layers"][i], f"l{i}."
        if again:
            x = x + x0
        h = over_rms(x, eps) * (1.0 + w[p + "norm1"])
        x = x + mixers[lc["type"]](h, lc["mixer"], w, p + "mix.", eps)
        if lc.get("mlp"):
            h = over_rms(x, eps) * (1.0 + w[p + "norm2"])
            x = x + (glu(h, w, p + "mlp.", gelu_tanh) if lc["mlp"]["kind"] == "dense" else experts(h, lc["mlp"], w, p + "mlp."))
        if stream is not None:
            stream.append(x.copy())
    return (over_rms(x, eps) * (1.0 + w["final.norm"])) @ w["head"].T


def greedy(cfg_json, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg_json, w, toks)[-1])))
    return toks[len(prompt):]
