"""Plain float64 restatement of the Sozurax design, one function per mechanism, numpy only.

It shares no code with the product path: whole sequences, loops over tokens and heads, no cache,
no state slots.  `forward(cfg_json, weights, tokens)` returns the logits of every position.

Notation: x [T, W] is the residual stream, h what a sublayer reads, names of `weights` are the
checkpoint's ("l<i>.mix.q", ...), linears are [out, in]."""
import math

import numpy as np


# ------------------------------------------------------------------ small pieces
def layer_norm(x, weight, bias, eps):
    """Every row minus its mean, over sqrt(mean squared deviation + eps), times weight plus bias."""
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * weight + bias


def over_rms(z, eps):
    """z / sqrt(mean(z^2) + eps) along the last axis."""
    return z / np.sqrt((z * z).mean(axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def causal_conv(u, taps_w):
    """y_t = sum_j taps_w[:, j] * u_(t - n + 1 + j), n taps, the last column meets u_t itself;
    u is zero before the sequence's start.  u [T, C], taps_w [C, n]."""
    T, C = u.shape
    n = taps_w.shape[1]
    y = np.zeros((T, C))
    for t in range(T):
        for j in range(n):
            src = t - n + 1 + j
            if src >= 0:
                y[t] += taps_w[:, j] * u[src]
    return y


def rotate_pairs(x, dims, base, positions):
    """Entries (2i, 2i + 1) of the first `dims` turn by the angle position * base^(-2i / dims);
    the rest stays.  x [T, heads, n]."""
    y = x.copy()
    for i in range(dims // 2):
        ang = positions * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(ang)[:, None], np.sin(ang)[:, None]
        a, b = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = a * c - b * s
        y[:, :, 2 * i + 1] = b * c + a * s
    return y


def windowed_softmax(scores, window):
    """Row i over the keys j with 0 <= i - j < window (window 0: every j <= i)."""
    T = scores.shape[0]
    out = np.zeros((T, T))
    for i in range(T):
        lo = max(0, i - window + 1) if window else 0
        s = scores[i, lo:i + 1]
        e = np.exp(s - s.max())
        out[i, lo:i + 1] = e / e.sum()
    return out


# ------------------------------------------------------------------ mixers
def gated_state_scan(q, f, v):
    """One head: S <- diag(f_t) S + (1 - f_t) v_t^T, read out as S^T q_t; S starts at zero.
    q, f [T, n], v [T, m]."""
    T, n = q.shape
    S = np.zeros((n, v.shape[1]))
    o = np.zeros((T, v.shape[1]))
    for t in range(T):
        S = f[t][:, None] * S + np.outer(1.0 - f[t], v[t])
        o[t] = S.T @ q[t]
    return o


def hgrn2(h, mx, w, pre, eps):
    """Linear attention whose forget gate, bounded below, also says how much is written."""
    T = h.shape[0]
    H, n, m = mx["heads"], mx["dim"], mx["vdim"]
    q = silu(h @ w[pre + "q"].T).reshape(T, H, n)
    v = (h @ w[pre + "v"].T).reshape(T, H, m)
    low = w[pre + "lower"]
    f = (low + (1.0 - low) * sigmoid(h @ w[pre + "f"].T + w[pre + "f.b"])).reshape(T, H, n)
    o = np.stack([gated_state_scan(q[:, a], f[:, a], v[:, a]) for a in range(H)], axis=1)
    return (over_rms(o, eps) * w[pre + "norm"]).reshape(T, H * m) @ w[pre + "o"].T


def latent_attention(h, mx, w, pre, eps, caches, layer):
    """Keys and values are expanded per head from one normed latent per token; a rotated key part
    is shared by the heads.  caches[layer] keeps (latent, rotated part); `kv_from` reads another's."""
    T = h.shape[0]
    H, d, r, m, R = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    pos = np.arange(T, dtype=np.float64)
    rot = mx["rot"]
    q = ((over_rms(h @ w[pre + "dq"].T, eps) * w[pre + "dq.norm"]) @ w[pre + "uq"].T).reshape(T, H, d + r)
    q_rot = rotate_pairs(q[:, :, d:], rot["dims"], rot["base"], pos)
    if mx.get("kv_from") is None:
        u = h @ w[pre + "dkv"].T
        c = over_rms(u[:, :R], eps) * w[pre + "dkv.norm"]
        k_rot = rotate_pairs(u[:, None, R:], rot["dims"], rot["base"], pos)[:, 0]
        caches[layer] = (c, k_rot)
    else:
        c, k_rot = caches[mx["kv_from"]]
    k = (c @ w[pre + "uk"].T).reshape(T, H, d)
    v = (c @ w[pre + "uv"].T).reshape(T, H, m)
    out = np.zeros((T, H, m))
    for a in range(H):
        s = (q[:, a, :d] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * mx["scale"]
        out[:, a] = windowed_softmax(s, (mx.get("mask") or {}).get("size", 0)) @ v[:, a]
    return out.reshape(T, H * m) @ w[pre + "o"].T


# ------------------------------------------------------------------ feed-forward
def poly_norm(z, coef, eps):
    """A cubic whose powers are each divided by their own root mean square over the row."""
    a, b, c, e = coef
    return a * over_rms(z, eps) + b * over_rms(z ** 2, eps) + c * over_rms(z ** 3, eps) + e


def dense(h, w, pre, eps):
    return poly_norm(h @ w[pre + "up"].T, w[pre + "act"], eps) @ w[pre + "down"].T


def gated(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(z, top):
    """The `top` largest of one token's logits and their softmax among themselves."""
    idx = sorted(range(len(z)), key=lambda e: (-z[e], e))[:top]
    p = np.exp(z[idx] - z[idx].max())
    return idx, p / p.sum()


def experts(h, m, w, pre):
    z = h @ w[pre + "router"].T + w[pre + "router.b"]
    out = gated(h, w, pre + "shared.") if m.get("shared") else np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(*route(z[t], m["router"]["top"])):
            out[t] += p * gated(h[t:t + 1], w, f"{pre}e{e}.")[0]
    return out


# ------------------------------------------------------------------ the model
def forward(j, weights, tokens, stream=None):
    """Logits [T, vocab].  `stream`: a list that receives x after every layer."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = j["norm"]["eps"]

    def read(x, p, which):  # what a sublayer reads: the norm, then the convolution on top
        h = layer_norm(x, w[p + "norm" + which], w[p + "norm" + which + ".b"], eps)
        return h + causal_conv(h, w[p + "canon" + which])

    x = w["embed"][np.asarray(tokens)] * j["embedding"]["scale"]
    caches = {}
    for i, lc in enumerate(j["layers"]):
        p = f"l{i}."
        h = read(x, p, "1")
        if lc["type"] == "hgrn2":
            x = x + hgrn2(h, lc["mixer"], w, p + "mix.", eps)
        elif lc["type"] == "latent_attention":
            x = x + latent_attention(h, lc["mixer"], w, p + "mix.", eps, caches, i)
        else:
            raise ValueError(lc["type"])
        if lc.get("mlp"):
            h = read(x, p, "2")
            x = x + (dense(h, w, p + "mlp.", eps) if lc["mlp"]["kind"] == "dense" else experts(h, lc["mlp"], w, p + "mlp."))
        if stream is not None:
            stream.append(x.copy())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T


def greedy(cfg_json, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg_json, w, toks)[-1])))
    return toks[len(prompt):]
