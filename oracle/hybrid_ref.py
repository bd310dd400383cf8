"""Plain restatement of the layer-list ("hybrid") decoder designs: one function per mechanism, whole sequences at
once, float64, loops where a loop is the definition.  Shares no code with the product path; used by tests only.

``HybridOracle(config, weights)`` takes the configuration dictionary and the weights as arrays by tensor name;
``forward(tokens)`` returns the logits of every position and the residual stream after every layer run.
"""
from __future__ import annotations

import math

import numpy as np

F = np.float64


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms_unit(x, eps):
    """Each vector of the last axis over its root mean square."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_zero_centred(x, w, eps):
    return rms_unit(x, eps) * (1.0 + w)


def causal_conv_residual(h, w):
    """h_t + sum_j w[:, j] h_{t - taps + 1 + j}, nothing before the first token."""
    T, _ = h.shape
    taps = w.shape[1]
    out = h.copy()
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def visible(i, j, size, keep_first):
    """Does position i see position j: causal, the last ``size`` positions or one of the first ``keep_first``."""
    return j <= i and (i - j < size or j < keep_first)


def softmax_attention(q, k, v, scale, size, keep_first):
    """One attention map: q [T, d], k [T, d], v [T, dv] -> [T, dv]."""
    T = q.shape[0]
    out = np.zeros((T, v.shape[1]), F)
    for i in range(T):
        cols = [j for j in range(i + 1) if visible(i, j, size, keep_first)]
        s = (k[cols] @ q[i]) * scale
        p = np.exp(s - s.max())
        out[i] = (p / p.sum()) @ v[cols]
    return out


def differential_lambda(lq1, lk1, lq2, lk2, diff):
    return math.exp(float(np.sum(lq1 * lk1))) - math.exp(float(np.sum(lq2 * lk2))) + diff


def mixer_attention(h, w, mx, eps):
    """Two softmax maps over the same values, their weighted difference normed per head, gated, projected."""
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    size = mx["mask"]["size"] if mx.get("mask") else T + 1
    keep = mx["mask"].get("keep_first", 0) if mx.get("mask") else 0
    q = (h @ w["q"].T).reshape(T, H, 2, d)
    k = (h @ w["k"].T).reshape(T, G, 2, d)
    v = (h @ w["v"].T).reshape(T, G, dv)
    lam = differential_lambda(w["lq1"], w["lk1"], w["lq2"], w["lk2"], mx["diff"])
    heads = []
    for a in range(H):
        g = a // (H // G)
        m1, m2 = (softmax_attention(q[:, a, m], k[:, g, m], v[:, g], mx["scale"], size, keep) for m in (0, 1))
        heads.append(rms_unit(m1 - lam * m2, eps) * (1.0 - mx["diff"]))
    o = np.concatenate(heads, axis=1) * sigmoid(h @ w["g"].T)
    return o @ w["o"].T


def gated_recurrence(q, f, v):
    """S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T, o_t = S_t^T q_t for one head, token by token."""
    T = q.shape[0]
    S = np.zeros((q.shape[1], v.shape[1]), F)
    out = np.zeros((T, v.shape[1]), F)
    for t in range(T):
        S = f[t][:, None] * S + np.outer(1.0 - f[t], v[t])
        out[t] = S.T @ q[t]
    return out


def mixer_hgrn2(h, w, mx, eps):
    T = h.shape[0]
    H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
    zq = h @ w["q"].T
    q = (zq * sigmoid(zq)).reshape(T, H, d)
    f = (w["lower"] + (1.0 - w["lower"]) * sigmoid(h @ w["f"].T + w["f.b"])).reshape(T, H, d)
    v = (h @ w["v"].T).reshape(T, H, dv)
    o = [rms_unit(gated_recurrence(q[:, a], f[:, a], v[:, a]), eps) * w["norm"] for a in range(H)]
    return np.concatenate(o, axis=1) @ w["o"].T


def polynorm(z, coef, eps):
    a, b, c, e = (float(t) for t in coef)
    return a * rms_unit(z, eps) + b * rms_unit(z ** 2, eps) + c * rms_unit(z ** 3, eps) + e


def ff_dense(h, w, eps):
    return polynorm(h @ w["up"].T, w["act"], eps) @ w["down"].T


MIXERS = {"attention": mixer_attention, "hgrn2": mixer_hgrn2}


def layer_order(config):
    """(layer index, begins a repeated pass) of every layer run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, False) for i in range(a)]
    for r in range(times):
        runs += [(i, r > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


class HybridOracle:
    def __init__(self, config, weights):
        self.config = config
        self.w = {k: np.asarray(v, F) for k, v in weights.items()}

    def sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def forward(self, tokens):
        c, w = self.config, self.w
        eps, m = c["norm"]["eps"], c.get("residual_mult", 1.0)
        emb = w["embed"][np.asarray(tokens, np.int64)]
        x = emb.copy()
        stream = []
        for i, again in layer_order(c):
            lc, p = c["layers"][i], f"l{i}."
            if again:
                x = x + emb
            h = norm_zero_centred(x, w[p + "norm1"], eps)
            h = causal_conv_residual(h, w[p + "canon1"])
            x = x + m * MIXERS[lc["type"]](h, self.sub(p + "mix."), lc["mixer"], eps)
            if lc.get("mlp"):
                x = x + m * ff_dense(norm_zero_centred(x, w[p + "norm2"], eps), self.sub(p + "mlp."), eps)
            stream.append(x.copy())
        logits = norm_zero_centred(x, w["final.norm"], eps) @ w["head"].T
        cap = c.get("logit_softcap")
        if cap:
            logits = cap * np.tanh(logits / cap)
        return logits, stream
