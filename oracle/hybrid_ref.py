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


# ---------------------------------------------------------------------- channel-wise gated delta rule
def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def causal_conv(h, w):
    """sum_j w[:, j] h_{t - taps + 1 + j}, nothing before the first token."""
    T, _ = h.shape
    taps = w.shape[1]
    out = np.zeros_like(h)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def channel_decay(low, a2, dt_bias, a_log, heads):
    """exp(-exp(A_log_h) softplus(z)) per head and key channel."""
    z = (low @ a2.T + dt_bias).reshape(low.shape[0], heads, -1)
    return np.exp(-np.exp(a_log)[None, :, None] * softplus(z))


def delta_rule(q, k, v, g, beta):
    """One head, token by token: the rows of S decay, then the error of what S holds for k is written back at rate beta."""
    T = q.shape[0]
    S = np.zeros((k.shape[1], v.shape[1]), F)
    out = np.zeros((T, v.shape[1]), F)
    for t in range(T):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def mixer_channel_delta(h, w, mx, eps):
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.reshape(T, G, d)) * d ** -0.5
    k = unit(k.reshape(T, G, d))
    v = v.reshape(T, H, dv)
    beta = sigmoid(h @ w["b"].T)
    g = channel_decay(h @ w["a1"].T, w["a2"], w["dt_bias"], w["A_log"], H)
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T).reshape(T, H, dv)
    heads = []
    for a in range(H):
        s = a // (H // G)
        heads.append(rms_unit(delta_rule(q[:, s], k[:, s], v[:, a], g[:, a], beta[:, a]), eps) * w["norm"] * gate[:, a])
    return np.concatenate(heads, axis=1) @ w["o"].T


# ---------------------------------------------------------------------- latent attention
def rotation_frequencies(rot):
    """Angle per position of every pair, and the factor on cos and sin (YaRN interpolation when the rotation is scaled)."""
    n, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)], F)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    pair_of = lambda turns: n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair_of(sc["fast"])), 0), min(math.ceil(pair_of(sc["slow"])), n - 1)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_interleaved(x, pos, rot):
    """Pairs (2i, 2i + 1) of the first rot.dims of the last axis; x [T, ..., n]."""
    f, mag = rotation_frequencies(rot)
    out = x.copy()
    for t, p in enumerate(pos):
        for i, fi in enumerate(f):
            c, s = mag * math.cos(p * fi), mag * math.sin(p * fi)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i], out[t, ..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def mixer_latent_attention(h, w, mx, eps):
    T = h.shape[0]
    H, d, r, dv, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    q = (h @ w["q"].T).reshape(T, H, d + r)
    qr = rotate_interleaved(q[..., d:], range(T), mx["rot"])
    z = h @ w["dkv"].T
    c = rms_unit(z[:, :rank], eps) * w["dkv.norm"]
    kr = rotate_interleaved(z[:, rank:], range(T), mx["rot"])
    k = (c @ w["uk"].T).reshape(T, H, d)
    v = (c @ w["uv"].T).reshape(T, H, dv)
    heads = [softmax_attention(np.concatenate([q[:, a, :d], qr[:, a]], 1), np.concatenate([k[:, a], kr], 1), v[:, a], mx["scale"], T + 1, 0)
             for a in range(H)]
    return np.concatenate(heads, axis=1) @ w["o"].T


# ---------------------------------------------------------------------- gated feed-forwards
def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def ff_gated(h, w, mlp, eps):
    return (gelu_tanh(h @ w["gate"].T + w["gate.b"]) * (h @ w["up"].T + w["up.b"])) @ w["down"].T + w["down.b"]


def expert(h, gate, up, down, limit):
    g = np.minimum(gate @ h, limit)
    u = np.clip(up @ h, -limit, limit)
    return down @ (g * sigmoid(1.702 * g) * (u + 1.0))


def ff_experts(h, w, mlp, eps):
    """Every token through its ``top`` experts by sigmoid score, the score on the expert's input."""
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        s = sigmoid(w["router"] @ h[t])
        for e in sorted(range(len(s)), key=lambda e: -s[e])[:mlp["router"]["top"]]:
            out[t] += expert(s[e] * h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], mlp["expert"]["limit"])
    return out


MIXERS = {"attention": mixer_attention, "hgrn2": mixer_hgrn2, "channel_delta": mixer_channel_delta,
          "latent_attention": mixer_latent_attention}
FEED_FORWARDS = {"Zaverax": {"dense": lambda h, w, mlp, eps: ff_dense(h, w, eps)},
                 "Zokelix": {"dense": ff_gated, "moe": ff_experts}}
NORMED_OUTPUTS = {"Zokelix"}             # designs whose norms sit on the sublayers' outputs, with plain weights


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
        ffs, after = FEED_FORWARDS[c["architecture"]], c["architecture"] in NORMED_OUTPUTS
        emb = w["embed"][np.asarray(tokens, np.int64)]
        x = emb.copy()
        stream = []
        for i, again in layer_order(c):
            lc, p = c["layers"][i], f"l{i}."
            if again:
                x = x + emb
            mixer, mix = MIXERS[lc["type"]], self.sub(p + "mix.")
            mlp = lc.get("mlp")
            if after:
                x = x + rms_unit(mixer(x, mix, lc["mixer"], eps), eps) * w[p + "norm1"]
                if mlp:
                    x = x + rms_unit(ffs[mlp["kind"]](x, self.sub(p + "mlp."), mlp, eps), eps) * w[p + "norm2"]
            else:
                h = norm_zero_centred(x, w[p + "norm1"], eps)
                h = causal_conv_residual(h, w[p + "canon1"])
                x = x + m * mixer(h, mix, lc["mixer"], eps)
                if mlp:
                    x = x + m * ffs[mlp.get("kind", "dense")](norm_zero_centred(x, w[p + "norm2"], eps), self.sub(p + "mlp."), mlp, eps)
            stream.append(x.copy())
        final = rms_unit(x, eps) * w["final.norm"] if after else norm_zero_centred(x, w["final.norm"], eps)
        logits = final @ w["head"].T
        cap = c.get("logit_softcap")
        if cap:
            logits = cap * np.tanh(logits / cap)
        return logits, stream
