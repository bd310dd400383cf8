"""Small configurations and weights of the layer-list designs, for the tests."""
import numpy as np
import torch


def attention(heads=4, kv_heads=2, dim=24, vdim=40, size=20, keep_first=2, diff=0.25, scale=None, ff=None):
    mx = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, diff=diff, scale=scale or dim ** -0.5,
              mask=dict(size=size, keep_first=keep_first))
    return dict(type="attention", mixer=mx, mlp=dict(kind="dense", ff=ff) if ff else None)


def recurrence(heads=3, dim=20, vdim=28, ff=None):
    return dict(type="hgrn2", mixer=dict(heads=heads, dim=dim, vdim=vdim), mlp=dict(kind="dense", ff=ff) if ff else None)


def config(layers, width=88, vocab=150, taps=3, eps=1e-5, m=0.8, cap=25.0, loop=None):
    return dict(architecture="Zaverax", vocab=vocab, width=width, layers=layers, canon=dict(taps=taps), norm=dict(eps=eps),
                residual_mult=m, logit_softcap=cap, loop=loop)


def mixed(**kw):
    """Both mixers, a repeated range, unequal layers."""
    return config([recurrence(ff=72), attention(ff=136), recurrence(heads=2, dim=36, vdim=12), attention(heads=2, kv_heads=2, size=9, keep_first=3, ff=100),
                   recurrence(ff=72)], loop=dict(start=1, stop=4, times=2), **kw)


def weights(cfg, seed=0):
    """bf16 weights by tensor name; written from the configuration alone."""
    g = torch.Generator().manual_seed(seed)
    W, out = cfg["width"], {}

    def put(name, shape, std, mean=0.0):
        out[name] = (mean + std * torch.randn(shape, generator=g)).to(torch.bfloat16)

    put("embed", (cfg["vocab"], W), 1.0)
    put("head", (cfg["vocab"], W), 2.5 * W ** -0.5)
    put("final.norm", (W,), 0.2)
    for i, l in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", l["mixer"]
        H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
        put(p + "norm1", (W,), 0.2)
        put(p + "canon1", (W, cfg["canon"]["taps"]), 0.4)
        s = W ** -0.5
        if l["type"] == "attention":
            G = mx["kv_heads"]
            put(p + "mix.q", (H * 2 * d, W), 1.5 * s)
            put(p + "mix.k", (G * 2 * d, W), 1.5 * s)
            put(p + "mix.v", (G * dv, W), s)
            put(p + "mix.g", (H * dv, W), s)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                put(p + "mix." + n, (d,), 0.15)
        else:
            put(p + "mix.q", (H * d, W), s)
            put(p + "mix.f", (H * d, W), s)
            put(p + "mix.f.b", (H * d,), 2.5, 2.0)
            out[p + "mix.lower"] = torch.rand((H * d,), generator=g).mul(0.9).to(torch.bfloat16)
            put(p + "mix.v", (H * dv, W), s)
            put(p + "mix.norm", (dv,), 0.2, 1.0)
        put(p + "mix.o", (W, H * dv), (H * dv) ** -0.5)
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            put(p + "norm2", (W,), 0.2)
            put(p + "mlp.up", (ff, W), s)
            put(p + "mlp.down", (W, ff), ff ** -0.5)
            put(p + "mlp.act", (4,), 0.3, 0.4)
    return out


def as_numpy(w):
    return {k: v.float().numpy().astype(np.float64) for k, v in w.items()}


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed + 1000).integers(0, cfg["vocab"], n)


def plant_pair(cfg, w, layer, asks, answers, strength=6.0):
    """Make token ``asks`` look for token ``answers``: in the first map of every head of attention layer ``layer`` their
    query and key point the same way with a score that stands out, whatever lies between.  The layer must be the first
    one (its input is the normed embedding)."""
    mx, W, p = cfg["layers"][layer]["mixer"], cfg["width"], f"l{layer}."
    H, G, d = mx["heads"], mx["kv_heads"], mx["dim"]
    w[p + "norm1"].zero_()
    w[p + "canon1"].zero_()
    w["embed"][:, :2] = 0
    for tok, ch in ((asks, 0), (answers, 1)):
        w["embed"][tok] = 0.02 * w["embed"][tok]
        w["embed"][tok, ch] = 3.0
    s = (strength / mx["scale"]) ** 0.5 / W ** 0.5          # the normed embedding has sqrt(W) at its one channel
    q, k = w[p + "mix.q"].view(H, 2, d, W), w[p + "mix.k"].view(G, 2, d, W)
    q[:, 0, :, 0], k[:, 0, :, 1] = 0, 0
    q[:, 0, 3, 0], k[:, 0, 3, 1] = 2 * s, 2 * s
