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


def delta(heads=4, kv_heads=2, dim=20, vdim=28, conv=3, mlp=None):
    return dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), mlp=mlp)


def latent(heads=3, dim=24, rot_dim=10, vdim=20, kv_rank=40, base=1000.0, scaling=True, scale=None, mlp=None):
    sc = dict(factor=6.0, original=48, fast=8.0, slow=1.0) if scaling is True else scaling
    return dict(type="latent_attention", mlp=mlp, mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank,
                scale=scale or (dim + rot_dim) ** -0.5, rot=dict(dims=rot_dim, base=base, **({"scaling": sc} if sc else {}))))


def dense(ff=72):
    return dict(kind="dense", ff=ff)


def moe(experts=7, top=2, ff=44, limit=1.5):
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff, limit=limit))


def zokelix(layers, width=104, vocab=150, eps=1e-5):
    return dict(architecture="Zokelix", vocab=vocab, width=width, layers=layers, norm=dict(eps=eps))


def zokelix_mixed(**kw):
    """Both mixers, unequal layers, all feed-forwards and none."""
    return zokelix([delta(mlp=moe()), latent(mlp=dense()), delta(heads=2, kv_heads=2, dim=36, vdim=12, conv=4), latent(heads=5, kv_rank=24, rot_dim=6, mlp=moe(5, 3, 20)),
                    delta(heads=3, kv_heads=1, conv=2, mlp=dense(50))], **kw)


def zokelix_weights(cfg, seed=0, ranks=(11, 7)):
    """bf16 weights by tensor name.  The routers rank the experts by channels of their own, which the layers' norms leave as the
    embedding set them: every choice is clear-cut, so that rounding cannot change it."""
    g = torch.Generator().manual_seed(seed)
    W, out = cfg["width"], {}

    def put(name, shape, std, mean=0.0):
        out[name] = (mean + std * torch.randn(shape, generator=g)).to(torch.bfloat16)

    most = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"], default=0)
    assert most < W // 2
    put("embed", (cfg["vocab"], W), 1.0)
    for t in range(cfg["vocab"]):
        out["embed"][t, :most] = torch.linspace(-2.0, 2.0, most)[torch.randperm(most, generator=g)] if most > 1 else 1.0
    put("head", (cfg["vocab"], W), 2.5 * W ** -0.5)
    put("final.norm", (W,), 0.2, 1.0)
    s = W ** -0.5
    for i, l in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", l["mixer"]
        H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
        put(p + "norm1", (W,), 0.2, 0.8)
        out[p + "norm1"][:most] = 0
        if l["type"] == "channel_delta":
            G = mx["kv_heads"]
            for n, c in (("q", G * d), ("k", G * d), ("v", H * dv)):
                put(p + "mix." + n, (c, W), s)
                put(p + "mix." + n + ".conv", (c, mx["conv"]), 0.7)
            put(p + "mix.b", (H, W), s)
            put(p + "mix.A_log", (H,), 0.5)
            put(p + "mix.dt_bias", (H * d,), 1.0, -3.0)
            put(p + "mix.norm", (dv,), 0.2, 1.0)
            for n, r, c in (("a", ranks[0], H * d), ("g", ranks[1], H * dv)):
                put(p + f"mix.{n}1", (r, W), s)
                put(p + f"mix.{n}2", (c, r), r ** -0.5)
        else:
            r, rank = mx["rot_dim"], mx["kv_rank"]
            put(p + "mix.q", (H * (d + r), W), 1.5 * s)
            put(p + "mix.dkv", (rank + r, W), 1.5 * s)
            put(p + "mix.dkv.norm", (rank,), 0.2, 1.0)
            put(p + "mix.uk", (H * d, rank), rank ** -0.5)
            put(p + "mix.uv", (H * dv, rank), rank ** -0.5)
        put(p + "mix.o", (W, H * dv), (H * dv) ** -0.5)
        if l["mlp"]:
            put(p + "norm2", (W,), 0.2, 0.8)
            out[p + "norm2"][:most] = 0
            if l["mlp"]["kind"] == "dense":
                ff = l["mlp"]["ff"]
                for n in ("gate", "up"):
                    put(p + "mlp." + n, (ff, W), s)
                    put(p + f"mlp.{n}.b", (ff,), 0.4)
                put(p + "mlp.down", (W, ff), ff ** -0.5)
                put(p + "mlp.down.b", (W,), 0.3)
            else:
                n_e, ff = l["mlp"]["router"]["experts"], l["mlp"]["expert"]["ff"]
                put(p + "mlp.router", (n_e, W), 0.002)
                out[p + "mlp.router"][torch.arange(n_e), torch.randperm(most, generator=g)[:n_e]] = 1.5
                for e in range(n_e):
                    put(p + f"mlp.e{e}.gate", (ff, W), 2 * s)
                    put(p + f"mlp.e{e}.up", (ff, W), 2 * s)
                    put(p + f"mlp.e{e}.down", (W, ff), ff ** -0.5)
    return out


def weights(cfg, seed=0):
    """bf16 weights by tensor name; written from the configuration alone."""
    if cfg["architecture"] == "Zokelix":
        return zokelix_weights(cfg, seed)
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


def plant_latent_pair(cfg, w, layer, asks, answers, strength=7.0):
    """The same for a latent attention layer, through the unrotated parts: one latent channel is filled by the token ``answers``
    alone, and every head's query of ``asks`` looks for it.  The layer must be the first one (it reads the embedding)."""
    mx, p = cfg["layers"][layer]["mixer"], f"l{layer}.mix."
    H, d, r, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["kv_rank"]
    w["embed"][:, -2:] = 0
    for tok, ch in ((asks, -2), (answers, -1)):
        w["embed"][tok] = 0.02 * w["embed"][tok]
        w["embed"][tok, ch] = 3.0
    w[p + "dkv"][0] = 0
    w[p + "dkv"][:, -2:] = 0
    w[p + "dkv"][0, -1] = 3.0
    w[p + "dkv.norm"][0] = 1.0
    q, uk = w[p + "q"].view(H, d + r, -1), w[p + "uk"].view(H, d, rank)
    q[:, :, -2:] = 0
    uk[:, :, 0] = 0
    s = strength / mx["scale"] / 3.0 / rank ** 0.5          # (the latent of ``answers`` is sqrt(rank) in its channel)
    q[:, 3, -2], uk[:, 3, 0] = 2 * s, 1.0


def plant_delta_pair(cfg, w, layer, asks, answers):
    """For a delta layer: key and query channel 0 of every head belong to these two tokens, nothing decays, so what ``answers``
    wrote stays until ``asks`` reads it.  The layer must be the first one."""
    mx, p = cfg["layers"][layer]["mixer"], f"l{layer}.mix."
    G, d = mx["kv_heads"], mx["dim"]
    w["embed"][:, -2:] = 0
    for tok, ch in ((asks, -2), (answers, -1)):
        w["embed"][tok] = 0.02 * w["embed"][tok]
        w["embed"][tok, ch] = 3.0
    w[p + "dt_bias"].fill_(-14.0)
    for n, ch in (("q", -2), ("k", -1)):
        m, c = w[p + n].view(G, d, -1), w[p + n + ".conv"].view(G, d, -1)
        m[:, :, -2:] = 0
        m[:, 0] = 0
        m[:, 0, ch] = 4.0
        c[:, 0] = 0
        c[:, 0, -1] = 1.0
