"""Decoders given as a list of layers, each with its own token mixer and feed-forward (``libb200hybrid.so``).

A configuration names the layers in order (``layers``: mixer type and sizes, feed-forward), a range of layers that is
run several times with the same weights (``loop``), the norm, the input convolution, the residual factor and the logit
soft cap.  ``DESIGNS`` holds what an architecture fixes beside that: where its norms sit and which feed-forward a name means.
Mixers are looked up by name in ``MIXERS``; a design built from the same parts needs only an entry there and a
configuration, a new mechanism one more class and its kernel.

``HybridModel`` has the interface of ``llama.Model`` towards the decoding loop (``__call__`` for prompts and chains,
``forward_device`` for the tree passes, ``make_cache``), so ``eagle.SpecDecoder`` and the command line drive it like
the 4-bit models.  What differs is the cache: besides K/V rows, every layer run carries the last inputs of its
convolution and, where the mixer is a recurrence, a state matrix.  These cannot be rewound by moving an offset, so a
tree pass leaves them alone (its rows wait in *pending* buffers) and ``commit_rows`` advances them over the rows that
were accepted.

Weights are bf16; activations and cache are bf16 (``dtype="bfloat16"``, tensor-core products with fp32 accumulation)
or fp32 (``dtype="float32"``, plain fp32 multiply-adds).  Norms, softmax, the residual stream, gates of the recurrence
and its state are fp32 in both.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass, field, replace
from typing import Dict, List, Optional, Sequence, Union

import torch

from . import _lib
from .llama import FwdInputs, KVCache, MAX_ROWS, MAX_TAIL

PENDING_ROWS = 64            # B200_HYBRID_PENDING
NO_WINDOW = (1 << 31) - 1
MIXER_ATTENTION, MIXER_RECURRENCE, MIXER_DELTA, MIXER_LATENT = 0, 1, 2, 3
FF_POLYNORM, FF_GATED, FF_EXPERTS = 0, 1, 2
ALIGN = 256                  # byte alignment of the parts of a cache


def _up(v: int, m: int) -> int:
    return (v + m - 1) // m * m


@dataclass
class LayerSpec:
    """One entry of the layer list."""
    type: str
    mixer: dict
    mlp: Optional[dict]


@dataclass
class HybridArgs:
    architecture: str
    vocab_size: int
    width: int
    layers: List[LayerSpec]
    eps: float
    taps: int
    residual_mult: float = 1.0
    logit_softcap: float = 0.0
    loop: Optional[dict] = None
    model_type: str = field(default="hybrid", init=False)

    @staticmethod
    def from_config(config: dict) -> "HybridArgs":
        if config["architecture"] not in DESIGNS:
            raise _lib.B200Error(f"no design {config['architecture']!r}; known: {sorted(DESIGNS)}")
        ffs = DESIGNS[config["architecture"]].feed_forwards
        layers = [LayerSpec(l["type"], dict(l["mixer"]), dict(l["mlp"]) if l.get("mlp") else None) for l in config["layers"]]
        for l in layers:
            if l.type not in MIXERS:
                raise _lib.B200Error(f"no mixer {l.type!r}; known: {sorted(MIXERS)}")
            if l.mlp is not None and l.mlp.get("kind", "dense") not in ffs:
                raise _lib.B200Error(f"no feed-forward {l.mlp.get('kind')!r}; known: {sorted(ffs)}")
        loop = config.get("loop") or None
        if loop is not None:
            loop = {k: int(loop[k]) for k in ("start", "stop", "times")}
            if not (0 <= loop["start"] < loop["stop"] <= len(layers)) or loop["times"] < 1:
                raise _lib.B200Error(f"loop {loop} does not fit {len(layers)} layers")
        return HybridArgs(
            architecture=config["architecture"], vocab_size=int(config["vocab"]), width=int(config["width"]), layers=layers,
            eps=float(config["norm"]["eps"]), taps=int((config.get("canon") or {}).get("taps", 1)),
            residual_mult=float(config.get("residual_mult", 1.0)), logit_softcap=float(config.get("logit_softcap") or 0.0),
            loop=loop)

    @property
    def design(self) -> "Design":
        return DESIGNS[self.architecture]

    def feed_forward(self, spec: LayerSpec):
        return self.design.feed_forwards[spec.mlp.get("kind", "dense")]

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def runs(self) -> List[tuple]:
        """(layer, is the embedding output added after it) of every layer run of a pass: the loop's layers appear once
        per repetition, and each repetition but the first begins with the embedding output added to the stream."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        a, b, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        out = [(i, False) for i in range(a)]
        for r in range(times):
            out += [(i, i == b - 1 and r + 1 < times) for i in range(a, b)]
        return out + [(i, False) for i in range(b, n)]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.runs)


# ---------------------------------------------------------------------- mechanisms
class Mixer:
    """A token mixer: its tensors, what a request's cache and the pending buffer hold for a run of it (bytes by the run
    table's field name: ``state`` is zero at the start of a sequence, ``rows`` grow with the cache), its columns in the
    activation buffers, and how its weights go into the layer table."""

    @staticmethod
    def resolve(mx: dict, shapes: Dict[str, tuple]) -> dict:
        """``mx`` with the sizes that only the tensors' shapes give."""
        return mx

    @staticmethod
    def state(mx: dict, es: int) -> Dict[str, int]:
        return {}

    @staticmethod
    def rows(mx: dict, es: int, rows: int) -> Dict[str, int]:
        return {}

    @staticmethod
    def pending(mx: dict, es: int) -> Dict[str, int]:
        return {}


class Attention(Mixer):
    """Softmax attention; two maps per head (differential) when the configuration has ``diff``; sliding window with
    kept first keys from ``mask``; output gate."""
    launches = 4                 # projections, splits, their merge, output product (decoding)

    @staticmethod
    def maps(mx: dict) -> int:
        return 2 if mx.get("diff") is not None else 1

    @staticmethod
    def shapes(mx: dict, width: int) -> Dict[str, tuple]:
        H, G, d, dv, n = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], Attention.maps(mx)
        if H % G:
            raise _lib.B200Error("query heads must be a multiple of the key/value heads")
        s = {"q": (H * n * d, width), "k": (G * n * d, width), "v": (G * dv, width), "g": (H * dv, width), "o": (width, H * dv)}
        if n == 2:
            s.update({k: (d,) for k in ("lq1", "lk1", "lq2", "lk2")})
        return s

    @staticmethod
    def rows(mx: dict, es: int, rows: int) -> Dict[str, int]:
        per = es * mx["kv_heads"] * rows
        return {"k_off": per * Attention.maps(mx) * _up(mx["dim"], 16), "v_off": per * _up(mx["vdim"], 16)}

    @staticmethod
    def buffers(mx: dict) -> Dict[str, int]:
        mix = mx["heads"] * mx["vdim"]
        return dict(qb=mx["heads"] * Attention.maps(mx) * _up(mx["dim"], 16), gb=mix, ab=_up(mix, 64))

    @staticmethod
    def bind(model: "HybridModel", layer: "_lib.HybridLayer", mx: dict, w: Dict[str, torch.Tensor]):
        n = Attention.maps(mx)
        layer.mixer, layer.maps = MIXER_ATTENTION, n
        layer.heads, layer.kv_heads, layer.dim, layer.vdim = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        mask = mx.get("mask") or {}
        layer.window = min(int(mask.get("size") or NO_WINDOW), NO_WINDOW)
        layer.keep_first = int(mask.get("keep_first") or 0)
        layer.scale, layer.out_scale = float(mx["scale"]), 1.0
        if n == 2:
            dot = lambda a, b: math.exp(float((w[a].double() * w[b].double()).sum()))
            layer.lambda_ = dot("lq1", "lk1") - dot("lq2", "lk2") + float(mx["diff"])
            layer.out_scale = 1.0 - float(mx["diff"])
        layer.in_ = model.linear(w["q"], w["k"], w["v"], w["g"])
        layer.out = model.linear(w["o"])


class GatedRecurrence(Mixer):
    """HGRN2: a linear recurrence whose forget gate (with a lower bound per channel) also decides what is written."""
    launches = 4                 # projections, scan, head norm, output product

    @staticmethod
    def shapes(mx: dict, width: int) -> Dict[str, tuple]:
        H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
        return {"q": (H * d, width), "f": (H * d, width), "f.b": (H * d,), "lower": (H * d,), "v": (H * dv, width),
                "norm": (dv,), "o": (width, H * dv)}

    @staticmethod
    def state(mx: dict, es: int) -> Dict[str, int]:
        return {"state_off": 4 * mx["heads"] * mx["dim"] * mx["vdim"]}

    @staticmethod
    def pending(mx: dict, es: int) -> Dict[str, int]:
        return {"pend_g": 4 * mx["heads"] * mx["dim"], "pend_v": es * mx["heads"] * mx["vdim"]}

    @staticmethod
    def buffers(mx: dict) -> Dict[str, int]:
        d, dv = mx["heads"] * mx["dim"], mx["heads"] * mx["vdim"]
        return dict(qb=d, gf=d, vb=dv, o32=dv, ab=_up(dv, 64))

    @staticmethod
    def bind(model: "HybridModel", layer: "_lib.HybridLayer", mx: dict, w: Dict[str, torch.Tensor]):
        layer.mixer, layer.maps = MIXER_RECURRENCE, 1
        layer.heads = layer.kv_heads = mx["heads"]
        layer.dim, layer.vdim = mx["dim"], mx["vdim"]
        layer.gate_bias, layer.gate_lower = model.vector(w["f.b"]), model.vector(w["lower"])
        layer.head_norm = model.vector(w["norm"])
        layer.in_ = model.linear(w["q"], w["f"], w["v"])
        layer.out = model.linear(w["o"])


class ChannelDelta(Mixer):
    """Gated delta rule with a decay per key channel; short convolutions on queries, keys and values; low-rank decay and
    output gate (their ranks are given by the tensors)."""
    launches = 4                 # projections, low-rank products, step, output product (decoding)

    @staticmethod
    def ranks(mx: dict) -> tuple:
        return int(mx.get("decay_rank", mx["dim"])), int(mx.get("gate_rank", mx["vdim"]))

    @staticmethod
    def channels(mx: dict) -> int:
        return 2 * mx["kv_heads"] * mx["dim"] + mx["heads"] * mx["vdim"]

    @staticmethod
    def resolve(mx: dict, shapes: Dict[str, tuple]) -> dict:
        return dict(mx, decay_rank=shapes["a1"][0], gate_rank=shapes["g1"][0])

    @staticmethod
    def shapes(mx: dict, width: int) -> Dict[str, tuple]:
        H, G, d, dv, taps = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["conv"]
        if H % G:
            raise _lib.B200Error("heads must be a multiple of the query/key heads")
        if not (1 <= taps <= 8):
            raise _lib.B200Error("the convolutions have 1 to 8 taps")
        ra, rg = ChannelDelta.ranks(mx)
        s = {"o": (width, H * dv), "b": (H, width), "A_log": (H,), "dt_bias": (H * d,), "norm": (dv,), "a1": (ra, width), "a2": (H * d, ra),
             "g1": (rg, width), "g2": (H * dv, rg)}
        for n, c in (("q", G * d), ("k", G * d), ("v", H * dv)):
            s[n], s[n + ".conv"] = (c, width), (c, taps)
        return s

    @staticmethod
    def state(mx: dict, es: int) -> Dict[str, int]:
        return {"state_off": 4 * mx["heads"] * mx["dim"] * mx["vdim"], "mix_off": es * (mx["conv"] - 1) * _up(ChannelDelta.channels(mx), 8)}

    @staticmethod
    def pending(mx: dict, es: int) -> Dict[str, int]:
        return {"pend_g": 4 * mx["heads"] * mx["dim"], "pend_v": es * mx["heads"] * mx["vdim"], "pend_c": es * _up(ChannelDelta.channels(mx), 8),
                "pend_k": 4 * mx["kv_heads"] * mx["dim"], "pend_b": 4 * mx["heads"]}

    @staticmethod
    def buffers(mx: dict) -> Dict[str, int]:
        d, dv, k = mx["heads"] * mx["dim"], mx["heads"] * mx["vdim"], mx["kv_heads"] * mx["dim"]
        return dict(cb=_up(ChannelDelta.channels(mx), 8), beta=mx["heads"], lowb=_up(sum(ChannelDelta.ranks(mx)), 64), q32=k, k32=k, vb=dv, gf=d,
                    gb=dv, o32=dv, ab=_up(dv, 64))

    @staticmethod
    def bind(model: "HybridModel", layer: "_lib.HybridLayer", mx: dict, w: Dict[str, torch.Tensor]):
        layer.mixer, layer.maps = MIXER_DELTA, 1
        layer.heads, layer.kv_heads, layer.dim, layer.vdim = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        layer.conv_taps = mx["conv"]
        layer.mix_conv = model.vector(torch.cat([w[n + ".conv"] for n in ("q", "k", "v")]).t())
        layer.decay_bias = model.vector(w["dt_bias"])
        layer.decay_rate = model.vector(w["A_log"].double().exp().repeat_interleave(mx["dim"]))
        layer.head_norm = model.vector(w["norm"])
        layer.in_ = model.linear(w["q"], w["k"], w["v"], w["b"], w["a1"], w["g1"])
        # both low-rank products as one: the decay's rows read the first columns of their inputs, the gate's the others
        ra, rg = ChannelDelta.ranks(mx)
        layer.low_rank = ra + rg
        layer.low = model.linear(torch.nn.functional.pad(w["a2"], (0, rg)), torch.nn.functional.pad(w["g2"], (ra, 0)))
        layer.out = model.linear(w["o"])


def rotation(rot: dict) -> tuple:
    """Angle per position of every pair of a rotary embedding (fp64), and the factor on cos and sin: plain, or with the
    frequencies between the two turn counts of ``scaling`` interpolated (YaRN)."""
    n, base = int(rot["dims"]), float(rot["base"])
    f = base ** (-torch.arange(0, n, 2, dtype=torch.float64) / n)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    pair = lambda turns: n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(pair(sc["fast"])), 0), min(math.ceil(pair(sc["slow"])), n - 1)
    ramp = ((torch.arange(n // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


class LatentAttention(Mixer):
    """Softmax attention whose keys and values are products of one cached low-rank latent; a rotated key part, cached too,
    is shared by all heads."""
    launches = 7                 # projections, norm + rotation, query products, splits, merge, value products, output product

    @staticmethod
    def shapes(mx: dict, width: int) -> Dict[str, tuple]:
        H, d, r, dv, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
        if int(mx["rot"]["dims"]) != r or r % 2:
            raise _lib.B200Error("the rotated part is rotated as a whole, in pairs")
        return {"q": (H * (d + r), width), "dkv": (rank + r, width), "dkv.norm": (rank,), "uk": (H * d, rank), "uv": (H * dv, rank),
                "o": (width, H * dv)}

    @staticmethod
    def rows(mx: dict, es: int, rows: int) -> Dict[str, int]:
        return {"k_off": es * rows * (_up(mx["kv_rank"], 16) + _up(mx["rot_dim"], 16))}

    @staticmethod
    def buffers(mx: dict) -> Dict[str, int]:
        H, d, r, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["kv_rank"]
        return dict(qb=H * (_up(max(d, rank), 16) + _up(r, 16)), lat32=H * r + rank + r, qn=H * _up(d, 64), ob=H * _up(rank, 64),
                    ab=_up(H * mx["vdim"], 64))

    @staticmethod
    def expanded(mx: dict) -> tuple:
        """Columns per cache row of the keys and of the values of all heads."""
        return mx["heads"] * _up(mx["dim"], 16), mx["heads"] * _up(mx["vdim"], 16)

    @staticmethod
    def bind(model: "HybridModel", layer: "_lib.HybridLayer", mx: dict, w: Dict[str, torch.Tensor]):
        H, d, r, dv, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
        layer.mixer, layer.maps = MIXER_LATENT, 1
        layer.heads, layer.kv_heads, layer.dim, layer.vdim = H, 1, d, dv
        layer.kv_rank, layer.rot_dim, layer.window = rank, r, NO_WINDOW
        layer.scale, layer.out_scale = float(mx["scale"]), 1.0
        freq, layer.rot_mag = rotation(mx["rot"])
        layer.rot_freq, layer.latent_norm = model.vector(freq), model.vector(w["dkv.norm"])
        q = w["q"].view(H, d + r, -1)
        layer.in_ = model.linear(q[:, :d].reshape(H * d, -1), q[:, d:].reshape(H * r, -1), w["dkv"])
        layer.absorb = model.stack([u.t() for u in w["uk"].view(H, d, rank)])
        layer.value = model.stack(list(w["uv"].view(H, dv, rank)))
        layer.expand = model.linear(w["uk"], w["uv"])
        layer.out = model.linear(w["o"])


class PolyNormFF:
    """W_down act(W_up h) with act = a N(z) + b N(z^2) + c N(z^3) + e, N: over the root mean square of the vector."""
    launches = 3                 # products, activation

    @staticmethod
    def shapes(mlp: dict, width: int) -> Dict[str, tuple]:
        return {"up": (mlp["ff"], width), "down": (width, mlp["ff"]), "act": (4,)}

    @staticmethod
    def buffers(mlp: dict, width: int) -> Dict[str, int]:
        return dict(zb=_up(mlp["ff"], 64), zab=_up(mlp["ff"], 64))

    @staticmethod
    def bind(model: "HybridModel", layer: "_lib.HybridLayer", mlp: dict, w: Dict[str, torch.Tensor]):
        layer.ff, layer.ff_kind = mlp["ff"], FF_POLYNORM
        for i, v in enumerate(w["act"].float().tolist()):
            layer.act[i] = v
        layer.up, layer.down = model.linear(w["up"]), model.linear(w["down"])


def _alternate(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """Rows gate_0, up_0, gate_1, ...: both branches of a channel in neighbouring columns of one product."""
    return torch.stack([gate, up], 1).reshape(2 * gate.shape[0], *gate.shape[1:])


class GatedFF:
    """W_down (gelu_tanh(W_gate h + b) (W_up h + b)) + b."""
    launches = 2

    @staticmethod
    def shapes(mlp: dict, width: int) -> Dict[str, tuple]:
        f = mlp["ff"]
        return {"gate": (f, width), "gate.b": (f,), "up": (f, width), "up.b": (f,), "down": (width, f), "down.b": (width,)}

    @staticmethod
    def buffers(mlp: dict, width: int) -> Dict[str, int]:
        return dict(zb32=_up(2 * mlp["ff"], 64), zab=_up(mlp["ff"], 64), y=width)

    @staticmethod
    def bind(model: "HybridModel", layer: "_lib.HybridLayer", mlp: dict, w: Dict[str, torch.Tensor]):
        layer.ff, layer.ff_kind = mlp["ff"], FF_GATED
        layer.up, layer.down = model.linear(_alternate(w["gate"], w["up"])), model.linear(w["down"])
        layer.up_bias, layer.down_bias = model.vector(_alternate(w["gate.b"], w["up.b"])), model.vector(w["down.b"])


class ExpertsFF:
    """Mixture of experts: sigmoid scores, the largest ``top`` of them as they are on the experts' inputs; clipped gated
    experts, swish with slope ``alpha`` and the other branch shifted by ``shift``."""
    launches = 3                 # router, both expert products
    alpha, shift = 1.702, 1.0

    @staticmethod
    def shapes(mlp: dict, width: int) -> Dict[str, tuple]:
        f = mlp["expert"]["ff"]
        s = {"router": (mlp["router"]["experts"], width)}
        for e in range(mlp["router"]["experts"]):
            s.update({f"e{e}.gate": (f, width), f"e{e}.up": (f, width), f"e{e}.down": (width, f)})
        return s

    @staticmethod
    def buffers(mlp: dict, width: int) -> Dict[str, int]:
        top = mlp["router"]["top"]
        return dict(zab=top * _up(mlp["expert"]["ff"], 64), y=top * width, xg=top * _up(width, 64), zr=mlp["router"]["experts"])

    @staticmethod
    def bind(model: "HybridModel", layer: "_lib.HybridLayer", mlp: dict, w: Dict[str, torch.Tensor]):
        n, top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
        if not (1 <= top <= min(n, 16)) or n > 512:
            raise _lib.B200Error("1 to 16 of at most 512 experts per token")
        layer.ff, layer.ff_kind, layer.experts, layer.top = mlp["expert"]["ff"], FF_EXPERTS, n, top
        layer.act[0], layer.act[1], layer.act[2] = float(mlp["expert"]["limit"]), ExpertsFF.alpha, ExpertsFF.shift
        layer.router = model.linear(w["router"])
        layer.up = model.stack([_alternate(w[f"e{e}.gate"], w[f"e{e}.up"]) for e in range(n)])
        layer.down = model.stack([w[f"e{e}.down"] for e in range(n)])


MIXERS = {"attention": Attention, "hgrn2": GatedRecurrence, "channel_delta": ChannelDelta, "latent_attention": LatentAttention}


@dataclass(frozen=True)
class Design:
    """What an architecture fixes beside its configuration."""
    feed_forwards: dict              # by the configuration's ``kind``
    norm_out: bool = False           # norms on the sublayers' outputs (else on their inputs)
    norm_offset: float = 0.0         # added to the norm weights of the stream
    input_conv: bool = False         # a causal convolution in front of every mixer


DESIGNS = {
    "Zaverax": Design({"dense": PolyNormFF}, norm_offset=1.0, input_conv=True),
    "Zokelix": Design({"dense": GatedFF, "moe": ExpertsFF}, norm_out=True),
}


def weight_shapes(args: HybridArgs) -> Dict[str, tuple]:
    """Every tensor of a checkpoint with its shape."""
    W = args.width
    s = {"embed": (args.vocab_size, W)}
    for i, l in enumerate(args.layers):
        s[f"l{i}.norm1"] = (W,)
        if args.design.input_conv:
            s[f"l{i}.canon1"] = (W, args.taps)
        s.update({f"l{i}.mix.{k}": v for k, v in MIXERS[l.type].shapes(l.mixer, W).items()})
        if l.mlp is not None:
            s[f"l{i}.norm2"] = (W,)
            s.update({f"l{i}.mlp.{k}": v for k, v in args.feed_forward(l).shapes(l.mlp, W).items()})
    s["final.norm"] = (W,)
    s["head"] = (args.vocab_size, W)
    return s


def resolve(args: HybridArgs, weights: Dict[str, torch.Tensor]) -> HybridArgs:
    """``args`` with the sizes that the tensors' shapes give."""
    layers = []
    for i, l in enumerate(args.layers):
        p = f"l{i}.mix."
        try:
            mx = MIXERS[l.type].resolve(l.mixer, {k[len(p):]: tuple(v.shape) for k, v in weights.items() if k.startswith(p)})
        except KeyError as e:
            raise _lib.B200Error(f"checkpoint has no tensor {p}{e.args[0]}")
        layers.append(LayerSpec(l.type, mx, l.mlp))
    return replace(args, layers=layers)


# ---------------------------------------------------------------------- cache
class HybridCache(KVCache):
    """K/V rows and recurrent state of one request, one allocation: first every run's convolution inputs and state
    matrices (zero at the start of a sequence), then the K/V rows.  ``offset`` is the committed length; it moves forward
    only (through passes and commits) or back to zero (``reset``)."""

    def __init__(self, model: "HybridModel", rows: int):
        self.model, self.rows = model, int(rows)
        self.layout = model.cache_layout(self.rows)
        model.reserve(self.rows)
        self.data = torch.zeros(self.layout.nbytes, dtype=torch.uint8, device=model.device)
        self.offset = 0

    def reset(self):
        self.data[: self.layout.state_bytes].zero_()
        self.offset = 0

    def accept(self, indices: torch.Tensor, accept_length: int, offset: int):
        """Commit the root row and ``indices`` (rows of the last tree pass)."""
        m = self.model
        rows = torch.zeros(PENDING_ROWS, dtype=torch.int32)
        rows[0] = accept_length
        rows[1:1 + accept_length] = indices.reshape(-1)[:accept_length].to(torch.int32).cpu()
        rows = rows.to(m.device)
        m.fwd.prefix.fill_(offset)
        m.commit_rows(self, rows, rows, m.last_tree_rows, m.fwd.prefix, compact=True)
        self.offset = offset + accept_length + 1


class _Layout:
    """Where the parts of a request's cache are, for a number of K/V rows; host and device run tables."""

    def __init__(self, model: "HybridModel", rows: int):
        a, es = model.args, model.elem
        runs = (_lib.HybridRun * len(a.runs))()
        off = 0

        def take(nbytes):
            nonlocal off
            at, off = off, _up(off + nbytes, ALIGN)
            return at

        for r, (li, inject) in zip(runs, a.runs):
            l = a.layers[li]
            r.layer, r.inject = li, int(inject)
            r.conv_off = take(4 * (a.taps - 1) * a.width)
            for name, nbytes in MIXERS[l.type].state(l.mixer, es).items():
                setattr(r, name, take(nbytes))
        self.state_bytes = off
        for r, (li, _) in zip(runs, a.runs):
            l = a.layers[li]
            for name, nbytes in MIXERS[l.type].rows(l.mixer, es, rows).items():
                setattr(r, name, take(nbytes))
        self.nbytes = max(off, ALIGN)
        off = 0
        for r, (li, _) in zip(runs, a.runs):
            l = a.layers[li]
            if a.design.input_conv:
                r.pend_h = take(4 * PENDING_ROWS * a.width)
            for name, nbytes in MIXERS[l.type].pending(l.mixer, es).items():
                setattr(r, name, take(PENDING_ROWS * nbytes))
        self.pending_bytes = off
        self.runs = runs
        self.dev_runs = _device_bytes(runs, model.device)


def _device_bytes(struct, device) -> torch.Tensor:
    return torch.frombuffer(bytearray(bytes(struct)), dtype=torch.uint8).to(device)


# ---------------------------------------------------------------------- model
class HybridModel:
    tp = None                       # (not built for tensor parallelism)
    vocab_offset = 0
    stateful = True                 # the cache holds recurrent state: a pass is undone only by not committing it

    def __init__(self, args: HybridArgs, weights: Dict[str, torch.Tensor], device, dtype: str = "bfloat16", max_rows: int = 1024):
        if dtype not in ("bfloat16", "float32"):
            raise _lib.B200Error("dtype must be bfloat16 or float32")
        if not (1 <= args.taps <= 8):
            raise _lib.B200Error("the input convolution has 1 to 8 taps")
        args = resolve(args, weights)
        offset = args.design.norm_offset
        self.args, self.device, self.dtype = args, torch.device(device), dtype
        self.model_type = args.model_type
        self.act = torch.float32 if dtype == "float32" else torch.bfloat16
        self.elem = 4 if dtype == "float32" else 2
        self.max_rows = max(256, int(max_rows))
        self._keep: List[torch.Tensor] = []                 # everything the tables point to
        self._weight_bytes = 0
        for name, shape in weight_shapes(args).items():
            if name not in weights:
                raise _lib.B200Error(f"checkpoint has no tensor {name}")
            if tuple(weights[name].shape) != tuple(shape):
                raise _lib.B200Error(f"{name}: expected {tuple(shape)}, found {tuple(weights[name].shape)}")
        self.embed = weights["embed"].to(self.device, torch.bfloat16).contiguous()
        self.layers = (_lib.HybridLayer * len(args.layers))()
        for i, (l, spec) in enumerate(zip(self.layers, args.layers)):
            sub = lambda p: {k[len(p):]: v for k, v in weights.items() if k.startswith(p)}
            l.taps = args.taps
            l.norm1 = self.vector(weights[f"l{i}.norm1"], offset)
            if args.design.input_conv:
                l.conv = self.vector(weights[f"l{i}.canon1"].t())
            MIXERS[spec.type].bind(self, l, spec.mixer, sub(f"l{i}.mix."))
            if spec.mlp is not None:
                l.norm2 = self.vector(weights[f"l{i}.norm2"], offset)
                args.feed_forward(spec).bind(self, l, spec.mlp, sub(f"l{i}.mlp."))
        self.final_norm = self.vector(weights["final.norm"], offset)
        self.head = self.linear(weights["head"])
        self._dev_layers = _device_bytes(self.layers, self.device)
        self._layouts: Dict[int, _Layout] = {}
        self.fwd = FwdInputs(self.device)
        self.tail_pos = torch.zeros(PENDING_ROWS, dtype=torch.int32, device=self.device)
        self.last_tree_rows = 1
        self.dump: Optional[torch.Tensor] = None            # [runs][M][width] fp32: residual stream after every run of the next passes
        self._allocate()

    # ------------------------------------------------------------------ construction
    def vector(self, t: torch.Tensor, add: float = 0.0) -> int:
        v = (t.to(self.device).float() + add).contiguous()
        self._keep.append(v)
        return v.data_ptr()

    def linear(self, *parts: torch.Tensor) -> "_lib.Linear":
        """The row blocks ``parts`` as one matrix: bf16, rows padded to 128, columns to 64."""
        n, k = sum(p.shape[0] for p in parts), parts[0].shape[1]
        w = torch.zeros(_up(n, 128), _up(k, 64), dtype=torch.bfloat16, device=self.device)
        r = 0
        for p in parts:
            w[r:r + p.shape[0], :k].copy_(p)
            r += p.shape[0]
        self._keep.append(w)
        self._weight_bytes += n * k * 2
        return _lib.Linear(w.data_ptr(), n, k, w.shape[1], 0)

    def stack(self, matrices: Sequence[torch.Tensor]) -> "_lib.Linear":
        """Equal matrices one after the other, each padded like ``linear``'s."""
        n, k = matrices[0].shape
        w = torch.zeros(len(matrices), _up(n, 128), _up(k, 64), dtype=torch.bfloat16, device=self.device)
        for i, m in enumerate(matrices):
            w[i, :n, :k].copy_(m)
        self._keep.append(w)
        self._weight_bytes += len(matrices) * n * k * 2
        return _lib.Linear(w.data_ptr(), n, k, w.shape[2], len(matrices))

    def _allocate(self):
        a, R, dev = self.args, self.max_rows, self.device
        act, f32, single = self.act, torch.float32, self.dtype == "float32"
        cols = dict(hb=_up(a.width, 64))
        for spec in a.layers:
            need = [MIXERS[spec.type].buffers(spec.mixer)]
            if spec.mlp is not None:
                need.append(a.feed_forward(spec).buffers(spec.mlp, a.width))
            for k, v in (kv for d in need for kv in d.items()):
                if k in ("zb32", "xg") and single != (k == "zb32"):
                    continue                                # products only one form finishes in its epilogue, or gathers rows for
                k = "zb" if k == "zb32" else k
                cols[k] = max(cols.get(k, 0), v)
        if a.design.norm_out:
            cols["y"] = max(cols.get("y", 0), a.width)
        wide = {"gf", "o32", "y", "q32", "k32", "beta", "lat32", "zr"}       # fp32 in both forms
        z = lambda cols, dt: torch.zeros(R, cols, dtype=dt, device=dev)
        injects = any(i for _, i in a.runs)
        b = dict(x=z(a.width, f32), emb=z(a.width, f32) if injects else None)
        b.update({k: z(v, f32 if k in wide else act) for k, v in cols.items() if v > 0})
        self.buffers = b
        experts = [l for l in self.layers if l.ff_kind == FF_EXPERTS]
        top, n_exp = max([l.top for l in experts], default=0), max([l.experts for l in experts], default=0)
        self.route = torch.zeros(max(_lib.hybrid().b200_hybrid_route_ints(R, top, n_exp), 4), dtype=torch.int32, device=dev)
        deltas = [l for l in self.layers if l.mixer == MIXER_DELTA]
        chunk = max([_lib.hybrid().b200_hybrid_chunk_floats(R, l.heads, l.dim) for l in deltas], default=0)
        self.chunk = torch.zeros(max(chunk, 4), dtype=f32, device=dev)
        self.expanded: List[torch.Tensor] = []
        self.tok_buf = torch.zeros(R, dtype=torch.int32, device=dev)
        self.pos_buf = torch.zeros(R, dtype=torch.int32, device=dev)
        self.prefix_buf = torch.zeros(1, dtype=torch.int32, device=dev)
        self.error = torch.zeros(1, dtype=torch.int32, device=dev)
        self.logits32 = torch.zeros(MAX_ROWS, a.vocab_size, dtype=f32, device=dev)
        self.logits = torch.zeros(MAX_ROWS, a.vocab_size, dtype=torch.float16, device=dev)
        d = _lib.HybridModelDesc()
        d.act_type = 1 if self.dtype == "float32" else 0
        d.width, d.vocab, d.n_layers, d.n_runs, d.max_rows = a.width, a.vocab_size, len(a.layers), len(a.runs), R
        d.injects, d.conv_max_taps = int(injects), a.taps
        d.eps, d.residual_mult, d.softcap, d.norm_out = a.eps, a.residual_mult, a.logit_softcap, int(a.design.norm_out)
        d.embed, d.final_norm, d.head = self.embed.data_ptr(), self.final_norm, self.head
        d.layers = ctypes.cast(self.layers, ctypes.POINTER(_lib.HybridLayer))
        d.dev_layers = self._dev_layers.data_ptr()
        for k, t in b.items():
            setattr(d, k, t.data_ptr() if t is not None else None)
        d.route, d.route_top, d.route_experts = self.route.data_ptr(), top, n_exp
        d.chunk = self.chunk.data_ptr()
        d.error = self.error.data_ptr()
        self._desc = d
        self.pending = torch.zeros(max(self.cache_layout(64).pending_bytes, ALIGN), dtype=torch.uint8, device=dev)
        d.pending = self.pending.data_ptr()
        nbytes = _lib.hybrid().b200_hybrid_attention_workspace_bytes(ctypes.byref(d), R if self._rows_attention() else PENDING_ROWS)
        self.attn_part = torch.zeros(max(nbytes, 16), dtype=torch.uint8, device=dev)
        d.attn_part, d.attn_part_bytes = self.attn_part.data_ptr(), self.attn_part.numel()

    def _rows_attention(self) -> bool:
        """Do prompts too go through the few-row attention kernel (fp32, or head sizes past the prompt kernel's)?"""
        def large(s):
            mx = s.mixer
            if MIXERS[s.type] is Attention:
                return mx["dim"] > 128 or mx["vdim"] > 128
            return MIXERS[s.type] is LatentAttention and (_up(mx["dim"], 16) + _up(mx["rot_dim"], 16) > 256 or mx["vdim"] > 128)
        return self.dtype == "float32" or any(large(s) for s in self.args.layers)

    def reserve(self, rows: int):
        """Room for the keys and values of all heads of a latent layer's ``rows`` cache rows (bf16 prompts; one buffer for all
        layers and caches)."""
        sizes = [LatentAttention.expanded(s.mixer) for s in self.args.layers if MIXERS[s.type] is LatentAttention]
        if self.dtype == "float32" or not sizes or rows <= self._desc.x_rows:
            return
        self.expanded = [torch.zeros(rows * max(c), dtype=self.act, device=self.device) for c in zip(*sizes)]
        self._desc.kx, self._desc.vx, self._desc.x_rows = self.expanded[0].data_ptr(), self.expanded[1].data_ptr(), rows

    @staticmethod
    def random_init(args: HybridArgs, seed: int, device, gen_device=None, dtype: str = "bfloat16", max_rows: int = 1024) -> "HybridModel":
        """Seeded random weights of the design's shapes (stands in for a checkpoint)."""
        device = torch.device(device)
        gdev = torch.device(gen_device) if gen_device is not None else device
        return HybridModel(args, random_weights(args, seed, gdev), device, dtype, max_rows)

    def cache_layout(self, rows: int) -> _Layout:
        if rows not in self._layouts:
            self._layouts[rows] = _Layout(self, rows)
        return self._layouts[rows]

    def make_cache(self, rows: int) -> HybridCache:
        return HybridCache(self, rows)

    def make_batch_cache(self, rows: int, requests: int):
        raise _lib.B200Error("several requests per pass are not built for layer-list decoders")

    def relayout(self):
        """Nothing to do: weights are read as they are stored."""
        return self

    def can_fuse(self) -> bool:
        """False: a pass is a sequence of kernels, not the persistent kernel of the 4-bit models (its step can still be
        captured into a CUDA graph)."""
        return False

    @property
    def launches_per_forward(self) -> int:
        n = 3                                               # embedding, final norm, head
        for li, _ in self.args.runs:
            s = self.args.layers[li]
            n += 1 + MIXERS[s.type].launches                # + a norm before or after each sublayer
            if s.mlp is not None:
                n += 1 + self.args.feed_forward(s).launches
        return n

    @property
    def vocab_local(self) -> int:
        return self.args.vocab_size

    def linear_weight_bytes(self) -> int:
        """Bytes of matrix weights a pass over one token streams: every layer run (of its experts the chosen ones), and the head."""
        def nbytes(x):
            n = sum(l.n * l.k * 2 * max(l.groups, 1) for l in (x.in_, x.out, x.low, x.absorb, x.value, x.router))
            return n + sum(l.n * l.k * 2 * (x.top if x.ff_kind == FF_EXPERTS else 1) for l in (x.up, x.down))
        per = [nbytes(x) for x in self.layers]
        return sum(per[li] for li, _ in self.args.runs) + self.head.n * self.head.k * 2

    def greedy_token(self, logits_row: torch.Tensor) -> int:
        return int(torch.argmax(logits_row.float(), dim=-1))

    def check_fused_error(self):
        """Raise if a bounded wait inside a kernel ever gave up (synchronises)."""
        code = int(self.error)
        if code != 0:
            self.error.zero_()
            raise _lib.B200Error(f"a bounded wait gave up inside a kernel of the pass (code {code})")

    # ------------------------------------------------------------------ passes
    def _run(self, p: "_lib.HybridPass", cache: HybridCache):
        d = self._desc
        d.runs = ctypes.cast(cache.layout.runs, ctypes.POINTER(_lib.HybridRun))
        d.dev_runs = cache.layout.dev_runs.data_ptr()
        p.cache, p.cache_rows = cache.data.data_ptr(), cache.rows
        p.tail_pos = self.tail_pos.data_ptr()
        p.dump = self.dump.data_ptr() if self.dump is not None else None
        _lib.check(_lib.hybrid().b200_hybrid_forward(ctypes.byref(d), ctypes.byref(p), _lib.stream_ptr(self.device)),
                   "b200_hybrid_forward")

    def forward_device(self, M: int, cache: HybridCache, write_off: int, tail: int, fwd: Optional[FwdInputs] = None,
                       logits_rows: Optional[int] = None, row_index: Optional[torch.Tensor] = None, requests: int = 1,
                       commit: bool = False):
        """One pass over ``M`` rows whose tokens / positions / masks / committed length sit in ``fwd`` (device memory).
        Default: tail rows ``write_off ..`` after ``prefix`` committed ones under the tree mask, as ``llama.Model``'s;
        nothing is committed (``commit_rows`` does that).  ``commit=True``: the rows continue the sequence and are
        committed by the pass (masks unused).  Returns fp16 logits; ``logits32`` holds the fp32 ones."""
        if requests != 1:
            raise _lib.B200Error("several requests per pass are not built for layer-list decoders")
        if not (1 <= M <= MAX_ROWS and 1 <= tail <= MAX_TAIL and write_off + M <= tail):
            raise _lib.B200Error("forward_device: need 1 <= M <= 32, tail <= 64, write_off + M <= tail")
        f = fwd or self.fwd
        rows = M if logits_rows is None else logits_rows
        p = _lib.HybridPass()
        p.M, p.tree, p.write_off, p.tail, p.rows_out, p.max_keys = M, int(not commit), write_off, tail, rows, cache.rows
        p.tokens, p.pos, p.mask, p.prefix = f.tokens.data_ptr(), f.pos.data_ptr(), f.mask.data_ptr(), f.prefix.data_ptr()
        p.row_index = row_index.data_ptr() if row_index is not None else None
        p.logits, p.logits16 = self.logits32.data_ptr(), self.logits.data_ptr()
        self.last_tree_rows = M
        self._run(p, cache)
        return self.logits[:rows]

    def commit_rows(self, cache: HybridCache, count: torch.Tensor, rows: Optional[torch.Tensor], tree_rows: int,
                    prefix: Optional[torch.Tensor], compact: bool):
        """Advance the cache over ``count[0] + 1`` rows of the last tree pass: row 0, then ``rows[1 ..]`` (None: 1 ..)."""
        d, ptr = self._desc, _lib.ptr
        d.runs = ctypes.cast(cache.layout.runs, ctypes.POINTER(_lib.HybridRun))
        d.dev_runs = cache.layout.dev_runs.data_ptr()
        _lib.check(_lib.hybrid().b200_hybrid_commit(ctypes.byref(d), ptr(cache.data), cache.rows, ptr(count), ptr(rows), tree_rows,
                                                    ptr(prefix), int(compact), _lib.stream_ptr(self.device)), "b200_hybrid_commit")

    # hooks of the decoding loop ------------------------------------------------------------------
    def commit_catchup(self, cache: HybridCache, accept: torch.Tensor):
        """After a draft's catch-up pass: its first ``accept[0] + 1`` rows are part of the sequence."""
        self.commit_rows(cache, accept, None, MAX_ROWS, None, compact=False)

    def commit_accepted(self, cache: HybridCache, accept_rows: torch.Tensor, ctl: torch.Tensor, tree_rows: int):
        """After acceptance: the root and the accepted nodes are part of the sequence, their K/V rows move together."""
        self.commit_rows(cache, accept_rows, accept_rows, tree_rows, self.fwd.prefix, compact=True)

    def argmax_rows(self, logits: torch.Tensor, rows: int, key: torch.Tensor):
        _lib.check(_lib.lib().b200_logits_argmax_f32(_lib.ptr(self.logits32), rows, self.args.vocab_size, _lib.ptr(key),
                                                     _lib.stream_ptr(self.device)), "b200_logits_argmax_f32")

    # ------------------------------------------------------------------ prompts and chains
    def __call__(self, inputs: torch.Tensor, cache: Optional[HybridCache] = None, mask: Optional[torch.Tensor] = None,
                 position_ids: Optional[Union[torch.Tensor, int]] = None, flat_rope: bool = False, logits_last_only: bool = False,
                 want: Optional[Sequence[int]] = None) -> Optional[torch.Tensor]:
        """fp32 logits ``(1, L, V)`` of the next ``L`` tokens of the sequence in ``cache``, any ``L`` (passes of up to
        ``max_rows`` rows); ``logits_last_only``: of the last token; ``want``: of the given places among the tokens
        (in their order; None when empty).  With an additive ``mask`` ``(1,1,L,offset+L)`` of 0 / -inf the rows form a tree
        after the committed sequence: nothing is committed until ``cache.accept``."""
        if cache is None:
            raise _lib.B200Error("a cache is required")
        inputs = inputs.reshape(-1).to(torch.int32)
        n = inputs.numel()
        if cache.offset + n > cache.rows:
            raise _lib.B200Error("KV cache is full")
        if mask is not None:
            return self._tree_call(inputs, cache, mask, position_ids)
        if position_ids is not None:
            raise _lib.B200Error("explicit positions need an explicit mask")
        if logits_last_only:
            want = [n - 1]
        elif want is None:
            want = range(n)
        want = list(want)
        out = torch.empty(len(want), self.args.vocab_size, dtype=torch.float32, device=self.device) if want else None
        done = 0
        for c0 in range(0, n, self.max_rows):
            m = min(self.max_rows, n - c0)
            here = [(i, w - c0) for i, w in enumerate(want) if c0 <= w < c0 + m]
            self.tok_buf[:m].copy_(inputs[c0:c0 + m])
            torch.arange(cache.offset, cache.offset + m, dtype=torch.int32, out=self.pos_buf[:m])
            self.prefix_buf.fill_(cache.offset)
            p = _lib.HybridPass()
            p.M, p.rows_out, p.max_keys = m, len(here), cache.offset + m
            p.tokens, p.pos, p.prefix = self.tok_buf.data_ptr(), self.pos_buf.data_ptr(), self.prefix_buf.data_ptr()
            if here:
                if len(here) > m:
                    raise _lib.B200Error("each place can be wanted once")
                rows = torch.tensor([w for _, w in here], dtype=torch.int32).to(self.device)
                contiguous = [i for i, _ in here] == list(range(done, done + len(here)))
                dst = out[done:done + len(here)] if contiguous else torch.empty(len(here), self.args.vocab_size, dtype=torch.float32,
                                                                                device=self.device)
                p.out_rows, p.logits = rows.data_ptr(), dst.data_ptr()
            self._run(p, cache)
            if here and not contiguous:
                out[torch.tensor([i for i, _ in here], device=self.device)] = dst
            done += len(here)
            cache.offset += m
        return out.unsqueeze(0) if out is not None else None

    def _tree_call(self, inputs: torch.Tensor, cache: HybridCache, mask: torch.Tensor, position_ids):
        n, off = inputs.numel(), cache.offset
        if n > MAX_ROWS or not isinstance(position_ids, torch.Tensor):
            raise _lib.B200Error("a tree pass has at most 32 rows and explicit positions")
        vis = (mask.reshape(n, -1).float().cpu() == 0)
        if vis.shape[1] != off + n or not bool(vis[:, :off].all()):
            raise _lib.B200Error("mask must have cache.offset + L columns and show every committed one")
        bits = [sum(1 << j for j in range(n) if vis[i, off + j]) for i in range(n)]
        f = self.fwd
        f.tokens[:n].copy_(inputs)
        f.pos[:n].copy_(position_ids.reshape(-1).to(torch.int32))
        f.mask[:n].copy_(torch.tensor(bits, dtype=torch.int64))
        f.prefix.fill_(off)
        self.forward_device(n, cache, 0, n)
        cache.offset = off + n
        return self.logits32[:n].clone().unsqueeze(0)


# ---------------------------------------------------------------------- random stand-ins
def random_weights(args: HybridArgs, seed: int, device) -> Dict[str, torch.Tensor]:
    """Seeded bf16 weights of a design's shapes, scaled so that the stream keeps its size through the layers."""
    gen = torch.Generator(device=device).manual_seed(seed)
    out: Dict[str, torch.Tensor] = {}
    for name, shape in weight_shapes(args).items():
        r = torch.randn(shape, generator=gen, device=device)
        leaf, flat = name.rsplit(".", 1)[-1], len(shape) == 1
        if name == "embed":
            t = r
        elif leaf.startswith("norm") or name == "final.norm":
            t = 0.1 * r + (1.0 if ".mix." in name else 1.0 - args.design.norm_offset)
        elif leaf == "canon1":
            t = 0.3 * r
        elif leaf == "conv":
            t = r * shape[1] ** -0.5
        elif leaf == "act":
            t = 0.4 + 0.1 * r
        elif leaf == "b" and flat and ".mix." in name:
            t = 2.0 + 2.0 * r
        elif leaf == "lower":
            t = torch.sigmoid(r - 1.0)
        elif leaf == "A_log":
            t = 0.5 * r
        elif leaf == "dt_bias":
            t = 0.5 * r - 3.0
        elif flat:
            t = 0.1 * r
        else:
            t = r * shape[1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


def _preset(vocab, width, ff, period, count, attn, rec, window, keep, loop=None, taps=4):
    layers = []
    for i in range(count):
        a = i % period == 0
        layers.append(dict(type="attention" if a else "hgrn2", mlp=dict(kind="dense", ff=ff),
                           mixer=dict(heads=attn[0], kv_heads=attn[1], dim=attn[2], vdim=attn[3], diff=0.4, scale=attn[2] ** -0.5,
                                      mask=dict(size=window, keep_first=keep)) if a
                           else dict(heads=rec[0], dim=rec[1], vdim=rec[2])))
    return dict(architecture="Zaverax", vocab=vocab, width=width, layers=layers, canon=dict(taps=taps), norm=dict(eps=1e-5),
                residual_mult=0.7, logit_softcap=20.0, loop=loop)


def _zokelix_preset(vocab, width, count, period, delta, latent, ff, experts, top, expert_ff, original=4096):
    """Every ``period``-th layer latent attention, the others delta rules; a dense feed-forward in the first layer, experts in
    the others.  delta: heads, kv_heads, dim, vdim; latent: heads, dim, rot_dim, vdim, kv_rank."""
    heads, dim, rot, vdim, rank = latent
    layers = []
    for i in range(count):
        if i % period == period - 1:
            spin = dict(dims=rot, base=10000.0, scaling=dict(factor=8.0, original=original, fast=32.0, slow=1.0))
            mx, kind = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, scale=(dim + rot) ** -0.5, rot=spin), "latent_attention"
        else:
            mx, kind = dict(zip(("heads", "kv_heads", "dim", "vdim"), delta), conv=4), "channel_delta"
        mlp = dict(kind="dense", ff=ff) if i == 0 else dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=expert_ff, limit=7.0))
        layers.append(dict(type=kind, mixer=mx, mlp=mlp))
    return dict(architecture="Zokelix", vocab=vocab, width=width, layers=layers, norm=dict(eps=1e-5))


def preset_config(name: str) -> dict:
    """Configurations with random-init weights: tiny ones for tests, others whose layers have the size of real models'."""
    presets = {
        "tiny-zaverax": lambda: _preset(512, 192, 320, 2, 4, (6, 2, 32, 64), (3, 40, 48), 24, 3, dict(start=1, stop=3, times=2)),
        # the width, feed-forward and layer count of the 4-bit presets llama3.2-1b and llama3-8b
        "zaverax-1b": lambda: _preset(128256, 2048, 8192, 4, 16, (16, 4, 64, 128), (16, 128, 128), 1024, 4),
        "zaverax-8b": lambda: _preset(128256, 4096, 14336, 4, 32, (32, 8, 64, 128), (32, 128, 128), 2048, 4),
        "tiny-zokelix": lambda: _zokelix_preset(512, 176, 4, 2, (4, 2, 40, 24), (3, 32, 12, 48, 72), 208, 10, 3, 56, original=64),
        # the same widths and layer counts, with as many feed-forward weights per token
        "zokelix-1b": lambda: _zokelix_preset(128256, 2048, 16, 4, (16, 16, 128, 128), (16, 128, 64, 128, 512), 5504, 32, 4, 1408),
        "zokelix-8b": lambda: _zokelix_preset(128256, 4096, 32, 4, (32, 32, 128, 128), (32, 128, 64, 128, 512), 9600, 32, 4, 2432),
    }
    if name not in presets:
        raise KeyError(f"unknown configuration {name!r}; known: {sorted(presets)}")
    return presets[name]()
