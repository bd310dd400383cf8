"""Layer-list decoders, what needs no GPU: configuration, tables, ABI, oracle sanity, runner conventions."""
import ctypes
import json
import os
import re
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_cases as hc
from oracle import hybrid_ref

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_header_symbols_are_exported(be):
    text = re.sub(r"/\*.*?\*/", "", open(os.path.join(ROOT, "include", "b200_hybrid.h")).read(), flags=re.S)
    names = set(re.findall(r"\b(b200_hybrid_[a-z0-9_]+)\s*\(", text))
    assert {"b200_hybrid_forward", "b200_hybrid_commit", "b200_hybrid_linear"} <= names
    for n in names:
        assert hasattr(be._lib.hybrid(), n), n


def test_struct_mirrors(be, tmp_path):
    """Sizes and field offsets of the ctypes mirrors against the header, as a C compiler lays it out."""
    L = be._lib
    mirrors = {"b200_linear": L.Linear, "b200_hybrid_layer": L.HybridLayer, "b200_hybrid_run": L.HybridRun, "b200_hybrid_model": L.HybridModelDesc,
               "b200_hybrid_pass": L.HybridPass}
    fields = [(s, c, f[0]) for s, c in mirrors.items() for f in c._fields_]
    c_name = {"in_": "in", "lambda_": "lambda"}
    prog = "#include <stdio.h>\n#include <stddef.h>\n#include \"b200_hybrid.h\"\nint main(void) {\n"
    prog += "".join(f'printf("%zu\\n", sizeof({s}));\n' for s in mirrors)
    prog += "".join(f'printf("%zu\\n", offsetof({s}, {c_name.get(f, f)}));\n' for s, _, f in fields) + "return 0; }\n"
    (tmp_path / "sizes.c").write_text(prog)
    subprocess.run(["gcc", "-I", os.path.join(ROOT, "include"), str(tmp_path / "sizes.c"), "-o", str(tmp_path / "sizes")], check=True, timeout=120)
    got = [int(x) for x in subprocess.run([str(tmp_path / "sizes")], capture_output=True, text=True, check=True, timeout=60).stdout.split()]
    assert got == [ctypes.sizeof(c) for c in mirrors.values()] + [getattr(c, f).offset for _, c, f in fields]


def test_bad_arguments_are_refused_before_any_launch(be):
    L = be._lib.hybrid()
    m, p = be._lib.HybridModelDesc(), be._lib.HybridPass()
    assert L.b200_hybrid_forward(ctypes.byref(m), ctypes.byref(p), None) == -1
    assert L.b200_hybrid_commit(ctypes.byref(m), None, 0, None, None, 0, None, 0, None) == -1


def test_runs_of_a_loop(be):
    c = hc.mixed()
    a = be.HybridArgs.from_config(c)
    assert a.runs == [(0, False), (1, False), (2, False), (3, True), (1, False), (2, False), (3, False), (4, False)]
    assert [i for i, _ in hybrid_ref.layer_order(c)] == [i for i, _ in a.runs]
    one = hc.mixed()
    one["loop"] = dict(start=0, stop=5, times=3)
    a = be.HybridArgs.from_config(one)
    assert [i for i, _ in a.runs] == [0, 1, 2, 3, 4] * 3 and [j for j, (_, s) in enumerate(a.runs) if s] == [4, 9]
    one["loop"] = None
    assert be.HybridArgs.from_config(one).num_hidden_layers == 5


def test_unknown_parts_raise(be):
    c = hc.mixed()
    c["layers"][0]["type"] = "other"
    with pytest.raises(be._lib.B200Error):
        be.HybridArgs.from_config(c)
    with pytest.raises(be._lib.B200Error):
        be.load.model_builder({"architecture": "other"})
    with pytest.raises(be._lib.B200Error):
        be.load.model_builder({"model_type": "other"})


def test_checkpoint_tensors_are_checked(be):
    c = hc.mixed()
    w = hc.weights(c)
    assert set(w) == set(be.hybrid.weight_shapes(be.HybridArgs.from_config(c)))
    bad = dict(w)
    bad.pop("l1.mix.g")
    with pytest.raises(be._lib.B200Error):
        be.HybridModel(be.HybridArgs.from_config(c), bad, "cpu")
    bad = dict(w, **{"l1.mix.g": w["l1.mix.g"][1:]})
    with pytest.raises(be._lib.B200Error):
        be.HybridModel(be.HybridArgs.from_config(c), bad, "cpu")


def test_cache_parts_do_not_overlap(be):
    c = hc.mixed()
    m = be.HybridModel(be.HybridArgs.from_config(c), hc.weights(c), "cpu")
    rows = 77
    lay = m.cache_layout(rows)
    parts = []
    for r, (li, _) in zip(lay.runs, m.args.runs):
        mx = c["layers"][li]["mixer"]
        parts.append((r.conv_off, 4 * 2 * c["width"]))
        if c["layers"][li]["type"] == "hgrn2":
            parts.append((r.state_off, 4 * mx["heads"] * mx["dim"] * mx["vdim"]))
        else:
            parts.append((r.k_off, 2 * mx["kv_heads"] * rows * 2 * -(-mx["dim"] // 16) * 16))
            parts.append((r.v_off, 2 * mx["kv_heads"] * rows * -(-mx["vdim"] // 16) * 16))
    parts.sort()
    for (a, n), (b, _) in zip(parts, parts[1:] + [(lay.nbytes, 0)]):
        assert a % 256 == 0 and a + n <= b
    states = [r.state_off for r, (li, _) in zip(lay.runs, m.args.runs) if c["layers"][li]["type"] == "hgrn2"]
    assert len(set(states)) == len(states) and max(states) < lay.state_bytes <= min(
        r.k_off for r, (li, _) in zip(lay.runs, m.args.runs) if c["layers"][li]["type"] == "attention")
    cache = m.make_cache(rows)
    cache.data.fill_(1)
    cache.offset = 5
    cache.reset()
    assert cache.offset == 0 and int(cache.data[: lay.state_bytes].sum()) == 0 and int(cache.data[lay.state_bytes]) == 1


def test_differential_constants(be):
    c = hc.config([hc.attention(diff=0.35)])
    w = hc.weights(c, 3)
    m = be.HybridModel(be.HybridArgs.from_config(c), w, "cpu")
    n = hc.as_numpy(w)
    lam = hybrid_ref.differential_lambda(*(n["l0.mix." + k] for k in ("lq1", "lk1", "lq2", "lk2")), 0.35)
    assert abs(m.layers[0].lambda_ - lam) < 1e-6 and abs(m.layers[0].out_scale - 0.65) < 1e-6
    assert m.layers[0].window == 20 and m.layers[0].keep_first == 2


def test_oracle_mechanisms():
    """The restatement against closed forms."""
    rng = np.random.default_rng(0)
    h = rng.standard_normal((6, 4))
    w = np.zeros((4, 3))
    w[:, 1] = 2.0                                            # the middle of three taps: the previous token
    out = hybrid_ref.causal_conv_residual(h, w)
    assert np.allclose(out[0], h[0]) and np.allclose(out[1:], h[1:] + 2 * h[:-1])
    f, q, v = rng.uniform(0.1, 0.9, (5, 3)), rng.standard_normal((5, 3)), rng.standard_normal((5, 2))
    o = hybrid_ref.gated_recurrence(q, f, v)
    want = sum(np.sum(q[4] * (1 - f[j]) * np.prod(f[j + 1:5], axis=0)) * v[j] for j in range(5))
    assert np.allclose(o[4], want)
    vis = [[hybrid_ref.visible(i, j, 3, 2) for j in range(8)] for i in range(8)]
    assert [j for j in range(8) if vis[7][j]] == [0, 1, 5, 6, 7] and [j for j in range(8) if vis[1][j]] == [0, 1]
    z = rng.standard_normal((2, 9))
    y = hybrid_ref.polynorm(z, (0.0, 0.0, 1.0, 0.5), 0.0)
    assert np.allclose(np.mean((y - 0.5) ** 2, axis=1), 1.0)


def test_replay_keeps_and_reuses_caches(be):
    class Fake:
        made = 0

        def make_cache(self, rows):
            Fake.made += 1

            class C:
                def reset(self):
                    self.seen = []
            return C()

        def __call__(self, toks, cache, want):
            cache.seen += toks.tolist()
            return torch.tensor([[[float(sum(cache.seen))]] * len(want)]).reshape(1, len(want), 1) if want else None

        def check_fused_error(self):
            pass

    r = be.trace.Replay(Fake(), 64)
    assert r.step(dict(entries=[dict(id="a", tokens=[1, 2], want=[])], end=[])) is None
    assert r.step(dict(entries=[dict(id="b", tokens=[5], want=[0]), dict(id="a", tokens=[3], want=[0])], end=["a"])).flatten().tolist() == [5.0, 6.0]
    assert r.step(dict(entries=[dict(id="c", tokens=[7], want=[0])], end=["c", "b"])).flatten().tolist() == [7.0]
    assert Fake.made == 2 and len(r.free) == 2 and not r.live


def test_runner_refuses_fp32_where_there_is_none(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "llama"}))
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path)], input="", capture_output=True, text=True, timeout=300)
    assert p.returncode == 3


def test_presets(be):
    for n in ("tiny-zaverax", "zaverax-1b", "zaverax-8b", "tiny-zokelix", "zokelix-1b", "zokelix-8b"):
        be.HybridArgs.from_config(be.hybrid.preset_config(n))
    with pytest.raises(KeyError):
        be.hybrid.preset_config("none")


# ---------------------------------------------------------------------- Zokelix
def test_zokelix_tensors_and_ranks(be):
    c = hc.zokelix_mixed()
    w = hc.zokelix_weights(c, 0, (13, 5))
    a = be.hybrid.resolve(be.HybridArgs.from_config(c), w)
    assert a.layers[0].mixer["decay_rank"] == 13 and a.layers[0].mixer["gate_rank"] == 5
    assert {k: tuple(v.shape) for k, v in w.items()} == be.hybrid.weight_shapes(a)
    m = be.HybridModel(be.HybridArgs.from_config(c), w, "cpu")
    assert m.layers[0].low_rank == 18 and m.layers[0].low.n == 4 * (20 + 28) and m.layers[0].low.k == 18
    for bad in ("l0.mix.a1", "l1.mix.uk", "l3.mlp.e4.down", "l1.mlp.down.b"):
        v = dict(w)
        v.pop(bad)
        with pytest.raises(be._lib.B200Error):
            be.HybridModel(be.HybridArgs.from_config(c), v, "cpu")
    with pytest.raises(be._lib.B200Error):
        be.HybridModel(be.HybridArgs.from_config(c), dict(w, **{"l0.mix.a2": w["l0.mix.a2"][:, 1:]}), "cpu")
    c["layers"][1]["mlp"]["kind"] = "other"
    with pytest.raises(be._lib.B200Error):
        be.HybridArgs.from_config(c)


def test_zokelix_weight_layouts(be):
    """What the kernels read, taken apart again: alternating branches, reordered queries, transposed stacks, block rows."""
    c = hc.zokelix_mixed()
    w = hc.weights(c, 1)
    m = be.HybridModel(be.HybridArgs.from_config(c), w, "cpu")
    at = {t.data_ptr(): t for t in m._keep}
    up = at[m.layers[1].up.w]
    ff = c["layers"][1]["mlp"]["ff"]
    assert torch.equal(up[0:2 * ff:2, :104], w["l1.mlp.gate"]) and torch.equal(up[1:2 * ff:2, :104], w["l1.mlp.up"])
    assert torch.equal(at[m.layers[1].up_bias][1::2], w["l1.mlp.up.b"].float())
    ex, ey = at[m.layers[3].up.w], at[m.layers[3].down.w]
    assert torch.equal(ex[4, 1:40:2, :104], w["l3.mlp.e4.up"]) and torch.equal(ey[2, :104, :20], w["l3.mlp.e2.down"])
    assert m.layers[3].up.groups == 5 and not bool(ex[:, 40:].any())
    mx = c["layers"][1]["mixer"]
    H, d, r, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["kv_rank"]
    q = w["l1.mix.q"].view(H, d + r, -1)
    rows = at[m.layers[1].in_.w]
    assert torch.equal(rows[d:2 * d, :104], q[1, :d]) and torch.equal(rows[H * d + r:H * d + 2 * r, :104], q[1, d:])
    ab = at[m.layers[1].absorb.w]
    assert ab.shape == (H, 128, 64) and torch.equal(ab[2, :rank, :d], w["l1.mix.uk"].view(H, d, rank)[2].t())
    low = at[m.layers[0].low.w]
    assert torch.equal(low[:80, :11], w["l0.mix.a2"]) and not bool(low[:80, 11:].any()) and not bool(low[80:, :11].any())
    rate = at[m.layers[0].decay_rate]
    assert np.allclose(rate.numpy(), np.exp(w["l0.mix.A_log"].double().numpy()).repeat(20), rtol=1e-6)


def test_rotation_frequencies(be):
    for rot in (dict(dims=10, base=1000.0), dict(dims=64, base=10000.0, scaling=dict(factor=8.0, original=4096, fast=32.0, slow=1.0)),
                dict(dims=6, base=77.0, scaling=dict(factor=2.5, original=300, fast=3.0, slow=3.0)),
                dict(dims=8, base=50.0, scaling=dict(factor=4.0, original=10, fast=64.0, slow=32.0))):
        f, mag = be.hybrid.rotation(rot)
        g, want = hybrid_ref.rotation_frequencies(rot)
        assert np.allclose(f.numpy(), g, rtol=1e-12) and abs(mag - want) < 1e-12
    f, mag = be.hybrid.rotation(dict(dims=64, base=10000.0, scaling=dict(factor=8.0, original=4096, fast=32.0, slow=1.0)))
    plain = be.hybrid.rotation(dict(dims=64, base=10000.0))[0]
    assert float(f[0]) == float(plain[0]) and abs(float(f[-1] / plain[-1]) - 1 / 8) < 1e-12 and abs(mag - (0.1 * np.log(8) + 1)) < 1e-12


def test_zokelix_cache_parts_do_not_overlap(be):
    c = hc.zokelix_mixed()
    for dtype, es in (("bfloat16", 2), ("float32", 4)):
        m = be.HybridModel(be.HybridArgs.from_config(c), hc.weights(c), "cpu", dtype)
        rows = 77
        lay = m.cache_layout(rows)
        state, grows, pend = [], [], []
        for r, l in zip(lay.runs, c["layers"]):
            mx = l["mixer"]
            if l["type"] == "channel_delta":
                C = -(-(2 * mx["kv_heads"] * mx["dim"] + mx["heads"] * mx["vdim"]) // 8) * 8
                state += [(r.state_off, 4 * mx["heads"] * mx["dim"] * mx["vdim"]), (r.mix_off, es * (mx["conv"] - 1) * C)]
                pend += [(r.pend_c, 64 * es * C), (r.pend_k, 256 * mx["kv_heads"] * mx["dim"]), (r.pend_b, 256 * mx["heads"]),
                         (r.pend_g, 256 * mx["heads"] * mx["dim"]), (r.pend_v, 64 * es * mx["heads"] * mx["vdim"])]
            else:
                grows.append((r.k_off, es * rows * (-(-mx["kv_rank"] // 16) * 16 + -(-mx["rot_dim"] // 16) * 16)))
        for parts, end in ((sorted(state), lay.state_bytes), (sorted(grows), lay.nbytes), (sorted(pend), lay.pending_bytes)):
            for (a, n), (b, _) in zip(parts, parts[1:] + [(end, 0)]):
                assert a % 256 == 0 and a + n <= b
        assert min(a for a, _ in grows) >= lay.state_bytes
        cache = m.make_cache(rows)
        assert (m._desc.x_rows == rows) == (dtype == "bfloat16")
        cache.data.fill_(1)
        cache.reset()
        assert int(cache.data[: lay.state_bytes].sum()) == 0 and int(cache.data[lay.state_bytes]) == 1


def test_zokelix_oracle_mechanisms():
    rng = np.random.default_rng(1)
    # one key channel, full rate, no decay: the state holds the last value written for that key
    k, v = np.zeros((4, 3)), rng.standard_normal((4, 2))
    k[[0, 2], 0], k[[1, 3], 1] = 1.0, 1.0
    q = np.tile(np.array([1.0, 0.0, 0.0]), (4, 1))
    o = hybrid_ref.delta_rule(q, k, v, np.ones((4, 3)), np.ones(4))
    assert np.allclose(o, [v[0], v[0], v[2], v[2]])
    o = hybrid_ref.delta_rule(q, k, v, np.full((4, 3), 0.5), np.ones(4))
    assert np.allclose(o, [v[0], v[0] / 2, v[2], v[2] / 2])
    h = rng.standard_normal((6, 4))
    w = np.zeros((4, 3))
    w[:, 0] = 2.0
    out = hybrid_ref.causal_conv(h, w)
    assert not out[:2].any() and np.allclose(out[2:], 2 * h[:-2])
    # scores of rotated vectors depend on the distance alone
    rot = dict(dims=4, base=30.0)
    a, b = rng.standard_normal((1, 4)), rng.standard_normal((1, 4))
    s = [float(hybrid_ref.rotate_interleaved(a, [p + 5], rot)[0] @ hybrid_ref.rotate_interleaved(b, [p], rot)[0]) for p in (0, 7, 100)]
    assert np.allclose(s, s[0])
    assert np.allclose(hybrid_ref.gelu_tanh(np.array([0.0, 30.0, -30.0])), [0.0, 30.0, 0.0])
    y = hybrid_ref.expert(np.array([1.0]), np.array([[9.0]]), np.array([[-9.0]]), np.array([[1.0]]), 2.0)
    assert np.allclose(y, 2.0 * hybrid_ref.sigmoid(3.404) * -1.0)
