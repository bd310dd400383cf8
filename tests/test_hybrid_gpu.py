"""Layer-list decoders on the GPU against the plain restatement (``oracle/hybrid_ref.py``)."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_cases as hc
from oracle import hybrid_ref

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 3e-2}
DTYPES = ("float32", "bfloat16")


def build(be, cfg, w, dtype, max_rows=256):
    return be.HybridModel(be.HybridArgs.from_config(cfg), w, "cuda:0", dtype, max_rows=max_rows)


def feed(model, toks, cuts=None, cache=None):
    """Logits of every position, the tokens given in portions of ``cuts`` (the last repeated to the end)."""
    cache = cache if cache is not None else model.make_cache(max(64, len(toks)))
    out, at, cuts = [], 0, list(cuts or [len(toks)])
    while at < len(toks):
        n = min(cuts[0] if len(cuts) == 1 else cuts.pop(0), len(toks) - at)
        out.append(model(torch.tensor(toks[at:at + n], dtype=torch.int32), cache)[0])
        at += n
    model.check_fused_error()
    return torch.cat(out).double().cpu().numpy()


def errors(got, ref):
    """Per position, relative to the size of the logits."""
    return np.sqrt(((got - ref) ** 2).mean(1)) / np.sqrt((ref ** 2).mean())


def agree(got, ref, dtype):
    e = errors(got, ref)
    assert e.max() < TOL[dtype], f"position {e.argmax()}: {e.max():.2e}"


def check(be, cfg, n, dtype, cuts=None, seed=0, w=None, toks=None):
    w = w or hc.weights(cfg, seed)
    toks = hc.tokens(cfg, n, seed) if toks is None else toks
    ref, _ = hybrid_ref.HybridOracle(cfg, hc.as_numpy(w)).forward(toks)
    for c in (cuts or [None]):
        agree(feed(build(be, cfg, w, dtype), toks, c), ref, dtype)


# ---------------------------------------------------------------------- products
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,k", [(40, 24), (128, 64), (300, 200), (1000, 1040), (256, 4096)])
def test_linear(be, cuda, dtype, n, k):
    cfg = hc.config([hc.recurrence()])
    m = build(be, cfg, hc.weights(cfg), dtype, max_rows=512)
    g = torch.Generator().manual_seed(n + k)
    w = torch.randn(n, k, generator=g).bfloat16()
    lin = m.linear(w)
    x = torch.zeros(512, lin.pitch, dtype=m.act, device=cuda)
    x[:, :k] = torch.randn(512, k, generator=g).to(cuda)
    ref = x[:, :k].double().cpu() @ w.double().t()
    import ctypes
    for rows in (1, 3, 16, 17, 32, 50, 64, 100, 128, 129, 300, 512):
        y = torch.full((512, n + 3), 7.0, device=cuda)
        rc = be._lib.hybrid().b200_hybrid_linear(ctypes.byref(m._desc), ctypes.byref(lin), be._lib.ptr(x), lin.pitch, 512, be._lib.ptr(y),
                                                 n + 3, rows, be._lib.stream_ptr(cuda))
        assert rc == 0
        m.check_fused_error()
        err = (y[:rows, :n].double().cpu() - ref[:rows]).abs().max() / k ** 0.5
        assert err < 1e-4, (rows, float(err))            # sums of k terms: fp32 accumulation
        assert bool((y[rows:] == 7.0).all()) and bool((y[:, n:] == 7.0).all())


# ---------------------------------------------------------------------- one mechanism at a time
ATTN = {
    "window": hc.attention(size=20, keep_first=0),
    "kept": hc.attention(size=6, keep_first=5),
    "one": hc.attention(size=1, keep_first=1),
    "wide": hc.attention(size=4000, keep_first=0),
    "allkept": hc.attention(size=2, keep_first=500),
    "own_kv": hc.attention(heads=3, kv_heads=3, dim=16, vdim=16, size=30),
    "groups": hc.attention(heads=20, kv_heads=1, dim=8, vdim=24, size=70),
    "big": hc.attention(heads=2, kv_heads=1, dim=144, vdim=200, size=50, keep_first=4),
    "headdims": hc.attention(heads=2, kv_heads=2, dim=128, vdim=112, size=90, keep_first=70),
    "nodiff": hc.attention(diff=0.0),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ATTN))
def test_attention_alone(be, cuda, name, dtype):
    cfg = hc.config([ATTN[name]], taps=1)
    check(be, cfg, 150, dtype, [[150], [1], [64, 2, 17, 3, 1]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(3, 20, 28), (1, 64, 32), (2, 100, 130), (1, 200, 17), (5, 7, 3)])
def test_recurrence_alone(be, cuda, sizes, dtype):
    h, d, dv = sizes
    cfg = hc.config([hc.recurrence(heads=h, dim=d, vdim=dv)], taps=1)
    check(be, cfg, 120, dtype, [[120], [1], [2, 33, 16, 5]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 5, 8])
def test_input_convolution(be, cuda, taps, dtype):
    cfg = hc.config([hc.recurrence(), hc.attention()], taps=taps)
    check(be, cfg, 90, dtype, [[90], [1], [2], [3, 1, 70, 2, 1]], seed=taps)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [8, 75, 640])
def test_feed_forward_alone(be, cuda, ff, dtype):
    cfg = hc.config([hc.recurrence(ff=ff)], taps=1)
    w = hc.weights(cfg, ff)
    w["l0.mix.o"].zero_()                                   # the mixer contributes nothing
    check(be, cfg, 40, dtype, [[40], [1]], w=w)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", [dict(cap=None), dict(cap=2.0), dict(m=1.0), dict(m=0.3), dict(eps=0.3), dict(width=64, vocab=128), dict(width=201, vocab=77)])
def test_constants(be, cuda, kw, dtype):
    check(be, hc.config([hc.recurrence(ff=50), hc.attention(ff=60)], **kw), 40, dtype, [[40], [7, 1]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("loop", [None, dict(start=0, stop=1, times=2), dict(start=0, stop=3, times=3), dict(start=1, stop=2, times=4),
                                  dict(start=2, stop=3, times=2), dict(start=1, stop=3, times=1)])
def test_repeated_layers(be, cuda, loop, dtype):
    cfg = hc.config([hc.recurrence(ff=40), hc.attention(ff=30), hc.recurrence()], loop=loop)
    check(be, cfg, 40, dtype, [[40], [3, 20, 1]])


def test_stream_after_every_run(be, cuda):
    cfg = hc.mixed()
    w, toks = hc.weights(cfg, 5), hc.tokens(cfg, 50, 5)
    _, ref = hybrid_ref.HybridOracle(cfg, hc.as_numpy(w)).forward(toks)
    for dtype in DTYPES:
        m = build(be, cfg, w, dtype)
        m.dump = torch.zeros(len(ref), 50, cfg["width"], device=cuda)
        m(torch.tensor(toks), m.make_cache(64))
        for i, r in enumerate(ref):
            d = m.dump[i].double().cpu().numpy() - r
            assert np.abs(d).max() < 2 * TOL[dtype] * np.abs(r).max(), (dtype, i)


# ---------------------------------------------------------------------- portions, decoding, requests
@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_and_decoding(be, cuda, dtype):
    check(be, hc.mixed(), 200, dtype, [[200], [1], [2], [64, 48, 3, 37], [17], [130, 1, 1, 1, 2, 60]], seed=2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_longer_than_a_pass(be, cuda, dtype):
    check(be, hc.mixed(), 600, dtype, [[600], [300, 300]], seed=3)


def test_long_decoding(be, cuda):
    """Hundreds of single tokens after a short prompt: windows pass, states carry."""
    check(be, hc.mixed(), 420, "float32", [[5, 1]], seed=4)


def test_portions_do_not_change_the_result_beyond_rounding(be, cuda):
    cfg = hc.mixed()
    w, toks = hc.weights(cfg, 6), hc.tokens(cfg, 100, 6)
    m = build(be, cfg, w, "float32")
    a = feed(m, toks)
    for cuts in ([1], [2], [33, 3]):
        assert errors(feed(m, toks, cuts), a).max() < 5e-6


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_do_not_touch_each_other(be, cuda, dtype):
    """Unequal requests advanced in turn, caches given back and used again: bit for bit what each gives alone."""
    cfg = hc.mixed()
    m = build(be, cfg, hc.weights(cfg, 7), dtype)
    reqs = {r: hc.tokens(cfg, n, 70 + i) for i, (r, n) in enumerate(dict(a=90, b=33, c=57, d=90).items())}
    cuts = dict(a=[40, 1, 1, 20, 3, 25], b=[2, 30, 1], c=[17, 16, 24], d=[89, 1])

    def alone(r):
        return feed(m, reqs[r], cuts[r])

    rep = be.trace.Replay(m, 128)
    got, at = {r: [] for r in reqs}, dict.fromkeys(reqs, 0)
    order = ["a", "b", "a", "b", "a", "b!", "c", "a", "d", "c", "a", "c!", "a!", "d!"]
    left = {r: list(c) for r, c in cuts.items()}
    for s, name in enumerate(order):
        r = name.rstrip("!")
        n = left[r].pop(0)
        out = rep.step(dict(step=s, entries=[dict(id=r, tokens=reqs[r][at[r]:at[r] + n].tolist(), want=list(range(n)))],
                            end=[r] if name.endswith("!") else []))
        got[r].append(out)
        at[r] += n
    assert not rep.live and len(rep.free) == 3
    for r in reqs:
        assert at[r] == len(reqs[r])
        assert np.array_equal(torch.cat(got[r]).double().numpy(), alone(r)), r


def test_wanted_places(be, cuda):
    cfg = hc.mixed()
    m = build(be, cfg, hc.weights(cfg, 8), "float32")
    toks = hc.tokens(cfg, 300, 8)
    full = feed(m, toks)
    t = torch.tensor(toks)
    for want in ([299], [0, 1, 2], [7, 3, 290, 40], list(range(300))):
        got = m(t, m.make_cache(300), want=want)[0].double().cpu().numpy()
        assert errors(got, full[want]).max() < 1e-6
    c = m.make_cache(300)
    assert m(t, c, want=[]) is None and c.offset == 300
    assert m(t, m.make_cache(300), logits_last_only=True).shape == (1, 1, cfg["vocab"])
    with pytest.raises(be._lib.B200Error):
        m(t[:1], c)                                          # full


# ---------------------------------------------------------------------- keys just inside and just outside
EDGE = hc.config([hc.attention(heads=2, kv_heads=1, dim=32, vdim=32, size=70, keep_first=5)], width=96, taps=2)
FAR = hc.config([hc.attention(heads=2, kv_heads=2, dim=32, vdim=48, size=100000, keep_first=0)], width=96, taps=2)


def planted(cfg, ask_at, answer_at, n, seed=0):
    w, toks = hc.weights(cfg, seed), hc.tokens(cfg, n, seed)
    ask, ans = 3, 11
    hc.plant_pair(cfg, w, 0, ask, ans)
    toks[(toks == ask) | (toks == ans)] = 20
    toks[ask_at], toks[answer_at] = ask, ans
    return w, toks


def edge_cases():
    for ask in (100, 127, 128, 150, 191):
        for dist in (68, 69, 70, 71):                        # the window's edge: 69 is the last one seen
            yield ask, ask - dist
        for j in (0, 3, 4, 5, 6, 63, 64, 65):                # kept first keys, block borders
            if j < ask:
                yield ask, j


@pytest.mark.parametrize("dtype", DTYPES)
def test_window_edges_and_kept_keys(be, cuda, dtype):
    shown = 0
    for ask, ans in edge_cases():
        w, toks = planted(EDGE, ask, ans, 192)
        ref, _ = hybrid_ref.HybridOracle(EDGE, hc.as_numpy(w)).forward(toks)
        m = build(be, EDGE, w, dtype)
        for cuts in ([192], [ask, 1, 191], [64, 1]):
            agree(feed(m, toks, cuts), ref, dtype)
        # the case has teeth: one key more or less in the window or among the kept ones shows, where it is at the edge
        edge = {ask - 70: (71, 5), ask - 69: (69, 5), 5: (70, 6), 4: (70, 4)}.get(ans)
        if edge and not (ans in (4, 5) and ask - ans <= 70):
            wrong = copy.deepcopy(EDGE)
            wrong["layers"][0]["mixer"]["mask"] = dict(size=edge[0], keep_first=edge[1])
            bad, _ = hybrid_ref.HybridOracle(wrong, hc.as_numpy(w)).forward(toks)
            assert errors(bad, ref)[ask] > 5 * TOL[dtype], (ask, ans)
            shown += 1
    assert shown >= 15


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys(be, cuda, dtype):
    for ask, ans in ((699, 0), (699, 63), (640, 64), (576, 1), (500, 255), (321, 256)):
        w, toks = planted(FAR, ask, ans, 700, seed=1)
        ref, _ = hybrid_ref.HybridOracle(FAR, hc.as_numpy(w)).forward(toks)
        m = build(be, FAR, w, dtype)
        for cuts in ([700], [ask, 1, 64]):
            agree(feed(m, toks, cuts), ref, dtype)
        other = toks.copy()
        other[ans] = 20
        bad, _ = hybrid_ref.HybridOracle(FAR, hc.as_numpy(w)).forward(other)
        assert errors(bad, ref)[ask] > 5 * TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_reaches_far_back(be, cuda, dtype):
    """Gates near one: a token hundreds of positions back still decides the output."""
    cfg = hc.config([hc.recurrence(heads=1, dim=16, vdim=24)], taps=2, width=64)
    w = hc.weights(cfg, 9)
    w["l0.mix.f"].zero_()
    w["l0.mix.f.b"].fill_(9.0)
    toks = hc.tokens(cfg, 400, 9)
    other = toks.copy()
    other[0] = (toks[0] + 1) % cfg["vocab"]
    ref, _ = hybrid_ref.HybridOracle(cfg, hc.as_numpy(w)).forward(toks)
    bad, _ = hybrid_ref.HybridOracle(cfg, hc.as_numpy(w)).forward(other)
    assert errors(bad, ref)[399] > 20 * TOL["float32"]
    m = build(be, cfg, w, dtype)
    for cuts in ([400], [100, 1], [2]):
        agree(feed(m, toks, cuts), ref, dtype)


# ---------------------------------------------------------------------- generation through the decoding loop
def greedy(cfg, w, prompt, n):
    orc, toks = hybrid_ref.HybridOracle(cfg, hc.as_numpy(w)), list(prompt)
    margins = []
    for _ in range(n):
        l = orc.forward(np.array(toks))[0][-1]
        top = np.sort(l)[-2:]
        margins.append(top[1] - top[0])
        toks.append(int(l.argmax()))
    assert min(margins) > 1e-3                               # no near-ties in the chosen seeds
    return toks[len(prompt):]


GEN = hc.mixed(vocab=256, width=96)


def generate(be, base, draft, prompt, n, **kw):
    kw = dict(dict(depth=3, verify_num_tokens=15, max_tokens=n - 1, N=n, verbose=False, clip=True), **kw)
    return be.generate_step(torch.tensor(prompt), base, draft, **kw)


def test_greedy_generation_without_a_draft(be, cuda):
    w, prompt = hc.weights(GEN, 10), hc.tokens(GEN, 37, 10)
    ref = greedy(GEN, w, prompt, 30)
    m = build(be, GEN, w, "float32")
    for graph in (False, True):
        r = generate(be, m, None, prompt, 30, use_graph=graph)
        assert r["tokens"] == ref and set(r["accept_lengths"]) == {0}
    r = generate(be, m, None, prompt, 30, eos_token_id=ref[12])
    assert r["tokens"] == ref[:ref.index(ref[12]) + 1] and r["finish_reason"] == "eos"
    # decoding graphs replayed on the bf16 model: the same tokens as its own passes give
    mb = build(be, GEN, w, "bfloat16")
    got = generate(be, mb, None, prompt, 30)["tokens"]
    c, toks = mb.make_cache(128), list(prompt)
    nxt = int(mb(torch.tensor(prompt), c)[0, -1].argmax())
    own = [nxt]
    for _ in range(29):
        nxt = int(mb(torch.tensor([nxt]), c)[0, -1].argmax())
        own.append(nxt)
    assert got == own


@pytest.mark.parametrize("depth,verify", [(0, 7), (3, 15), (5, 31)])
def test_tree_speculation_gives_the_greedy_tokens(be, cuda, depth, verify):
    """The design as target and as draft: states advance over accepted nodes only, whatever the draft is worth."""
    w, prompt = hc.weights(GEN, 10), hc.tokens(GEN, 37, 10)
    ref = greedy(GEN, w, prompt, 30)
    base = build(be, GEN, w, "float32")
    good = build(be, GEN, w, "float32")
    noisy = {k: (v.float() * (1 + 0.15 * torch.randn(v.shape, generator=torch.Generator().manual_seed(1)))).bfloat16() for k, v in w.items()}
    some = build(be, GEN, noisy, "float32")
    none = build(be, GEN, hc.weights(GEN, 11), "bfloat16")
    means = []
    for draft in (good, some, none):
        r = generate(be, base, draft, prompt, 30, depth=depth, verify_num_tokens=verify)
        assert r["tokens"] == ref, (depth, verify)
        means.append(sum(r["accept_lengths"]) / len(r["accept_lengths"]))
    assert means[0] >= min(depth, 3) * 0.6 and means[0] >= means[1] >= means[2]


def test_speculation_with_a_four_bit_model(be, cuda):
    """Pairs of a 4-bit model and the design, either way round."""
    args = be.shape_preset("tiny-qwen2")
    q = be.Model.random_init(args, seed=11, device=cuda, gen_device="cpu").relayout()
    q.norm.mul_(8.0)
    cfg = hc.mixed(vocab=args.vocab_size, width=96)
    w, prompt = hc.weights(cfg, 12), hc.tokens(cfg, 20, 12)
    h = build(be, cfg, w, "float32")
    ref = greedy(cfg, w, prompt, 12)
    assert generate(be, h, q, prompt, 12)["tokens"] == ref
    plain = generate(be, q, None, prompt, 12)["tokens"]
    assert generate(be, q, h, prompt, 12)["tokens"] == plain
    q2 = be.Model.random_init(args, seed=12, device=cuda, gen_device="cpu").relayout()
    assert generate(be, q, q2, prompt, 12)["tokens"] == plain


def test_sampling(be, cuda):
    w, prompt = hc.weights(GEN, 10), hc.tokens(GEN, 37, 10)
    m, d = build(be, GEN, w, "float32"), build(be, GEN, w, "float32")
    ref = greedy(GEN, w, prompt, 20)
    for draft in (None, d):
        assert generate(be, m, draft, prompt, 20, temperature=1e-3)["tokens"] == ref
        a = generate(be, m, draft, prompt, 20, temperature=1.5, seed=5)["tokens"]
        assert a == generate(be, m, draft, prompt, 20, temperature=1.5, seed=5)["tokens"]
        assert a != generate(be, m, draft, prompt, 20, temperature=1.5, seed=6)["tokens"]
        assert a != ref and all(0 <= t < GEN["vocab"] for t in a)


def test_tree_pass_and_accept(be, cuda):
    """tree_decoding / accept_candidate: a branching tree's logits are those of its paths, the accepted path is kept."""
    w, toks = hc.weights(GEN, 13), hc.tokens(GEN, 60, 13)
    orc = hybrid_ref.HybridOracle(GEN, hc.as_numpy(w))
    m = build(be, GEN, w, "float32")
    c = m.make_cache(128)
    m(torch.tensor(toks[:40]), c)
    parent = [-1, 0, 0, 1, 1, 2, 3, 6, 7, 5]
    node = hc.tokens(GEN, len(parent), 14)
    paths = []
    for i, p in enumerate(parent):
        paths.append((paths[p] if p >= 0 else []) + [i])
    T = len(parent)
    mask = torch.zeros(T, T, dtype=torch.bool)
    for i, p in enumerate(paths):
        mask[i, p] = True
    pos = torch.tensor([len(p) - 1 for p in paths])
    for keep in ([1, 3, 6, 7, 8], [2, 5, 9], []):
        c.reset()
        m(torch.tensor(toks[:40]), c)
        got = be.eagle.tree_decoding(torch.tensor(node), mask, pos, m, c)[0].double().cpu().numpy()
        for i, p in enumerate(paths):
            ref = orc.forward(np.concatenate([toks[:40], node[p]]))[0]
            assert errors(got[i:i + 1], ref[-1:]).max() < TOL["float32"], i
        be.eagle.accept_candidate(c, torch.tensor(keep), len(keep), 40)
        assert c.offset == 41 + len(keep)
        tail = m(torch.tensor(toks[40:60]), c)[0].double().cpu().numpy()
        ref = orc.forward(np.concatenate([toks[:40], node[[0] + keep], toks[40:60]]))[0][-20:]
        assert errors(tail, ref).max() < TOL["float32"], keep


# ---------------------------------------------------------------------- files, runner, command line
def write_checkpoint(be, path, cfg, w):
    path.mkdir()
    be.load.write_safetensors(str(path / "model.safetensors"), w)
    (path / "config.json").write_text(json.dumps(cfg))


def test_checkpoint_runner_and_command_line(be, cuda, tmp_path, capsys):
    cfg = GEN
    w, toks = hc.weights(cfg, 15), hc.tokens(cfg, 70, 15)
    write_checkpoint(be, tmp_path / "m", cfg, w)
    ref, _ = hybrid_ref.HybridOracle(cfg, hc.as_numpy(w)).forward(toks)
    steps = [dict(step=0, entries=[dict(id="x", tokens=toks[:50].tolist(), want=[49, 3])], end=[]),
             dict(step=1, entries=[dict(id="x", tokens=toks[50:52].tolist(), want=[])], end=[]),
             dict(step=2, entries=[dict(id="x", tokens=toks[52:70].tolist(), want=[0, 17])], end=["x"]),
             dict(step=3, entries=[dict(id="y", tokens=toks[:1].tolist(), want=[0])], end=["y"])]
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out",
                            str(out), "--max-tokens", "70"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True,
                           timeout=600)
        assert p.returncode == 0, p.stderr
        assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
        for s, rows in ((0, [49, 3]), (2, [52, 69]), (3, [0])):
            got = np.fromfile(out / f"{s}.f32", "<f4").reshape(len(rows), -1)
            assert errors(got, ref[rows]).max() < TOL[dtype]
        assert not (out / "1.f32").exists()
    be.eagle.main(["--base-model", str(tmp_path / "m"), "--draft-model", "none", "--prompt", ",".join(map(str, toks[:9])), "--max-tokens",
                   "6", "-N", "8", "--dtype", "float32"])
    assert "Generated Tokens 6" in capsys.readouterr().out
    be.eagle.main(["--base-model", "tiny-zaverax", "--draft-model", "tiny-zaverax", "--prompt", "12", "--max-tokens", "6", "-N", "8"])
    assert "Mean Tokens Per Step" in capsys.readouterr().out


def test_several_requests_per_pass_are_refused(be, cuda):
    m = build(be, GEN, hc.weights(GEN, 10), "float32")
    with pytest.raises(be._lib.B200Error):
        be.BatchSpecDecoder(m, m, 1, 7, 128, 2)
