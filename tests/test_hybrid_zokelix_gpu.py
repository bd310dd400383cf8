"""The Zokelix design (delta rules with a decay per key channel, latent attention, expert feed-forwards, norms on the sublayers'
outputs) on the GPU against the plain restatement."""
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
from test_hybrid_gpu import DTYPES, TOL, agree, build, check, errors, feed, generate, greedy, write_checkpoint

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CUTS = [[150], [1], [2], [64, 2, 17, 33, 3, 1]]


def oracle(cfg, w, toks):
    return hybrid_ref.HybridOracle(cfg, hc.as_numpy(w)).forward(toks)


# Several layers of random weights with norms on their outputs amplify the rounding of bf16 activations: rounding the sublayers'
# inputs and intermediate vectors in the restatement gives errors up to 0.064 (mean 0.018) on the mixed configurations below.
MIXED = {"float32": (TOL["float32"], TOL["float32"]), "bfloat16": (0.12, 0.025)}


def agree_mixed(got, ref, dtype):
    e = errors(got, ref)
    assert e.max() < MIXED[dtype][0] and e.mean() < MIXED[dtype][1], f"position {e.argmax()}: {e.max():.2e}, mean {e.mean():.2e}"


def check_mixed(be, cfg, n, dtype, cuts, seed):
    w, toks = hc.weights(cfg, seed), hc.tokens(cfg, n, seed)
    ref, _ = oracle(cfg, w, toks)
    for c in cuts:
        agree_mixed(feed(build(be, cfg, w, dtype), toks, c), ref, dtype)


# ---------------------------------------------------------------------- one mechanism at a time
DELTA = {
    "plain": dict(),
    "own_keys": dict(heads=3, kv_heads=3, dim=16, vdim=16),
    "one_key_head": dict(heads=5, kv_heads=1, dim=12, vdim=40),
    "odd": dict(heads=2, kv_heads=1, dim=7, vdim=35, conv=2),
    "one_tap": dict(conv=1),
    "eight_taps": dict(conv=8),
    "tall": dict(heads=2, kv_heads=2, dim=100, vdim=36, conv=4),
    "wide": dict(heads=1, kv_heads=1, dim=24, vdim=132, conv=4),
    "tallest": dict(heads=1, kv_heads=1, dim=200, vdim=72),
    "square": dict(heads=2, kv_heads=1, dim=128, vdim=128, conv=4),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(DELTA))
def test_delta_alone(be, cuda, name, dtype):
    check(be, hc.zokelix([hc.delta(**DELTA[name])]), 150, dtype, CUTS)


@pytest.mark.parametrize("ranks", [(1, 1), (40, 3), (64, 64), (70, 130)])
def test_delta_ranks_come_from_the_tensors(be, cuda, ranks):
    cfg = hc.zokelix([hc.delta()])
    w = hc.zokelix_weights(cfg, 1, ranks)
    for dtype in DTYPES:
        check(be, cfg, 60, dtype, [[60], [1]], w=w)


@pytest.mark.parametrize("dtype", DTYPES)
def test_decays_of_every_size(be, cuda, dtype):
    """Channels that keep everything, lose everything at once, and all between."""
    cfg = hc.zokelix([hc.delta(heads=2, kv_heads=1, dim=32, vdim=20)])
    w = hc.weights(cfg, 4)
    w["l0.mix.dt_bias"] = torch.linspace(-25.0, 25.0, 64).bfloat16()
    w["l0.mix.A_log"] = torch.tensor([-2.0, 1.5]).bfloat16()
    check(be, cfg, 120, dtype, [[120], [1], [19, 40, 3]], w=w)


def test_decays_next_to_one_keep_their_precision(be, cuda):
    """Hundreds of tokens at decays of 1 - 1e-5: a decay rounded to fp32 would be off by up to 3e-8 every time."""
    cfg = hc.zokelix([hc.delta(heads=2, kv_heads=2, dim=16, vdim=16)])
    w, toks = hc.weights(cfg, 5), hc.tokens(cfg, 700, 5)
    for n in ("a1", "a2"):
        w[f"l0.mix.{n}"].zero_()
    w["l0.mix.dt_bias"].fill_(-11.5)
    w["l0.mix.b"][:, :] = 0
    ref, _ = oracle(cfg, w, toks)
    for cuts in ([700], [3, 1]):
        assert errors(feed(build(be, cfg, w, "float32"), toks, cuts), ref).max() < 4e-6


LATENT = {
    "plain": dict(),
    "unscaled": dict(scaling=None),
    "one_head": dict(heads=1, dim=8, rot_dim=2, vdim=50, kv_rank=16),
    "many_heads": dict(heads=21, dim=8, rot_dim=4, vdim=12, kv_rank=20),
    "wide_rotation": dict(dim=16, rot_dim=48, vdim=32, kv_rank=64, base=300.0),
    "all_slow": dict(scaling=dict(factor=3.0, original=4096, fast=0.02, slow=0.01)),
    "all_fast": dict(scaling=dict(factor=3.0, original=8, fast=64.0, slow=32.0)),
    "real_sizes": dict(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=512),
    "past_the_prompt_kernel": dict(heads=2, dim=250, rot_dim=20, vdim=136, kv_rank=72),
    "sharp": dict(scale=1.1),
    "wide_latent": dict(heads=9, dim=20, rot_dim=14, vdim=30, kv_rank=600),
    "middle_rank": dict(heads=6, dim=20, rot_dim=18, vdim=70, kv_rank=200),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(LATENT))
def test_latent_alone(be, cuda, name, dtype):
    check(be, hc.zokelix([hc.latent(**LATENT[name])]), 150, dtype, CUTS)


def test_rotation_matters_and_is_relative(be, cuda):
    """Scores through the rotated part alone: turning it off shows."""
    cfg = hc.zokelix([hc.latent(heads=2, rot_dim=16, scaling=None, scale=1.0)])
    w, toks = hc.weights(cfg, 2), hc.tokens(cfg, 120, 2)
    w["l0.mix.uk"].zero_()
    ref, _ = oracle(cfg, w, toks)
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["rot"]["base"] = 1e30
    assert errors(oracle(other, w, toks)[0], ref)[-60:].mean() > 5 * TOL["bfloat16"]
    for dtype in DTYPES:
        for cuts in CUTS:
            agree(feed(build(be, cfg, w, dtype), toks, cuts), ref, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [3, 72, 600])
def test_gated_feed_forward(be, cuda, ff, dtype):
    cfg = hc.zokelix([hc.delta(mlp=hc.dense(ff))])
    w = hc.weights(cfg, ff)
    w["l0.norm1"].zero_()                                   # the mixer contributes nothing
    check(be, cfg, 40, dtype, [[40], [1]], w=w)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp", [hc.moe(), hc.moe(1, 1, 30), hc.moe(2, 2, 9), hc.moe(16, 1, 33), hc.moe(40, 6, 65, 0.3), hc.moe(35, 10, 20, 100.0),
                                 hc.moe(3, 1, 300, 0.7), hc.moe(3, 2, 50)], ids=lambda m: "{experts}of{top}".format(**m["router"]))
def test_experts(be, cuda, mlp, dtype):
    cfg = hc.zokelix([hc.delta(mlp=mlp)], width=120)
    w = hc.weights(cfg, mlp["expert"]["ff"])
    w["l0.norm1"].zero_()
    check(be, cfg, 190, dtype, [[190], [1], [5, 40, 9, 2]], w=w)


def test_unequal_load_of_the_experts(be, cuda):
    """All tokens to one expert, whose token tiles are many; then none to most."""
    cfg = hc.zokelix([hc.delta(mlp=hc.moe(9, 2, 40))])
    w, toks = hc.weights(cfg, 3), np.full(200, 5)
    w["l0.norm1"].zero_()
    for dtype in DTYPES:
        check(be, cfg, 200, dtype, [[200], [130, 70]], w=w, toks=toks)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", [dict(eps=0.3), dict(width=64, vocab=128), dict(width=201, vocab=77), dict(width=320, vocab=1)])
def test_constants(be, cuda, kw, dtype):
    check(be, hc.zokelix([hc.delta(mlp=hc.moe()), hc.latent(mlp=hc.dense())], **kw), 40, dtype, [[40], [7, 1]])


@pytest.mark.parametrize("dtype", DTYPES)
def test_orders_of_layers(be, cuda, dtype):
    parts = [hc.latent(mlp=hc.moe()), hc.latent(), hc.delta(), hc.delta(mlp=hc.dense())]
    for order in ([0], [1, 0, 2], [3, 3, 1], [2, 1, 2, 0]):
        check(be, hc.zokelix([copy.deepcopy(parts[i]) for i in order]), 50, dtype, [[50], [3, 40, 1]], seed=order[0])


def test_stream_after_every_layer(be, cuda):
    cfg = hc.zokelix_mixed()
    w, toks = hc.weights(cfg, 5), hc.tokens(cfg, 50, 5)
    _, ref = oracle(cfg, w, toks)
    for dtype in DTYPES:
        m = build(be, cfg, w, dtype)
        m.dump = torch.zeros(len(ref), 50, cfg["width"], device=cuda)
        m(torch.tensor(toks), m.make_cache(64))
        for i, r in enumerate(ref):
            d = m.dump[i].double().cpu().numpy() - r
            assert np.abs(d).max() < 2 * TOL[dtype] * np.abs(r).max(), (dtype, i)


def test_mechanisms_in_the_other_norm_order(be, cuda):
    """The mixers and feed-forwards under normed inputs, convolution, residual factor and a repeated range."""
    name = "NormedInputs"
    H = be.hybrid
    z = H.DESIGNS["Zaverax"]
    H.DESIGNS[name] = H.Design(dict(dense=H.GatedFF, moe=H.ExpertsFF), norm_offset=z.norm_offset, input_conv=True)
    hybrid_ref.FEED_FORWARDS[name] = hybrid_ref.FEED_FORWARDS["Zokelix"]
    try:
        cfg = hc.zokelix([hc.delta(mlp=hc.dense(40)), hc.latent(mlp=hc.moe(3, 2, 20)), hc.delta()])
        w = hc.weights(cfg, 6)
        cfg.update(architecture=name, canon=dict(taps=3), residual_mult=0.6, loop=dict(start=1, stop=2, times=2), logit_softcap=9.0)
        g = torch.Generator().manual_seed(1)
        for i in range(3):
            w[f"l{i}.canon1"] = (0.3 * torch.randn(cfg["width"], 3, generator=g)).bfloat16()
        w["l1.mlp.router"].zero_()
        w["l1.mlp.router"][:, 50] = torch.tensor([0.5, -0.5, 0.0])         # (all experts but one are clear by the sign of a channel)
        toks = hc.tokens(cfg, 60, 6)
        ref, _ = oracle(cfg, w, toks)
        agree(feed(build(be, cfg, w, "float32"), toks), ref, "float32")
        agree(feed(build(be, cfg, w, "float32"), toks, [7, 2, 1]), ref, "float32")
    finally:
        del H.DESIGNS[name], hybrid_ref.FEED_FORWARDS[name]


# ---------------------------------------------------------------------- portions, decoding, requests
@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_and_decoding(be, cuda, dtype):
    check_mixed(be, hc.zokelix_mixed(), 200, dtype, [[200], [1], [2], [64, 48, 3, 37], [17], [31, 33, 32], [130, 1, 1, 1, 2, 60]], seed=2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_longer_than_a_pass(be, cuda, dtype):
    check_mixed(be, hc.zokelix_mixed(), 600, dtype, [[600], [300, 300], [257, 2]], seed=3)


def test_long_decoding(be, cuda):
    check(be, hc.zokelix_mixed(), 420, "float32", [[5, 1]], seed=4)


@pytest.mark.parametrize("dtype,bound", [("float32", 1e-5), ("bfloat16", 0.08)])
def test_portions_do_not_change_the_result_beyond_rounding(be, cuda, dtype, bound):
    cfg = hc.zokelix_mixed()
    w, toks = hc.weights(cfg, 6), hc.tokens(cfg, 100, 6)
    m = build(be, cfg, w, dtype)
    a = feed(m, toks)
    for cuts in ([1], [2], [33, 3]):
        assert errors(feed(m, toks, cuts), a).max() < bound


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_do_not_touch_each_other(be, cuda, dtype):
    """Unequal requests advanced in turn, caches given back and used again, a cache of other size between: bit for bit what
    each gives alone."""
    cfg = hc.zokelix_mixed()
    m = build(be, cfg, hc.weights(cfg, 7), dtype)
    reqs = {r: hc.tokens(cfg, n, 70 + i) for i, (r, n) in enumerate(dict(a=90, b=33, c=57, d=90).items())}
    cuts = dict(a=[40, 1, 1, 20, 3, 25], b=[2, 30, 1], c=[17, 16, 24], d=[89, 1])
    alone = {r: feed(build(be, cfg, hc.weights(cfg, 7), dtype), reqs[r], cuts[r]) for r in reqs}
    rep = be.trace.Replay(m, 128)
    got, at, left = {r: [] for r in reqs}, dict.fromkeys(reqs, 0), {r: list(c) for r, c in cuts.items()}
    for s, name in enumerate(["a", "b", "a", "b", "a", "b!", "c", "a", "d", "c", "a", "c!", "a!", "d!"]):
        r = name.rstrip("!")
        n = left[r].pop(0)
        out = rep.step(dict(step=s, entries=[dict(id=r, tokens=reqs[r][at[r]:at[r] + n].tolist(), want=list(range(n)))],
                            end=[r] if name.endswith("!") else []))
        got[r].append(out)
        at[r] += n
        if s == 6:
            feed(m, reqs["d"], [70, 20], m.make_cache(300))
    assert not rep.live and len(rep.free) == 3
    for r in reqs:
        assert at[r] == len(reqs[r])
        assert np.array_equal(torch.cat(got[r]).double().numpy(), alone[r]), r


def test_caches_start_empty_again(be, cuda):
    """A reset cache gives what a new one gives: states and convolution inputs are cleared, old rows not seen."""
    cfg = hc.zokelix_mixed()
    m = build(be, cfg, hc.weights(cfg, 8), "float32")
    toks, c = hc.tokens(cfg, 80, 8), m.make_cache(96)
    first = feed(m, toks[:30], [7, 1], c)
    c.reset()
    feed(m, toks[30:], [50], c)
    c.reset()
    assert np.array_equal(feed(m, toks[:30], [7, 1], c), first)


def test_wanted_places(be, cuda):
    cfg = hc.zokelix_mixed()
    m = build(be, cfg, hc.weights(cfg, 8), "float32")
    toks = hc.tokens(cfg, 300, 8)
    full, t = feed(m, toks), torch.tensor(toks)
    for want in ([299], [0, 1, 2], [7, 3, 290, 40], list(range(300))):
        assert errors(m(t, m.make_cache(300), want=want)[0].double().cpu().numpy(), full[want]).max() < 1e-6
    assert m(t, m.make_cache(300), want=[]) is None


# ---------------------------------------------------------------------- far back, block borders, first tokens
PLACES = [(299, 0), (299, 1), (299, 63), (256, 64), (255, 127), (257, 128), (200, 199), (64, 63), (65, 0), (3, 2), (1, 0), (270, 255), (270, 256)]


def far_case(plant, cfg, seed, ask_at, answer_at, n=300):
    w, toks = hc.weights(cfg, seed), hc.tokens(cfg, n, seed)
    ask, ans = 3, 11
    plant(cfg, w, 0, ask, ans)
    toks[(toks == ask) | (toks == ans)] = 20
    toks[ask_at], toks[answer_at] = ask, ans
    other = toks.copy()
    other[answer_at] = 20
    ref, bad = oracle(cfg, w, toks)[0], oracle(cfg, w, other)[0]
    assert errors(bad, ref)[ask_at] > 5 * TOL["bfloat16"], (ask_at, answer_at)       # the case has teeth
    return w, toks, ref


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_of_latent_attention(be, cuda, dtype):
    cfg = hc.zokelix([hc.latent(heads=2, dim=32, vdim=48, kv_rank=56)])
    for ask, ans in PLACES:
        w, toks, ref = far_case(hc.plant_latent_pair, cfg, 1, ask, ans)
        m = build(be, cfg, w, dtype)
        for cuts in ([300], [ask, 1, 64], [ans + 1, 2, 70]):
            agree(feed(m, toks, cuts), ref, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_state_reaches_far_back(be, cuda, dtype):
    cfg = hc.zokelix([hc.delta(heads=2, kv_heads=1, dim=16, vdim=24)])
    for ask, ans in PLACES:
        w, toks, ref = far_case(hc.plant_delta_pair, cfg, 2, ask, ans)
        m = build(be, cfg, w, dtype)
        for cuts in ([300], [ask, 1, 64], [ans + 1, 2, 70]):
            agree(feed(m, toks, cuts), ref, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_convolutions_over_portion_borders(be, cuda, dtype):
    """One tap alone, the farthest: every output rests on the token taps - 1 positions back, from whatever portion."""
    for taps in (2, 4, 8):
        cfg = hc.zokelix([hc.delta(conv=taps)])
        w = hc.weights(cfg, taps)
        for n in ("q", "k", "v"):
            w[f"l0.mix.{n}.conv"][:, 1:] *= 0.05
            w[f"l0.mix.{n}.conv"][:, 0] += 1.0
        check(be, cfg, 70, dtype, [[70], [1], [2], [taps - 1, 1], [taps, 2, 33]], w=w)


# ---------------------------------------------------------------------- generation through the decoding loop
GEN = hc.zokelix_mixed(vocab=256, width=96)


def test_greedy_generation_without_a_draft(be, cuda):
    w, prompt = hc.weights(GEN, 10), hc.tokens(GEN, 37, 10)
    ref = greedy(GEN, w, prompt, 30)
    m = build(be, GEN, w, "float32")
    for graph in (False, True):
        r = generate(be, m, None, prompt, 30, use_graph=graph)
        assert r["tokens"] == ref and set(r["accept_lengths"]) == {0}
    mb = build(be, GEN, w, "bfloat16")
    got = generate(be, mb, None, prompt, 30)["tokens"]
    c, nxt, own = mb.make_cache(128), None, []
    for i in range(30):
        nxt = int(mb(torch.tensor(prompt if i == 0 else [nxt]), c)[0, -1].argmax())
        own.append(nxt)
    assert got == own


@pytest.mark.parametrize("depth,verify", [(0, 7), (3, 15), (5, 31)])
def test_tree_speculation_gives_the_greedy_tokens(be, cuda, depth, verify):
    """The design as target and as draft: states advance over accepted nodes only, whatever the draft is worth."""
    w, prompt = hc.weights(GEN, 10), hc.tokens(GEN, 37, 10)
    ref = greedy(GEN, w, prompt, 30)
    base, good = build(be, GEN, w, "float32"), build(be, GEN, w, "float32")
    none = build(be, GEN, hc.weights(GEN, 11), "bfloat16")
    means = []
    for draft in (good, none):
        r = generate(be, base, draft, prompt, 30, depth=depth, verify_num_tokens=verify)
        assert r["tokens"] == ref, (depth, verify)
        means.append(sum(r["accept_lengths"]) / len(r["accept_lengths"]))
    assert means[0] >= min(depth, 3) * 0.6 and means[0] >= means[1]


def test_speculation_with_other_designs(be, cuda):
    w, prompt = hc.weights(GEN, 10), hc.tokens(GEN, 20, 12)
    base = build(be, GEN, w, "float32")
    zc = hc.mixed(vocab=256, width=96)
    other = build(be, zc, hc.weights(zc, 13), "float32")
    assert generate(be, base, other, prompt, 12)["tokens"] == greedy(GEN, w, prompt, 12)
    assert generate(be, other, base, prompt, 12)["tokens"] == generate(be, other, None, prompt, 12)["tokens"]


def test_sampling(be, cuda):
    w, prompt = hc.weights(GEN, 10), hc.tokens(GEN, 37, 10)
    m, d = build(be, GEN, w, "float32"), build(be, GEN, w, "float32")
    ref = greedy(GEN, w, prompt, 20)
    for draft in (None, d):
        assert generate(be, m, draft, prompt, 20, temperature=1e-3)["tokens"] == ref
        a = generate(be, m, draft, prompt, 20, temperature=1.5, seed=5)["tokens"]
        assert a == generate(be, m, draft, prompt, 20, temperature=1.5, seed=5)["tokens"] and a != ref


def test_tree_pass_and_accept(be, cuda):
    """A branching tree's logits are those of its paths, the accepted path is kept; both forms of the kernels."""
    w, toks = hc.weights(GEN, 13), hc.tokens(GEN, 60, 13)
    orc = hybrid_ref.HybridOracle(GEN, hc.as_numpy(w))
    parent = [-1, 0, 0, 1, 1, 2, 3, 6, 7, 5]
    node = hc.tokens(GEN, len(parent), 14)
    paths = []
    for i, p in enumerate(parent):
        paths.append((paths[p] if p >= 0 else []) + [i])
    mask = torch.zeros(len(parent), len(parent), dtype=torch.bool)
    for i, p in enumerate(paths):
        mask[i, p] = True
    pos = torch.tensor([len(p) - 1 for p in paths])
    for dtype in DTYPES:
        m = build(be, GEN, w, dtype)
        c = m.make_cache(128)
        for keep in ([1, 3, 6, 7, 8], [2, 5, 9], []):
            c.reset()
            m(torch.tensor(toks[:40]), c)
            got = be.eagle.tree_decoding(torch.tensor(node), mask, pos, m, c)[0].double().cpu().numpy()
            for i, p in enumerate(paths):
                ref = orc.forward(np.concatenate([toks[:40], node[p]]))[0]
                assert errors(got[i:i + 1], ref[-1:]).max() < MIXED[dtype][0], i
            be.eagle.accept_candidate(c, torch.tensor(keep), len(keep), 40)
            assert c.offset == 41 + len(keep)
            tail = m(torch.tensor(toks[40:60]), c)[0].double().cpu().numpy()
            ref = orc.forward(np.concatenate([toks[:40], node[[0] + keep], toks[40:60]]))[0][-20:]
            agree_mixed(tail, ref, dtype)


# ---------------------------------------------------------------------- files, runner, command line
def test_checkpoint_runner_and_command_line(be, cuda, tmp_path, capsys):
    w, toks = hc.weights(GEN, 15), hc.tokens(GEN, 70, 15)
    write_checkpoint(be, tmp_path / "m", GEN, w)
    ref, _ = oracle(GEN, w, toks)
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
        for s, rows in ((0, [49, 3]), (2, [52, 69]), (3, [0])):
            got = np.fromfile(out / f"{s}.f32", "<f4").reshape(len(rows), -1)
            assert errors(got, ref[rows]).max() < MIXED[dtype][0]
    be.eagle.main(["--base-model", str(tmp_path / "m"), "--draft-model", "none", "--prompt", ",".join(map(str, toks[:9])), "--max-tokens",
                   "6", "-N", "8", "--dtype", "float32"])
    assert "Generated Tokens 6" in capsys.readouterr().out
    be.eagle.main(["--base-model", "tiny-zokelix", "--draft-model", "tiny-zaverax", "--prompt", "12", "--max-tokens", "6", "-N", "8"])
    assert "Mean Tokens Per Step" in capsys.readouterr().out
