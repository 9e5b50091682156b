"""The Fasulix family on the layer-list runtime against the plain float64 statement in fasulix_plain.py.

Every test makes its own small configuration and seeded weights.  float32 mode is compared tightly (it shows any wrong key, a window
that is one token off, a lost state, a sink left out, a wrong expert or weight); bfloat16 mode within bf16 rounding.  Where random
weights would hide a fault the scores are sharpened (a large score scale, so that single keys dominate the softmax), or one query and
key are made to match."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import fasulix_plain as plain  # noqa: E402

pytestmark = pytest.mark.gpu

from calm_b200 import container, fasulix, registry, seqlib, serving  # noqa: E402


def moe(experts=5, top=2, ff=12, limit=0.9):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def gru(width=20, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def latent(size=0, heads=3, dim=8, rot_dim=4, vdim=6, q_rank=18, kv_rank=24, scale=0.5, base=300.0, kv_from=None, mlp=None):
    """size 0: full attention with a sink; else a sliding window without one"""
    mx = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale, "rot": {"dims": rot_dim, "base": base}}
    if size:
        mx["mask"] = {"size": size}
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return {"type": "latent_attention_2" if size else "latent_attention", "mixer": mx, "mlp": mlp}


def config(layers, width=48, vocab=97, eps=1e-5):
    return {"architecture": "Fasulix", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def weights(cfg, seed=0):
    return fasulix.random_tensors(cfg, seed)


def as_f64(t):
    return {k: v.float().numpy().astype(np.float64) for k, v in t.items()}


def tokens(cfg, n, seed=1):
    return [int(x) for x in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def clear_rows(cfg, t, toks, dtype):
    """Rows that routing coin tosses cannot reach.  In bfloat16 the router's input carries the rounding of everything before it, so a
    logit within a few hundredths of the next one may fall either way; that row then differs by an expert, not by rounding, and so does
    what later rows remember of it.  float32 needs no such care: every row counts."""
    keep = np.ones(len(toks), bool)
    if dtype == "float32":
        return keep
    plain.MARGINS.clear()
    plain.forward(cfg, as_f64(t), toks)
    for m in plain.MARGINS:
        keep &= m > 0.05
    if len(cfg["layers"]) > 1 and plain.MARGINS:
        keep = np.cumprod(keep).astype(bool)
    assert keep.sum() >= min(5, len(toks)), "too few rows with clear routing: choose another seed or a feed-forward without choices"
    return keep


def free_of_choices(dtype, **kw):
    """The feed-forward of tests that run in both modes with several layers: in bfloat16 every expert is taken (nothing to toss)."""
    ml = moe(**kw)
    if dtype != "float32":
        ml["router"]["top"] = ml["router"]["experts"]
    return ml


def rel_err(got, ref, dtype="float32"):
    """Error of the worst row, relative to the spread of the reference logits.  In bfloat16 a few rows sit far above the others without
    any fault (a norm over values that happen to be small multiplies the rounding of what came before): there the measure is the larger
    of the ninth decile and a sixth of the worst row (a row computed from a wrong key or state is off by about one)."""
    d = got - ref
    d = d - d.mean(-1, keepdims=True)
    r = ref - ref.mean(-1, keepdims=True)
    rows = np.sqrt((d * d).mean(-1)) / np.sqrt((r * r).mean())
    if dtype == "float32":
        return float(rows.max())
    return float(max(np.quantile(rows, 0.9), rows.max() / 6))


TOL = {"float32": 3e-5, "bfloat16": 4e-2}
SHOWS = 100 * TOL["float32"]


def whole(model, toks):
    s = model.open()
    out = model.step([s], [toks], list(range(len(toks))))
    model.close_seq(s)
    return out


def in_portions(model, toks, sizes):
    """the tokens cut into portions of the given sizes (the last size repeats), all rows"""
    s, rows, at, k = model.open(), [], 0, 0
    while at < len(toks):
        part = toks[at:at + sizes[min(k, len(sizes) - 1)]]
        rows.append(model.step([s], [part], list(range(len(part)))))
        at, k = at + len(part), k + 1
    model.close_seq(s)
    return np.concatenate(rows)


def check_all_ways(cfg, t, toks, dtype="float32", portions=(5, 2, 1), page=4):
    """whole prompt, prompt + token-by-token decoding, and portions: all against the plain statement."""
    ref = plain.forward(cfg, as_f64(t), toks)
    clear = clear_rows(cfg, t, toks, dtype)
    err = lambda got: rel_err(got[clear], ref[clear], dtype)  # noqa: E731
    with fasulix.from_tensors(cfg, t, dtype, max_tokens=4 * len(toks) + 64, max_seqs=4, page=page) as m:
        assert err(whole(m, toks)) < TOL[dtype]
        for first in {1, max(1, len(toks) // 2)}:
            assert err(in_portions(m, toks, [first, 1])) < TOL[dtype]
        for size in portions:
            grow = [size + k for k in range(30)] if size > 2 else [size]  # growing portions: edges fall at ever different places
            assert err(in_portions(m, toks, grow)) < TOL[dtype]
    return ref


LAYERS = {
    "recurrence": [gru()],
    "recurrence-of-one-channel": [gru(width=1)],
    "recurrence-wider-than-the-model": [gru(width=150)],
    "full-latent": [latent()],
    "full-latent-one-head-all-ranks-differ": [latent(heads=1, dim=16, rot_dim=2, vdim=10, q_rank=8, kv_rank=40)],
    "full-latent-more-rotated-than-unrotated": [latent(heads=2, dim=4, rot_dim=16, vdim=24, q_rank=32, kv_rank=8)],
    "window": [latent(size=7)],
    "window-of-one": [latent(size=1, heads=2)],
    "window-longer-than-the-prompt": [latent(size=64)],
    "window-shared-latents": [latent(size=7), latent(size=7, kv_from=0)],
    "shared-latents-of-a-full-layer-other-heads-and-window": [latent(heads=2, vdim=9), latent(size=5, heads=5, dim=4, vdim=3, q_rank=11, scale=0.9, kv_from=0)],
    "experts-top1": [gru(mlp=moe(experts=5, top=1))],
    "experts-top2-tight-clamp": [gru(mlp=moe(experts=4, top=2, limit=0.25))],
    "experts-all-loose-clamp": [latent(mlp=moe(experts=3, top=3, ff=20, limit=50.0))],
    "one-expert": [latent(size=6, mlp=moe(experts=1, top=1, ff=8))],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(LAYERS))
def test_each_mechanism_alone(name, dtype):
    cfg = config(LAYERS[name])
    check_all_ways(cfg, weights(cfg, 3), tokens(cfg, 37), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_align_with_nothing(dtype):
    """Width, head sizes, ranks, channel counts, expert widths and vocabulary that are multiples of neither 8 nor 4."""
    cfg = config([latent(heads=3, dim=5, rot_dim=6, vdim=7, q_rank=9, kv_rank=11, mlp=free_of_choices(dtype, experts=3, top=2, ff=9)),
                  gru(width=13, mlp=free_of_choices(dtype, experts=2, top=1, ff=3)),
                  latent(size=9, heads=2, dim=3, rot_dim=2, vdim=5, q_rank=7, kv_rank=15),
                  latent(size=4, heads=1, dim=9, rot_dim=2, vdim=11, q_rank=5, kv_rank=15, kv_from=2, base=300.0)], width=50, vocab=61)
    check_all_ways(cfg, weights(cfg, 31), tokens(cfg, 45), dtype, portions=(17, 2))


def test_wide_latents():
    """A latent beyond what the attention kernel keeps in registers per lane, with values wider than its two columns per thread, and one of
    exactly that width."""
    for rank, rot in ((600, 8), (512, 64)):
        cfg = config([latent(heads=2, dim=16, rot_dim=rot, vdim=8, q_rank=20, kv_rank=rank), latent(size=9, heads=2, dim=8, rot_dim=rot, vdim=8, q_rank=20, kv_rank=rank, kv_from=0)])
        check_all_ways(cfg, weights(cfg, 30), tokens(cfg, 29), portions=(7,))
        check_all_ways(cfg, weights(cfg, 30), tokens(cfg, 29), "bfloat16", portions=(7,))


def test_wide_rows():
    """Rows wider than a thread keeps in registers (more than 4096 columns, and more than 1024 of a width that is no multiple of 4)."""
    for width in (4200, 1234):
        cfg = config([gru(width=9), latent(size=5, heads=2)], width=width, vocab=33)
        check_all_ways(cfg, weights(cfg, 29), tokens(cfg, 11), portions=(3,))


def test_other_layer_orders():
    for k, order in enumerate(([latent(mlp=moe()), gru(), latent(size=5, mlp=moe(top=1)), gru(mlp=moe())], [latent(size=3), latent(), latent(size=8, kv_from=1), gru(), latent(size=2, kv_from=0, mlp=moe(experts=2))],
                               [gru()])):
        cfg = config(order, width=40)
        check_all_ways(cfg, weights(cfg, 5 + k), tokens(cfg, 41), portions=(6,))


def test_residual_stream_after_every_layer():
    cfg = config([gru(mlp=moe()), latent(), latent(size=5, mlp=moe(top=1)), latent(size=6, kv_from=2)])
    t, toks = weights(cfg, 8), tokens(cfg, 19)
    trace = []
    plain.forward(cfg, as_f64(t), toks, trace)
    with fasulix.from_tensors(cfg, t, "float32", max_tokens=64, max_seqs=2) as m:
        m.set_trace(True)
        whole(m, toks)
        got = m.read_trace(len(toks))
    assert got.shape[0] == len(trace) == 4
    for g, r in zip(got, trace):
        assert np.abs(g - r).max() < 1e-4 * max(1.0, np.abs(r).max())


def test_every_mechanism_shows(monkeypatch):
    """The runtime agrees with the plain statement; the plain statement with one mechanism left out or read otherwise (the gate, the depth
    average, the sink, the pairing of rotated channels, the recurrence's 1/2, the experts' + 1, the rotated part of shared latents, a window that is one position off) is far outside the tolerance."""
    cfg = config([gru(mlp=moe()), latent(scale=0.8), latent(size=6, scale=1.2, mlp=moe(top=1)), latent(size=6, scale=1.2, kv_from=2)])
    t, toks = weights(cfg, 11), tokens(cfg, 60)
    t["l1.mix.sink"] += 1.5
    ref = check_all_ways(cfg, t, toks, portions=(7, 2))
    p = as_f64(t)
    for knob, val in (("gate", False), ("depth", False), ("sink", False), ("interleaved", False), ("half", False), ("plus_one", False), ("share_rotated", False),
                      ("window_shift", 1), ("window_shift", -1)):
        monkeypatch.setitem(plain.KNOBS, knob, val)
        assert rel_err(plain.forward(cfg, p, toks), ref) > SHOWS, knob
        monkeypatch.undo()
    for layer, key, val in ((1, "rot", {"dims": 4, "base": 200.0}), (2, "scale", 1.1), (2, "mask", {"size": 7}), (3, "mask", {"size": 5})):
        wrong = copy.deepcopy(cfg)
        wrong["layers"][layer]["mixer"][key] = val
        assert rel_err(plain.forward(wrong, p, toks), ref) > SHOWS, key
    for key, val in (("limit", 0.8),):
        wrong = copy.deepcopy(cfg)
        wrong["layers"][0]["mlp"]["expert"][key] = val
        assert rel_err(plain.forward(wrong, p, toks), ref) > SHOWS
    wrong = copy.deepcopy(cfg)
    wrong["layers"][0]["mlp"]["router"]["top"] = 3
    assert rel_err(plain.forward(wrong, p, toks), ref) > SHOWS


def test_router_weights_are_the_scores_themselves(monkeypatch):
    """The norm behind the feed-forward hides a common factor of its input, all but its eps: a large one shows that the weights are softmax
    scores over all experts, not renormalised over the chosen ones."""
    cfg = config([gru(mlp=moe(experts=6, top=2)), gru(mlp=moe(experts=4, top=1))], eps=0.4)
    t, toks = weights(cfg, 13), tokens(cfg, 40)
    ref = check_all_ways(cfg, t, toks, portions=(9,))
    monkeypatch.setitem(plain.KNOBS, "renormalise", True)
    assert rel_err(plain.forward(cfg, as_f64(t), toks), ref) > SHOWS


@pytest.mark.parametrize("n", [31, 32, 33, 64, 65, 200])
def test_recurrence_over_chunk_edges(n):
    """A prompt's recurrence is cut into chunks of 32 tokens whose maps on the state are folded: lengths around the edges, portions that
    start inside a chunk, unequal portions in one step."""
    cfg = config([gru(width=70), gru(width=3)], width=24, vocab=41)
    t, toks = weights(cfg, 40), tokens(cfg, n)
    t["l0.mix.z.b"] = torch.full_like(t["l0.mix.z.b"], -3.0)  # a state that remembers dozens of tokens
    p = as_f64(t)
    ref = plain.forward(cfg, p, toks)
    for dtype in ("float32", "bfloat16"):
        with fasulix.from_tensors(cfg, t, dtype, max_tokens=3 * n + 64, max_seqs=3) as m:
            assert rel_err(whole(m, toks), ref, dtype) < TOL[dtype]
            assert rel_err(in_portions(m, toks, [n - 1, 1]), ref, dtype) < TOL[dtype]
            assert rel_err(in_portions(m, toks, [20, 40, 2, 34, 1]), ref, dtype) < TOL[dtype]
            a, b = m.open(), m.open()
            out = m.step([a, b], [toks[:-1], toks[:5]], list(range(n + 4)))
            assert rel_err(out[:n - 1], ref[:-1], dtype) < TOL[dtype] and rel_err(out[n - 1:], ref[:5], dtype) < TOL[dtype]
            out = m.step([a, b], [toks[-1:], toks[5:]], list(range(n - 4)))
            assert rel_err(out, np.concatenate([ref[-1:], ref[5:]]), dtype) < TOL[dtype]


def test_recurrence_over_thousands_of_tokens():
    """Beyond 64 chunks the chunks grow instead of their number: a prompt of 4500 tokens as one step, its last tokens decoded."""
    cfg = config([gru(width=6)], width=16, vocab=29)
    t, toks = weights(cfg, 41), tokens(cfg, 4510)
    t["l0.mix.z.b"] = torch.full_like(t["l0.mix.z.b"], -6.0)
    t["l0.mix.z"] = t["l0.mix.z"] * 0.2
    ref = plain.forward(cfg, as_f64(t), toks)
    changed = plain.forward(cfg, as_f64(t), toks[:4000] + [(x + 1) % 29 for x in toks[4000:4100]] + toks[4100:])
    assert rel_err(changed[4490:], ref[4490:]) > SHOWS  # the state does carry over hundreds of tokens
    with fasulix.from_tensors(cfg, t, "float32", max_tokens=4600, max_seqs=1) as m:
        s = m.open()
        want = list(range(0, 4500, 37)) + [4499]
        assert rel_err(m.step([s], [toks[:4500]], want), ref[want]) < TOL["float32"]
        assert rel_err(np.concatenate([m.step([s], [[x]], [0]) for x in toks[4500:]]), ref[4500:]) < TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_context_with_shared_out_keys(dtype):
    """Decoding few tokens over a context of several hundred: the attention kernel shares one query's keys out over several CTAs and folds
    the shares (the sink counts once); positions in the hundreds turn the rotated channels by hundreds of radians; a window of 200 and
    a layer that reads its latents through a narrower one; pages are crossed all along."""
    sharp = 1.5 if dtype == "float32" else 0.5
    cfg = config([latent(heads=4, rot_dim=16, base=50.0, scale=sharp), latent(size=200, scale=sharp), latent(size=130, heads=2, scale=sharp, kv_from=1)])
    t, toks = weights(cfg, 15), tokens(cfg, 330)
    ref = plain.forward(cfg, as_f64(t), toks)
    with fasulix.from_tensors(cfg, t, dtype, max_tokens=700, max_seqs=2, page=16) as m:
        s = m.open()
        rows = [m.step([s], [toks[:300]], list(range(300)))]
        for p in range(300, 330):
            rows.append(m.step([s], [[toks[p]]], [0]))
        assert rel_err(np.concatenate(rows), ref, dtype) < TOL[dtype]
        assert rel_err(in_portions(m, toks, [2]), ref, dtype) < TOL[dtype]  # beside the finished sequence


def matching_key(cfg, t, toks, layer=0, key_tok=5, query_tok=3):
    """Make the queries of `query_tok` match the key of `key_tok` and no other: the unrotated queries and keys read only the first half of
    the embedding columns, which the two tokens share, through the same latent; token key_tok's other half (its value) is the opposite
    of query_tok's (as large, so that the latent's norm leaves the two keys equal)."""
    p = f"l{layer}.mix."
    mx = cfg["layers"][layer]["mixer"]
    H, D, P, R, W = mx["heads"], mx["dim"], mx["rot_dim"], mx["kv_rank"], cfg["width"]
    g = torch.Generator().manual_seed(77)
    code = torch.randn(R, W // 2, generator=g) / (W // 2) ** 0.5
    dkv = torch.zeros(R + P, W)
    dkv[:R // 2, :W // 2] = code[:R // 2]              # half of the latent names the token ...
    dkv[R // 2:R, W // 2:] = torch.randn(R - R // 2, W - W // 2, generator=g) / (W // 2) ** 0.5  # ... the other half is what it says
    t[p + "dkv"] = dkv.bfloat16()
    t[p + "dq"] = torch.zeros(R // 2, W).bfloat16()
    t[p + "dq"][:, :W // 2] = code[:R // 2].bfloat16()
    t[p + "dq.norm"], t[p + "dkv.norm"] = torch.ones(R // 2).bfloat16(), torch.ones(R).bfloat16()
    m = torch.randn(D, R // 2, generator=g) / (R // 2) ** 0.5
    uq, uk = torch.zeros(H, D + P, R // 2), torch.zeros(H, D, R)
    uq[:, :D], uk[:, :, :R // 2] = m, m
    t[p + "uq"], t[p + "uk"] = uq.reshape(H * (D + P), -1).bfloat16(), uk.reshape(H * D, R).bfloat16()
    t[f"l{layer}.norm1"] = torch.ones(W).bfloat16()
    t["embed"][key_tok, :W // 2], t["embed"][key_tok, W // 2:] = t["embed"][query_tok, :W // 2], -t["embed"][query_tok, W // 2:]
    return [key_tok if i == 5 else 4 if x in (key_tok, query_tok) else x for i, x in enumerate(toks)]


FAR = {"heads": 2, "dim": 16, "rot_dim": 2, "vdim": 8, "q_rank": 16, "kv_rank": 32, "scale": 2.0}


@pytest.mark.parametrize("size,shared", [(120, None), (0, None), (120, 0), (120, 7)])
def test_a_far_key_stands_out_inside_the_window_and_not_outside(size, shared):
    """Position 5 holds a key that later queries match far above every other.  The queries sit where the window of 120 (page edges at
    every 16) just still sees it, just no longer, and far away; without a window they find it hundreds of positions back.  Prompt,
    portions and decoding alike; and once more for a layer that reads the latents of another one, whose own window (none, or 7) is
    not the reader's."""
    cfg = config([latent(size=size, **FAR)] if shared is None else [latent(size=shared, **FAR), latent(size=size, kv_from=0, **FAR)])
    t = weights(cfg, 16)
    toks = matching_key(cfg, t, tokens(cfg, 300))
    if shared is not None:  # the layer that makes the latents hands the stream on as it is
        for n in ("dq", "dq.norm", "uq", "uk"):
            t["l1.mix." + n] = t["l0.mix." + n].clone()
        t["l0.norm1b"], t["l1.norm1"] = torch.zeros_like(t["l0.norm1b"]), t["l0.norm1"].clone()
        t["l0.dwa"] = torch.tensor([0.0, 1.0]).bfloat16()
    for x in (124, 125, 299):  # just inside and just outside the window, and far away
        toks[x] = 3
    p = as_f64(t)
    ref = plain.forward(cfg, p, toks)
    gone = list(toks)
    gone[5] = 4  # without the key, rows that see it move, rows that do not see it stay as they are
    diff = plain.forward(cfg, p, gone)
    moved = lambda x: rel_err(diff[x:x + 1], ref[x:x + 1])  # noqa: E731
    assert moved(124) > SHOWS and all(moved(x) < 1e-9 if size else moved(x) > SHOWS for x in (125, 299))
    with fasulix.from_tensors(cfg, t, "float32", max_tokens=1024, max_seqs=2, page=16) as m:
        assert rel_err(whole(m, toks), ref) < TOL["float32"]
        s = m.open()
        rows = [m.step([s], [toks[:120]], list(range(120)))] + [m.step([s], [[x]], [0]) for x in toks[120:130]] + [m.step([s], [toks[130:290]], list(range(160)))]
        rows += [m.step([s], [[x]], [0]) for x in toks[290:]]
        assert rel_err(np.concatenate(rows), ref) < TOL["float32"]
        m.close_seq(s)
        assert rel_err(in_portions(m, toks, [124, 1, 2]), ref) < TOL["float32"]
    with fasulix.from_tensors(cfg, t, "bfloat16", max_tokens=1024, max_seqs=2, page=16) as m:
        for cut in ([300], [124, 1], [110, 20, 2]):
            got = in_portions(m, toks, cut)
            assert rel_err(got, ref, "bfloat16") < TOL["bfloat16"] and rel_err(got[[124, 125, 299]], ref[[124, 125, 299]]) < 2 * TOL["bfloat16"]


def test_the_sink_takes_its_share(monkeypatch):
    """A sink far above every score leaves almost nothing of the values, one far below changes nothing, and it is not scaled: from the
    first token of a sequence on, with few keys and with hundreds."""
    for level, scale in ((6.0, 0.2), (-30.0, 0.2), (1.0, 3.0)):
        cfg = config([latent(scale=scale)])
        t, toks = weights(cfg, 42), tokens(cfg, 150)
        t["l0.mix.sink"] = torch.tensor([level, level + 1, level - 1]).bfloat16()
        t["l0.norm1b"] = t["l0.norm1b"] * 0.5
        ref = plain.forward(cfg, as_f64(t), toks)
        monkeypatch.setitem(plain.KNOBS, "sink", False)
        gone = rel_err(plain.forward(cfg, as_f64(t), toks), ref)
        monkeypatch.undo()
        assert gone > SHOWS if level > -10 else gone < 1e-9
        for dtype in ("float32", "bfloat16"):
            with fasulix.from_tensors(cfg, t, dtype, max_tokens=512, max_seqs=2, page=8) as m:
                for cut in ([150], [1], [40, 1]):
                    assert rel_err(in_portions(m, toks, cut), ref, dtype) < TOL[dtype]


def test_prompt_attention_as_products_keeps_the_scores_exact(monkeypatch):
    """bfloat16 mode computes a long portion's attention as tensor-core products over gathered latents, short portions with the fused fp32
    kernel.  Scores and softmax weights keep fp32 accuracy on both (queries, keys and probabilities travel as bf16 value + remainder
    pairs), so with sharp scores the two agree as closely as the rest of the bf16 path allows, also for a portion that continues a cached
    prefix inside a window; a window that is one off shows far above that."""
    for size in (23, 4, 0):
        cfg = config([latent(size=size, scale=2.0), latent(size=9, heads=4, dim=8, scale=1.0, kv_from=0)])
        t, toks = weights(cfg, 17), tokens(cfg, 120)
        ref = plain.forward(cfg, as_f64(t), toks)
        errs = {}
        for products in ("1", "0"):
            monkeypatch.setenv("CALM_B200_SEQ_ATTN_PRODUCTS", products)
            with fasulix.from_tensors(cfg, t, "bfloat16", max_tokens=300, max_seqs=3, page=8) as m:
                s1, s2 = m.open(), m.open()
                a = m.step([s1], [toks[:50]], list(range(50)))
                b = m.step([s1, s2], [toks[50:], toks[:3]], list(range(73)))  # 70 more tokens on the products path beside a 3-token portion
                errs[products] = rel_err(np.concatenate([a, b[:70]]), ref, "bfloat16")
                assert rel_err(b[70:], ref[:3], "bfloat16") < TOL["bfloat16"]
        assert errs["1"] < TOL["bfloat16"] and errs["0"] < TOL["bfloat16"] and errs["1"] < 1.5 * errs["0"] + 1e-3
        if size:
            for off in (-1, 1):
                wrong = copy.deepcopy(cfg)
                wrong["layers"][0]["mixer"]["mask"]["size"] += off
                assert rel_err(plain.forward(wrong, as_f64(t), toks), ref) > 4 * errs["1"]


def test_decode_attention_on_tensor_cores_keeps_the_scores_exact(monkeypatch):
    """bfloat16 mode serves decoded tokens and short portions with a tensor-core kernel whose scores, weights and values enter as bf16 value +
    remainder: with sharp scores it stays as close to the plain statement as the fused fp32 kernel it replaces.  Seventeen heads make two
    head tiles, 40 keys more than one staged chunk, a latent width that is no multiple of 16 or 4 the unaligned copies."""
    for kw in (dict(heads=17, kv_rank=40, rot_dim=8), dict(heads=16, kv_rank=37, rot_dim=2, vdim=5), dict(heads=3, kv_rank=64, rot_dim=16)):
        cfg = config([latent(scale=1.5, **kw), latent(size=37, scale=1.5, kv_from=0, **kw)])
        t, toks = weights(cfg, 19), tokens(cfg, 90)
        t["l0.mix.sink"] += 1.0
        ref = plain.forward(cfg, as_f64(t), toks)
        errs = {}
        for mma in ("1", "0"):
            monkeypatch.setenv("CALM_B200_SEQ_ATTN_MMA", mma)
            with fasulix.from_tensors(cfg, t, "bfloat16", max_tokens=300, max_seqs=2, page=8) as m:
                errs[mma] = max(rel_err(in_portions(m, toks, cut), ref, "bfloat16") for cut in ([1], [15, 7], [80, 1]))
        assert errs["1"] < TOL["bfloat16"] and errs["0"] < TOL["bfloat16"] and errs["1"] < 1.5 * errs["0"] + 1e-3


@pytest.mark.parametrize("alternate", [1, 0])
def test_dense_units_in_sandwich_blocks(alternate):
    """A feed-forward of one routed expert weighs it by one, so the same weights bound as a dense clamped unit (its rows alternating or
    stacked, the residual gate a matrix of its own) must give the same logits."""
    cfg = config([gru(mlp=moe(experts=1, top=1, ff=20)), latent(size=5, mlp=moe(experts=1, top=1, ff=9))])
    t, toks = weights(cfg, 20), tokens(cfg, 33)
    ref = plain.forward(cfg, as_f64(t), toks)
    head, layers, up = fasulix.plan(cfg, t)
    W = cfg["width"]
    for i, rec in enumerate(layers):
        f = f"l{i}.mlp."
        up[f + "rg2"], up[f + "rg2.b"] = up[rec["w_router"]][:W].contiguous(), up[rec["b_router"]][:W].contiguous()
        if not alternate:
            up[rec["w_gate_up"]] = torch.cat([up[rec["w_gate_up"]][0::2], up[rec["w_gate_up"]][1::2]], 0).contiguous()
        for k in ("w_router", "b_router", "experts", "top", "route_mode", "route_scale", "expert_act"):
            del rec[k]
        rec.update(ff_kind=seqlib.FF_CLAMPED, glu_rows=alternate, w_rg2=f + "rg2", b_rg2=f + "rg2.b")
    for dtype in ("float32", "bfloat16"):
        with seqlib.SeqDeviceModel(head, layers, up, exact=dtype == "float32", max_tokens=128, max_seqs=2, page=8) as m:
            for cut in ([33], [20, 1]):
                assert rel_err(in_portions(m, toks, cut), ref, dtype) < TOL[dtype]


def test_tensor_core_products_match_the_warp_level_ones(monkeypatch):
    """bfloat16 mode runs products over many tokens on tcgen05 (the grouped ones of the experts and the split query product included) and
    everything else on mma.sync; same bf16 inputs, fp32 sums in another order."""
    cfg = config([latent(heads=4, dim=32, rot_dim=16, vdim=24, q_rank=40, kv_rank=64, mlp=moe(experts=5, top=5, ff=40)), gru(width=72, mlp=moe(experts=3, top=3, ff=72)),
                  latent(size=50, heads=2, dim=32, rot_dim=16, vdim=24, q_rank=48, kv_rank=64, kv_from=0)], width=88, vocab=131)
    t, toks = weights(cfg, 18), tokens(cfg, 300)
    outs = {}
    for tc in ("1", "0"):
        monkeypatch.setenv("CALM_B200_SEQ_TC", tc)
        with fasulix.from_tensors(cfg, t, "bfloat16", max_tokens=640, max_seqs=2, page=16) as m:
            s1 = m.open()
            outs[tc] = np.concatenate([m.step([s1], [toks[:237]], list(range(237))), m.step([s1], [toks[237:]], list(range(63)))])
            if tc == "1":
                m.perf(True)
                whole(m, toks)
                stats = m.perf_stats()
                m.perf(False)
                assert stats["gemm_tcgen05"][3] > 0 and stats["mingru_scan"][3] > 0
    assert rel_err(outs["1"], outs["0"]) < 5e-3  # identical inputs; intermediate bf16 roundings may flip on last-bit differences
    assert rel_err(outs["1"], plain.forward(cfg, as_f64(t), toks), "bfloat16") < TOL["bfloat16"]


def test_long_decoding_keeps_state():
    """130 tokens one by one: the recurrent state and the cache grow by single steps, over many window lengths and pages."""
    cfg = config([gru(), latent(mlp=moe()), latent(size=12), gru(width=5), latent(size=7, kv_from=2)])
    t, toks = weights(cfg, 14), tokens(cfg, 130)
    ref = plain.forward(cfg, as_f64(t), toks)
    with fasulix.from_tensors(cfg, t, "float32", max_tokens=200, max_seqs=2, page=8) as m:
        assert rel_err(in_portions(m, toks, [1]), ref) < TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_equals_each_alone(dtype):
    ml = free_of_choices(dtype)
    cfg = config([gru(mlp=ml), latent(), latent(size=4, mlp=ml), gru(width=31), latent(size=6, kv_from=2)])
    t = weights(cfg, 21)
    prompts = [tokens(cfg, n, seed=n) for n in (1, 9, 90, 2)]
    tails = [tokens(cfg, n, seed=50 + n) for n in (6, 3, 0, 6)]
    p = as_f64(t)
    refs = [plain.forward(cfg, p, a + b) for a, b in zip(prompts, tails)]
    with fasulix.from_tensors(cfg, t, dtype, max_tokens=320, max_seqs=5, page=4) as m:
        slots = [m.open() for _ in prompts]
        out = m.step(slots, prompts, list(range(sum(len(a) for a in prompts))))
        got, at = [], 0
        for a in prompts:
            got.append([out[at:at + len(a)]])
            at += len(a)
        for k in range(6):  # decoded together; the shorter ones leave earlier
            live = [i for i, b in enumerate(tails) if k < len(b)]
            o = m.step([slots[i] for i in live], [[tails[i][k]] for i in live], list(range(len(live))))
            for j, i in enumerate(live):
                got[i].append(o[j:j + 1])
        for i, r in enumerate(refs):
            assert rel_err(np.concatenate(got[i]), r, dtype) < TOL[dtype]
        if dtype == "float32":  # a row does not depend on what else is in the batch, beyond rounding
            alone = whole(m, prompts[2])
            assert np.abs(alone - np.concatenate(got[2])[:90]).max() < 1e-5 * np.abs(alone).max()


def test_many_sequences_decode_together():
    """More decoded tokens in a step than the one-CTA routing kernel takes (64), at different positions."""
    cfg = config([gru(mlp=moe()), latent(size=5, mlp=moe(top=1))])
    t = weights(cfg, 24)
    p = as_f64(t)
    seqs = [tokens(cfg, 3 + i % 9, seed=100 + i) for i in range(70)]
    with fasulix.from_tensors(cfg, t, "float32", max_tokens=1024, max_seqs=70, page=4) as m:
        slots = [m.open() for _ in seqs]
        m.step(slots, [s[:-2] for s in seqs], [])
        m.step(slots, [[s[-2]] for s in seqs], [])
        out = m.step(slots, [[s[-1]] for s in seqs], list(range(70)))
    ref = np.stack([plain.forward(cfg, p, s)[-1] for s in seqs])
    assert rel_err(out, ref) < TOL["float32"]


def test_slots_and_pages_are_used_again():
    """A slot that is opened again starts from zero state and fresh pages."""
    cfg = config([gru(), latent(mlp=moe()), latent(size=6), latent(size=6, kv_from=2)])
    t = weights(cfg, 22)
    p = as_f64(t)
    with fasulix.from_tensors(cfg, t, "float32", max_tokens=48, max_seqs=2, page=4) as m:
        free0 = m.free_pages()
        for rnd in range(4):  # every pass fills the pool almost completely, with other lengths than the pass before
            a, b = tokens(cfg, 20 + rnd, seed=rnd), tokens(cfg, 23 - rnd, seed=9 + rnd)
            sa, sb = m.open(), m.open()
            out = m.step([sa, sb], [a, b], list(range(len(a) + len(b))))
            assert rel_err(out[:len(a)], plain.forward(cfg, p, a)) < TOL["float32"]
            assert rel_err(out[len(a):], plain.forward(cfg, p, b)) < TOL["float32"]
            m.close_seq(sb if rnd % 2 else sa)
            m.close_seq(sa if rnd % 2 else sb)
            assert m.free_pages() == free0
        s = m.open()
        with pytest.raises(Exception):
            m.step([s], [tokens(cfg, 4 * free0 + 1)], [0])  # more than the pool holds: refused, nothing has run
        assert m.length(s) == 0
        one = tokens(cfg, 3, seed=77)
        assert rel_err(m.step([s], [one], [0, 1, 2]), plain.forward(cfg, p, one)) < TOL["float32"]


def test_greedy_generation_through_the_scheduler():
    cfg = config([gru(mlp=moe()), latent(mlp=moe()), latent(size=6)])
    t = weights(cfg, 23)
    p = as_f64(t)
    prompts = [tokens(cfg, n, seed=70 + n) for n in (5, 17, 1)]
    with fasulix.from_tensors(cfg, t, "float32", max_tokens=256, max_seqs=2, page=8) as m:
        outs = serving.generate(m, prompts, 12, max_batch=2)  # three requests, two slots: a second batch follows the first
        assert m.free_pages() == 256 // 8 + 2
    for pr, out in zip(prompts, outs):
        assert len(out) == 12
        lg = plain.forward(cfg, p, pr + out)
        for k, tok in enumerate(out):  # each generated token is the plain statement's argmax given the same history
            row = lg[len(pr) + k - 1]
            assert tok == int(row.argmax()) or row.max() - row[tok] < 1e-4 * np.abs(row).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_from_a_model_folder(tmp_path, dtype):
    """bin/trace_run end to end: a model folder written with the container writer and found through the registry, steps on
    standard input (a batch of unequal prompts, decoding together while requests leave, a second batch afterwards), logits
    files compared with the plain statement."""
    ml = free_of_choices(dtype)
    cfg = config([latent(size=11, heads=4, dim=16, rot_dim=8, vdim=12, q_rank=20, kv_rank=28, mlp=ml), gru(width=36, mlp=ml), latent(heads=2, vdim=8),
                  latent(size=3, heads=2, rot_dim=8, q_rank=12, kv_rank=28, kv_from=0)], width=72, vocab=211, eps=1e-6)
    t = weights(cfg, 41)
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir(), out.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    container.write_tensors(str(folder / "model.safetensors"), t)
    assert registry.architecture_of(str(folder)) == "Fasulix"
    reqs = {"a": tokens(cfg, 46, 1), "b": tokens(cfg, 9, 2), "c": tokens(cfg, 4, 7), "d": tokens(cfg, 30, 4), "e": tokens(cfg, 2, 5)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": reqs["a"][:40], "want": [0, 17, 39]}, {"id": "b", "tokens": reqs["b"][:6], "want": [5]},
                                     {"id": "c", "tokens": reqs["c"][:1], "want": [0]}], "end": []}]
    for k in range(3):
        ent = [{"id": "a", "tokens": [reqs["a"][40 + k]], "want": [0]}, {"id": "b", "tokens": [reqs["b"][6 + k]], "want": [0] if k != 1 else []},
               {"id": "c", "tokens": [reqs["c"][1 + k]], "want": [0]}]
        steps.append({"step": 1 + k, "entries": ent, "end": ["b", "c"] if k == 2 else []})
    for k in range(3):
        steps.append({"step": 4 + k, "entries": [{"id": "a", "tokens": [reqs["a"][43 + k]], "want": [0]}], "end": ["a"] if k == 2 else []})
    steps.append({"step": 7, "entries": [{"id": "d", "tokens": reqs["d"][:29], "want": [28]}, {"id": "e", "tokens": reqs["e"][:1], "want": []}], "end": []})
    steps.append({"step": 8, "entries": [{"id": "d", "tokens": reqs["d"][29:], "want": [0]}, {"id": "e", "tokens": reqs["e"][1:], "want": [0]}], "end": ["d", "e"]})
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "96"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == ["done %d" % s["step"] for s in steps]
    ref = {k: plain.forward(cfg, as_f64(t), v) for k, v in reqs.items()}
    at = {k: 0 for k in reqs}
    for s in steps:
        rows = []
        for e in s["entries"]:
            rows += [ref[e["id"]][at[e["id"]] + w] for w in e["want"]]
            at[e["id"]] += len(e["tokens"])
        path = out / ("%d.f32" % s["step"])
        if rows:
            got = np.fromfile(path, "<f4").reshape(len(rows), cfg["vocab"])
            assert rel_err(got, np.stack(rows), dtype) < TOL[dtype]
        else:
            assert not path.exists()
