"""The Tabisun family on the layer-list runtime against the plain float64 statement in tabisun_plain.py.

Every test makes its own small configuration and seeded weights.  float32 mode is compared tightly (it shows any wrong key, a chunk edge
that is one token off, a sink or a map left out, a wrong pairing of rotated channels); bfloat16 mode within bf16 rounding.  Where random
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
import tabisun_plain as plain  # noqa: E402

pytestmark = pytest.mark.gpu

from calm_b200 import container, registry, seqlib, serving, tabisun  # noqa: E402

DENSE = {"ff": 40, "kind": "dense"}


def diff(heads=4, kv_heads=2, dim=8, vdim=12, size=7, scale=0.6, lam=0.3, mlp=None, **more):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": lam, "mask": {"size": size}}, "mlp": mlp, **more}


def capped(heads=4, kv_heads=2, dim=12, rot=8, base=300.0, scale=0.5, softcap=6.0, factor=4.0, original=64, low=1.0, high=4.0, mlp=None, **more):
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "softcap": softcap,
                                             "rot": {"dims": rot, "base": base, "scaling": {"factor": factor, "original": original, "low": low, "high": high}}}, "mlp": mlp, **more}


def latent(heads=3, dim=8, rot_dim=8, vdim=6, kv_rank=24, scale=0.5, base=300.0, factor=3.0, original=64, fast=8.0, slow=1.0, mlp=None, **more):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                                  "rot": {"dims": rot_dim, "base": base, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}}, "mlp": mlp, **more}


def config(layers, width=48, vocab=97, eps=1e-5, cap=6.0):
    return {"architecture": "Tabisun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_softcap": cap}


def weights(cfg, seed=0):
    return tabisun.random_tensors(cfg, seed)


def as_f64(t):
    return {k: v.float().numpy().astype(np.float64) for k, v in t.items()}


def tokens(cfg, n, seed=1):
    return [int(x) for x in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def rel_err(got, ref, dtype="float32"):
    """Error of the worst row, relative to the spread of the reference logits.  In bfloat16 a few rows sit far above the others without
    any fault (two maps that almost cancel, and the norm behind them, multiply the rounding of what came before): there the measure is the
    larger of the ninth decile and a sixth of the worst row (a row computed from a wrong key is off by about one)."""
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
    with tabisun.from_tensors(cfg, t, dtype, max_tokens=4 * len(toks) + 64, max_seqs=4, page=page) as m:
        assert rel_err(whole(m, toks), ref, dtype) < TOL[dtype]
        for first in {1, max(1, len(toks) // 2)}:
            assert rel_err(in_portions(m, toks, [first, 1]), ref, dtype) < TOL[dtype]
        for size in portions:
            grow = [size + k for k in range(30)] if size > 2 else [size]  # growing portions: edges fall at ever different places
            assert rel_err(in_portions(m, toks, grow), ref, dtype) < TOL[dtype]
    return ref


LAYERS = {
    "differential": [diff()],
    "differential-dense": [diff(mlp=DENSE)],
    "differential-own-keys-per-head": [diff(heads=3, kv_heads=3, dim=16, vdim=8, size=5)],
    "differential-one-key-head": [diff(heads=5, kv_heads=1, dim=4, vdim=20)],
    "differential-chunks-of-one": [diff(size=1)],
    "differential-chunk-longer-than-the-prompt": [diff(size=64, lam=0.8)],
    "differential-one-head": [diff(heads=1, kv_heads=1, dim=32, vdim=8, size=16)],
    "capped": [capped()],
    "capped-full-rotation-own-keys-per-head": [capped(heads=2, kv_heads=2, dim=8, rot=8)],
    "capped-one-pair-turned-one-key-head": [capped(heads=6, kv_heads=1, rot=2)],
    "capped-one-head-tight-cap": [capped(heads=1, kv_heads=1, dim=32, rot=16, softcap=0.7, scale=1.0)],
    "capped-far-from-the-cap-no-blend": [capped(softcap=80.0, low=3.99, high=4.0, original=20)],
    "latent": [latent()],
    "latent-one-head": [latent(heads=1, dim=16, rot_dim=2, vdim=10, kv_rank=40)],
    "latent-more-rotated-than-unrotated": [latent(heads=2, dim=4, rot_dim=16, vdim=24, kv_rank=8, factor=1.5)],
    "latent-dense": [latent(mlp=DENSE)],
    "tensors-of-another-layer": [capped(), diff(mlp=DENSE), capped(weights_of=0), diff(mlp=DENSE, weights_of=1), latent(), latent(weights_of=4)],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(LAYERS))
def test_each_mechanism_alone(name, dtype):
    cfg = config(LAYERS[name])
    check_all_ways(cfg, weights(cfg, 3), tokens(cfg, 37), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_align_with_nothing(dtype):
    """Width, head sizes, ranks, feed-forward widths and vocabulary that are multiples of neither 8 nor 4."""
    cfg = config([latent(heads=3, dim=5, rot_dim=6, vdim=7, kv_rank=11, mlp={"ff": 13, "kind": "dense"}), diff(heads=6, kv_heads=2, dim=5, vdim=9, size=9),
                  capped(heads=3, kv_heads=1, dim=7, rot=6, mlp={"ff": 9, "kind": "dense"}), latent(heads=1, dim=9, rot_dim=2, vdim=11, kv_rank=15),
                  diff(heads=1, kv_heads=1, dim=3, vdim=5, size=4, mlp={"ff": 3, "kind": "dense"})], width=50, vocab=61)
    check_all_ways(cfg, weights(cfg, 31), tokens(cfg, 45), dtype, portions=(17, 2))


def test_wide_heads():
    """Value heads wider than the combining kernels keep in registers, a latent beyond what the attention kernel keeps per lane."""
    cfg = config([diff(heads=2, kv_heads=1, dim=40, vdim=300, size=11), diff(heads=2, kv_heads=2, dim=8, vdim=520, size=30), latent(heads=2, dim=16, rot_dim=8, vdim=8, kv_rank=600),
                  capped(heads=2, kv_heads=1, dim=264, rot=20, scale=0.1)])
    for dtype in ("float32", "bfloat16"):
        check_all_ways(cfg, weights(cfg, 30), tokens(cfg, 29), dtype, portions=(7,))


def test_wide_rows():
    """Rows wider than a thread keeps in registers (more than 4096 columns, and more than 1024 of a width that is no multiple of 4)."""
    for width in (4200, 1234):
        cfg = config([diff(size=5, mlp={"ff": 16, "kind": "dense"})], width=width, vocab=33)
        check_all_ways(cfg, weights(cfg, 29), tokens(cfg, 11), portions=(3,))


def test_other_layer_orders():
    for k, order in enumerate(([latent(mlp=DENSE), diff(), capped(), diff(size=3, mlp=DENSE)], [diff(size=2), diff(size=2, weights_of=0), latent(), capped(mlp=DENSE), diff(size=2, weights_of=1)],
                               [capped(weights_of=2), latent(), capped(), capped()])):
        cfg = config(order, width=40)
        check_all_ways(cfg, weights(cfg, 5 + k), tokens(cfg, 41), portions=(6,))


def test_residual_stream_after_every_layer():
    cfg = config([capped(mlp=DENSE), latent(), diff(mlp=DENSE), capped(mlp=DENSE, weights_of=0)])
    t, toks = weights(cfg, 8), tokens(cfg, 19)
    trace = []
    plain.forward(cfg, as_f64(t), toks, trace)
    with tabisun.from_tensors(cfg, t, "float32", max_tokens=64, max_seqs=2) as m:
        m.set_trace(True)
        whole(m, toks)
        got = m.read_trace(len(toks))
    assert got.shape[0] == len(trace) == 4
    for g, r in zip(got, trace):
        assert np.abs(g - r).max() < 1e-4 * max(1.0, np.abs(r).max())


def test_every_mechanism_shows(monkeypatch):
    """The runtime agrees with the plain statement; the plain statement with one mechanism left out or read otherwise is far outside the
    tolerance, and so is one with another constant.  (A large eps: the norm behind a sublayer hides a common factor of it, all but its eps.)"""
    cfg = config([capped(scale=1.0, mlp=DENSE), latent(scale=0.8, rot_dim=16, original=400), diff(size=6, scale=1.2), capped(softcap=3.0)], eps=0.05, cap=3.0)
    t, toks = weights(cfg, 11), tokens(cfg, 60)
    t["l1.mix.sink"] += 1.5
    ref = check_all_ways(cfg, t, toks, portions=(7, 2))
    p = as_f64(t)
    for knob, val in plain.KNOBS.items():
        for v in (1, -1) if knob == "chunk_shift" else (not val,):
            monkeypatch.setitem(plain.KNOBS, knob, v)
            assert rel_err(plain.forward(cfg, p, toks), ref) > SHOWS, knob
            monkeypatch.undo()
    for layer, path, val in ((0, ("scale",), 0.9), (0, ("softcap",), 7.0), (0, ("rot", "dims"), 6), (0, ("rot", "base"), 200.0), (0, ("rot", "scaling", "factor"), 3.0), (0, ("rot", "scaling", "original"), 90),
                             (0, ("rot", "scaling", "low"), 2.0), (0, ("rot", "scaling", "high"), 6.0), (1, ("scale",), 0.7), (1, ("rot", "base"), 200.0), (1, ("rot", "scaling", "factor"), 2.0),
                             (1, ("rot", "scaling", "original"), 20), (1, ("rot", "scaling", "fast"), 3.0), (1, ("rot", "scaling", "slow"), 0.05), (2, ("mask", "size"), 5), (2, ("mask", "size"), 7), (2, ("diff",), 0.35), (2, ("scale",), 1.0)):
        wrong = copy.deepcopy(cfg)
        at = wrong["layers"][layer]["mixer"]
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = val
        assert rel_err(plain.forward(wrong, p, toks), ref) > SHOWS, path
    for key, val in (("logit_softcap", 4.0), ("norm", {"eps": 0.04})):
        assert rel_err(plain.forward(dict(cfg, **{key: val}), p, toks), ref) > SHOWS, key


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_context_with_shared_out_keys(dtype):
    """Decoding few tokens over a context of several hundred: the attention kernels share one query's keys out over several CTAs and fold
    the shares (the sink counts once, the two maps fold on their own); positions in the hundreds turn the rotated channels by hundreds of
    radians; chunks of 200; pages are crossed all along."""
    sharp = 1.0 if dtype == "float32" else 0.4
    cfg = config([latent(heads=4, rot_dim=16, base=50.0, scale=sharp), diff(size=200, scale=sharp), capped(base=50.0, scale=sharp), diff(size=1000, heads=2, scale=sharp)])
    t, toks = weights(cfg, 15), tokens(cfg, 330)
    ref = plain.forward(cfg, as_f64(t), toks)
    with tabisun.from_tensors(cfg, t, dtype, max_tokens=700, max_seqs=2, page=16) as m:
        s = m.open()
        rows = [m.step([s], [toks[:300]], list(range(300)))]
        for p in range(300, 330):
            rows.append(m.step([s], [[toks[p]]], [0]))
        assert rel_err(np.concatenate(rows), ref, dtype) < TOL[dtype]
        assert rel_err(in_portions(m, toks, [2]), ref, dtype) < TOL[dtype]  # beside the finished sequence


FAR = {"attention": diff(heads=2, kv_heads=1, dim=16, vdim=8, size=120, scale=2.0), "attention-unbounded": diff(heads=2, kv_heads=1, dim=16, vdim=8, size=4096, scale=2.0),
       "attention_2": capped(heads=2, kv_heads=1, dim=16, rot=2, scale=2.0, softcap=40.0), "latent_attention": latent(heads=2, dim=16, rot_dim=2, vdim=8, kv_rank=32, scale=2.0)}


def matching_key(cfg, t, toks, key_tok=5, query_tok=3):
    """Make the queries of `query_tok` match the key of `key_tok` and no other: keys read the first half of the embedding columns, queries the
    second half through the same matrix, and the key token's first half is the query token's second half (their own keys and the values
    differ).  In differential attention it is the first map that matches."""
    lc, m = cfg["layers"][0], "l0.mix."
    mx, W = lc["mixer"], cfg["width"]
    H, D, h = mx["heads"], mx["dim"], W // 2
    g = torch.Generator().manual_seed(77)
    if lc["type"] == "latent_attention":
        R, P = mx["kv_rank"], mx["rot_dim"]
        code, uk = torch.randn(R, h, generator=g) / h ** 0.5, torch.randn(D, R, generator=g) / R ** 0.5
        down, q = torch.zeros(R + P, W), torch.zeros(H, D + P, W)
        down[:R, :h], q[:, :D, h:] = code, uk @ code
        t[m + "dkv"], t[m + "q"], t[m + "uk"], t[m + "dkv.norm"] = down.bfloat16(), q.reshape(-1, W).bfloat16(), uk.repeat(H, 1).bfloat16(), torch.ones(R).bfloat16()
        t[m + "sink"] = torch.full((H,), -4.0).bfloat16()
    else:
        maps, G = (2 if lc["type"] == "attention" else 1), mx["kv_heads"]
        code = torch.randn(D, h, generator=g) / h ** 0.5
        if maps == 1:
            code[:mx["rot"]["dims"]] = 0  # nothing of the match is turned
        q, k = t[m + "q"].float().reshape(H, maps, D, W), t[m + "k"].float().reshape(G, maps, D, W)
        q[:, 0], k[:, 0] = 0, 0
        q[:, 0, :, h:], k[:, 0, :, :h] = code, code
        t[m + "q"], t[m + "k"] = q.reshape(-1, W).bfloat16(), k.reshape(-1, W).bfloat16()
        t[m + "q.norm"] = t[m + "k.norm"] = torch.ones(D).bfloat16()
    t["embed"][key_tok, :h] = t["embed"][query_tok, h:]
    return [key_tok if i == 5 else 4 if x in (key_tok, query_tok) else x for i, x in enumerate(toks)]


@pytest.mark.parametrize("name", list(FAR))
def test_a_far_key_stands_out_where_it_is_seen(name):
    """Position 5 holds a key that later queries match far above every other.  The queries sit at the last position of its chunk of 120, at
    the first of the next one, and far away; without a bound they find it hundreds of positions back.  Prompt, portions and decoding
    alike, with page edges at every 16."""
    cfg = config([FAR[name]])
    t = weights(cfg, 16)
    toks = matching_key(cfg, t, tokens(cfg, 300))
    for x in (119, 120, 299):
        toks[x] = 3
    p = as_f64(t)
    ref = plain.forward(cfg, p, toks)
    gone = list(toks)
    gone[5] = 4  # without the key, rows that see it move, rows that do not see it stay as they are
    changed = plain.forward(cfg, p, gone)
    moved = lambda x: rel_err(changed[x:x + 1], ref[x:x + 1])  # noqa: E731
    assert moved(119) > 0.1 and all(moved(x) < 1e-9 if name == "attention" else moved(x) > 0.1 for x in (120, 299))
    with tabisun.from_tensors(cfg, t, "float32", max_tokens=1024, max_seqs=2, page=16) as m:
        assert rel_err(whole(m, toks), ref) < TOL["float32"]
        s = m.open()
        rows = [m.step([s], [toks[:115]], list(range(115)))] + [m.step([s], [[x]], [0]) for x in toks[115:130]] + [m.step([s], [toks[130:290]], list(range(160)))]
        rows += [m.step([s], [[x]], [0]) for x in toks[290:]]
        assert rel_err(np.concatenate(rows), ref) < TOL["float32"]
        m.close_seq(s)
        assert rel_err(in_portions(m, toks, [119, 1, 2]), ref) < TOL["float32"]
    with tabisun.from_tensors(cfg, t, "bfloat16", max_tokens=1024, max_seqs=2, page=16) as m:
        for cut in ([300], [119, 1], [110, 20, 2]):
            got = in_portions(m, toks, cut)
            assert rel_err(got, ref, "bfloat16") < TOL["bfloat16"] and rel_err(got[[119, 120, 299]], ref[[119, 120, 299]]) < 2 * TOL["bfloat16"]


def test_the_sink_takes_its_share(monkeypatch):
    """A sink far above every score leaves almost nothing of the values, one far below changes nothing, and it is not scaled: from the
    first token of a sequence on, with few keys and with hundreds."""
    for level, scale in ((6.0, 0.2), (-30.0, 0.2), (1.0, 3.0)):
        cfg = config([latent(scale=scale)], eps=1e-2)
        t, toks = weights(cfg, 42), tokens(cfg, 150)
        t["l0.mix.sink"] = torch.tensor([level, level + 1, level - 1]).bfloat16()
        ref = plain.forward(cfg, as_f64(t), toks)
        monkeypatch.setitem(plain.KNOBS, "sink", False)
        gone = rel_err(plain.forward(cfg, as_f64(t), toks), ref)
        monkeypatch.undo()
        assert gone > SHOWS if level > -10 else gone < 1e-9
        for dtype in ("float32", "bfloat16"):
            with tabisun.from_tensors(cfg, t, dtype, max_tokens=512, max_seqs=2, page=8) as m:
                for cut in ([150], [1], [40, 1]):
                    assert rel_err(in_portions(m, toks, cut), ref, dtype) < TOL[dtype]


def test_latent_scores_take_a_soft_cap_too(monkeypatch):
    """The soft cap is an option of the attention kernels, not of one mixer: a record of the latent attention takes it as well."""
    cfg = config([latent(scale=1.5)])
    t, toks = weights(cfg, 43), tokens(cfg, 70)
    head, layers, up = tabisun.plan(cfg, t)
    layers[0]["softcap"] = 1.5
    free, inner = plain.forward(cfg, as_f64(t), toks), plain.softmax_values
    monkeypatch.setattr(plain, "softmax_values", lambda *a, **kw: inner(*a, **dict(kw, cap=1.5)))
    ref = plain.forward(cfg, as_f64(t), toks)
    assert rel_err(free, ref) > SHOWS
    for dtype in ("float32", "bfloat16"):
        with seqlib.SeqDeviceModel(head, layers, up, exact=dtype == "float32", max_tokens=256, max_seqs=2, page=8) as m:
            for cut in ([70], [30, 1]):
                assert rel_err(in_portions(m, toks, cut), ref, dtype) < TOL[dtype]


def test_prompt_attention_as_products_keeps_the_scores_exact(monkeypatch):
    """bfloat16 mode computes a long portion's attention as tensor-core products over gathered keys, short portions with a fused kernel.
    Scores and softmax weights keep fp32 accuracy on both, so with sharp scores the two agree as closely as the rest of the bf16 path
    allows, also for a portion that continues a cached prefix inside a chunk and for both kinds of portion in one step; a chunk that is one
    off shows far above that."""
    for size in (23, 4, 300):
        cfg = config([diff(size=size, scale=1.5), capped(scale=1.0, mlp=DENSE), latent(scale=1.0)])
        t, toks = weights(cfg, 17), tokens(cfg, 120)
        ref = plain.forward(cfg, as_f64(t), toks)
        errs = {}
        for products in ("1", "0"):
            monkeypatch.setenv("CALM_B200_SEQ_ATTN_PRODUCTS", products)
            with tabisun.from_tensors(cfg, t, "bfloat16", max_tokens=300, max_seqs=3, page=8) as m:
                s1, s2 = m.open(), m.open()
                a = m.step([s1], [toks[:50]], list(range(50)))
                b = m.step([s1, s2], [toks[50:], toks[:3]], list(range(73)))  # 70 more tokens on the products path beside a 3-token portion
                errs[products] = rel_err(np.concatenate([a, b[:70]]), ref, "bfloat16")
                assert rel_err(b[70:], ref[:3], "bfloat16") < TOL["bfloat16"]
        assert errs["1"] < TOL["bfloat16"] and errs["0"] < TOL["bfloat16"] and errs["1"] < 1.5 * errs["0"] + 1e-3
        if size < 120:
            for off in (-1, 1):
                wrong = copy.deepcopy(cfg)
                wrong["layers"][0]["mixer"]["mask"]["size"] += off
                assert rel_err(plain.forward(wrong, as_f64(t), toks), ref) > 4 * errs["1"]


def test_decode_attention_on_tensor_cores_keeps_the_scores_exact(monkeypatch):
    """bfloat16 mode serves decoded tokens and short portions with a tensor-core kernel whose scores, weights and values enter as bf16 value +
    remainder: with sharp scores it stays as close to the plain statement as the fused fp32 kernel.  Seventeen and eighteen heads of one
    key head make two head tiles, odd head sizes the unaligned copies."""
    for kw in (dict(heads=17, kv_heads=1, dim=8), dict(heads=18, kv_heads=1, dim=10), dict(heads=6, kv_heads=3, dim=16)):
        cfg = config([diff(size=37, scale=1.0, vdim=kw["dim"] + 3, **kw), capped(scale=1.0, rot=4, **kw), latent(heads=kw["heads"], dim=kw["dim"], kv_rank=37, scale=1.0)])
        t, toks = weights(cfg, 19), tokens(cfg, 90)
        ref = plain.forward(cfg, as_f64(t), toks)
        errs = {}
        for mma in ("1", "0"):
            monkeypatch.setenv("CALM_B200_SEQ_ATTN_MMA", mma)
            with tabisun.from_tensors(cfg, t, "bfloat16", max_tokens=300, max_seqs=2, page=8) as m:
                errs[mma] = max(rel_err(in_portions(m, toks, cut), ref, "bfloat16") for cut in ([1], [15, 7], [80, 1]))
        assert errs["1"] < TOL["bfloat16"] and errs["0"] < TOL["bfloat16"] and errs["1"] < 1.5 * errs["0"] + 2e-3


def test_tensor_core_products_match_the_warp_level_ones(monkeypatch):
    """bfloat16 mode runs products over many tokens on tcgen05 (with the gate per channel, the gated unit and the split query rows in their
    epilogues) and everything else on mma.sync; same bf16 inputs, fp32 sums in another order."""
    cfg = config([latent(heads=4, dim=32, rot_dim=16, vdim=24, kv_rank=64, mlp={"ff": 72, "kind": "dense"}), diff(heads=4, kv_heads=2, dim=16, vdim=24, size=50),
                  capped(heads=4, kv_heads=2, dim=32, rot=16, mlp=DENSE)], width=88, vocab=131)
    t, toks = weights(cfg, 18), tokens(cfg, 300)
    outs = {}
    for tc in ("1", "0"):
        monkeypatch.setenv("CALM_B200_SEQ_TC", tc)
        with tabisun.from_tensors(cfg, t, "bfloat16", max_tokens=640, max_seqs=2, page=16) as m:
            s1 = m.open()
            outs[tc] = np.concatenate([m.step([s1], [toks[:237]], list(range(237))), m.step([s1], [toks[237:]], list(range(63)))])
            if tc == "1":
                m.perf(True)
                whole(m, toks)
                stats = m.perf_stats()
                m.perf(False)
                assert stats["gemm_tcgen05"][3] > 0
    ref = plain.forward(cfg, as_f64(t), toks)
    assert rel_err(outs["1"], outs["0"], "bfloat16") < 1e-2  # identical inputs; intermediate bf16 roundings may flip on last-bit differences
    assert rel_err(outs["1"], ref, "bfloat16") < TOL["bfloat16"]


def test_long_decoding():
    """130 tokens one by one: the cache grows by single steps, over many chunks and pages."""
    cfg = config([capped(), latent(mlp=DENSE), diff(size=12), capped(weights_of=0), diff(size=5)])
    t, toks = weights(cfg, 14), tokens(cfg, 130)
    ref = plain.forward(cfg, as_f64(t), toks)
    with tabisun.from_tensors(cfg, t, "float32", max_tokens=200, max_seqs=2, page=8) as m:
        assert rel_err(in_portions(m, toks, [1]), ref) < TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_equals_each_alone(dtype):
    cfg = config([capped(mlp=DENSE), latent(), diff(size=4, mlp=DENSE), capped(mlp=DENSE, weights_of=0)])
    t = weights(cfg, 21)
    prompts = [tokens(cfg, n, seed=n) for n in (1, 9, 90, 2)]
    tails = [tokens(cfg, n, seed=50 + n) for n in (6, 3, 0, 6)]
    p = as_f64(t)
    refs = [plain.forward(cfg, p, a + b) for a, b in zip(prompts, tails)]
    with tabisun.from_tensors(cfg, t, dtype, max_tokens=320, max_seqs=5, page=4) as m:
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_sequences_decode_together(dtype):
    """So many tokens in a step that no query's keys are shared out: the maps are then combined from single shares."""
    cfg = config([diff(size=5, heads=8, kv_heads=8, mlp=DENSE), capped()])
    t = weights(cfg, 24)
    p = as_f64(t)
    seqs = [tokens(cfg, 3 + i % 9, seed=100 + i) for i in range(70)]
    with tabisun.from_tensors(cfg, t, dtype, max_tokens=1024, max_seqs=70, page=4) as m:
        slots = [m.open() for _ in seqs]
        m.step(slots, [s[:-2] for s in seqs], [])
        m.step(slots, [[s[-2]] for s in seqs], [])
        out = m.step(slots, [[s[-1]] for s in seqs], list(range(70)))
    ref = np.stack([plain.forward(cfg, p, s)[-1] for s in seqs])
    assert rel_err(out, ref, dtype) < TOL[dtype]


def test_slots_and_pages_are_used_again():
    """A slot that is opened again starts from an empty cache and fresh pages."""
    cfg = config([capped(), latent(mlp=DENSE), diff(size=6), diff(size=6, weights_of=2)])
    t = weights(cfg, 22)
    p = as_f64(t)
    with tabisun.from_tensors(cfg, t, "float32", max_tokens=48, max_seqs=2, page=4) as m:
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
    cfg = config([capped(mlp=DENSE), latent(mlp=DENSE), diff(size=6), capped(mlp=DENSE, weights_of=0)])
    t = weights(cfg, 23)
    p = as_f64(t)
    prompts = [tokens(cfg, n, seed=70 + n) for n in (5, 17, 1)]
    with tabisun.from_tensors(cfg, t, "float32", max_tokens=256, max_seqs=2, page=8) as m:
        outs = serving.generate(m, prompts, 12, max_batch=2)  # three requests, two slots: a second batch follows the first
        assert m.free_pages() == 256 // 8 + 2
    for pr, out in zip(prompts, outs):
        assert len(out) == 12
        lg = plain.forward(cfg, p, pr + out)
        for k, tok in enumerate(out):  # each generated token is the plain statement's argmax given the same history
            row = lg[len(pr) + k - 1]
            assert tok == int(row.argmax()) or row.max() - row[tok] < 1e-4 * np.abs(row).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_and_generation_from_a_model_folder(tmp_path, dtype):
    """bin/trace_run end to end: a model folder written with the container writer and found through the registry, steps on
    standard input (a batch of unequal prompts, decoding together while requests leave, a second batch afterwards), logits
    files compared with the plain statement; then the command line generates from the same folder."""
    cfg = config([latent(heads=4, dim=16, rot_dim=8, vdim=12, kv_rank=28, mlp=DENSE), diff(heads=4, kv_heads=1, dim=16, vdim=8, size=11, mlp=DENSE), capped(heads=2, kv_heads=2, dim=16, rot=16),
                  latent(heads=4, dim=16, rot_dim=8, vdim=12, kv_rank=28, mlp=DENSE, weights_of=0)], width=72, vocab=211, eps=1e-6, cap=9.0)
    t = weights(cfg, 41)
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir(), out.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    container.write_tensors(str(folder / "model.safetensors"), t)
    assert registry.architecture_of(str(folder)) == "Tabisun"
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
    p = subprocess.run([sys.executable, "-m", "calm_b200.serving", str(folder), "--tokens", "5,17,3", "--tokens", "9", "-n", "6", "--dtype", dtype], cwd=root, capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    lines = [[int(x) for x in ln.split(",")] for ln in p.stdout.split()]
    assert [len(x) for x in lines] == [6, 6] and all(0 <= x < 211 for ln in lines for x in ln)
