"""Host-side tests of the Tabisun family (no GPU): the loader's plan, the registry, and properties of the plain statement that
the GPU tests lean on."""
import copy
import json
import math
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import tabisun_plain as plain  # noqa: E402

from calm_b200 import container, registry, seqlib, tabisun  # noqa: E402

DIFF = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 10, "scale": 0.4, "diff": 0.25, "mask": {"size": 5}}
CAP = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 8, "scale": 0.3, "softcap": 7.0, "rot": {"dims": 4, "base": 100.0, "scaling": {"factor": 4.0, "original": 32, "low": 1.0, "high": 4.0}}}
LAT = {"heads": 3, "dim": 5, "rot_dim": 4, "vdim": 7, "kv_rank": 9, "scale": 0.5, "rot": {"dims": 4, "base": 100.0, "scaling": {"factor": 2.0, "original": 40, "fast": 6.0, "slow": 1.0}}}
MLP = {"ff": 14, "kind": "dense"}
CFG = {"architecture": "Tabisun", "norm": {"eps": 1e-5}, "vocab": 53, "width": 24, "logit_softcap": 9.0,
       "layers": [{"type": "attention", "mixer": DIFF, "mlp": MLP}, {"type": "attention_2", "mixer": CAP, "mlp": None}, {"type": "latent_attention", "mixer": LAT, "mlp": MLP},
                  {"type": "attention", "mixer": DIFF, "mlp": MLP, "weights_of": 0}, {"type": "attention_2", "mixer": CAP, "mlp": None, "weights_of": 1}]}


def as_f64(t):
    return {k: v.float().numpy().astype(np.float64) for k, v in t.items()}


def test_plan_binds_every_size_from_the_config():
    t = tabisun.random_tensors(CFG, 1)
    assert not any(k.startswith(("l3.", "l4.")) for k in t)
    head, layers, up = tabisun.plan(CFG, t)
    assert head["block"] == seqlib.BLOCK_POST and head["norm_kind"] == seqlib.NORM_LN and head["norm_offset"] == 0.0 and head["logit_cap"] == 9.0
    assert head["embed"] == "embed" and head["head"] == "head"
    a, b, c, d, e = layers
    assert a["type"] == seqlib.SEQ_GQA and a["maps"] == 2 and a["chunk"] == 5 and a["diff_mul"] == 0.75 and "rot_dims" not in a and "softcap" not in a
    lam = sum(s * math.exp(float((t["l0.mix.lq" + n].double() * t["l0.mix.lk" + n].double()).sum())) for s, n in ((1, "1"), (-1, "2"))) + 0.25
    assert abs(a["diff_lambda"] - lam) < 1e-12
    w = up[a["w_in"]]
    assert w.shape == (4 * 2 * 6 + 2 * 2 * 6 + 2 * 10, 24)
    # queries by key head, map, head of the group: heads 0 and 1 share key head 0
    q = t["l0.mix.q"].reshape(4, 2, 6, 24)
    for row, (h, mp) in enumerate([(0, 0), (1, 0), (0, 1), (1, 1), (2, 0), (3, 0), (2, 1), (3, 1)]):
        assert torch.equal(w[6 * row:6 * row + 6], q[h, mp])
    assert torch.equal(w[48:72], t["l0.mix.k"]) and torch.equal(w[72:], t["l0.mix.v"])
    assert a["ff_kind"] == seqlib.FF_GATED and a["ff_act"] == seqlib.ACT_SILU and a["glu_rows"] == 1
    assert torch.equal(up[a["w_gate_up"]][0::2], t["l0.mlp.gate"]) and torch.equal(up[a["w_gate_up"]][1::2], t["l0.mlp.up"])
    assert b["v_from_k"] == b["rot_pairs"] == b["rot_kind"] == 1 and b["softcap"] == 7.0 and (b["rot_factor"], b["rot_original"], b["rot_low"], b["rot_high"]) == (4.0, 32.0, 1.0, 4.0)
    assert up[b["w_in"]].shape == (4 * 8 + 2 * 8, 24) and "ff" not in b and "norm2" not in b
    assert c["type"] == seqlib.SEQ_LATENT and c["q_rank"] == 0 and c["gate_channels"] == 1 and (c["rot_factor"], c["rot_original"], c["rot_fast"], c["rot_slow"]) == (2.0, 40.0, 6.0, 1.0)
    w = up[c["w_in"]]
    assert w.shape == (3 * 4 + 9 + 4 + 3 * 7 + 3 * 5, 24)
    q = t["l2.mix.q"].reshape(3, 9, 24)
    for h in range(3):  # rotated rows first, halves brought side by side
        assert torch.equal(w[4 * h:4 * h + 4], q[h, [5, 7, 6, 8]]) and torch.equal(w[46 + 5 * h:51 + 5 * h], q[h, :5])
    assert torch.equal(w[12:21], t["l2.mix.dkv"][:9]) and torch.equal(w[21:25], t["l2.mix.dkv"][[9, 11, 10, 12]]) and torch.equal(w[25:46], t["l2.mix.g"])
    assert up[c["w_ukT"]].shape == (3, 9, 5) and torch.equal(up[c["w_ukT"]][1].t(), t["l2.mix.uk"][5:10])
    assert d == a and d is not a and e == b  # records of their own over the same tensors


def test_layers_that_use_other_layers_tensors():
    cfg = copy.deepcopy(CFG)
    cfg["layers"][1]["weights_of"] = 4  # a later layer owns the tensors
    del cfg["layers"][4]["weights_of"]
    t = tabisun.random_tensors(cfg, 1)
    assert "l4.mix.q" in t and "l1.mix.q" not in t
    _, layers, up = tabisun.plan(cfg, t)
    assert layers[1] == layers[4] and torch.equal(up[layers[1]["w_in"]][:32], t["l4.mix.q"])
    assert tabisun.owner(cfg, 1) == plain.owner(cfg, 1) == 4
    chain = dict(CFG, layers=[CFG["layers"][1], dict(CFG["layers"][1], weights_of=0), dict(CFG["layers"][1], weights_of=1)])
    assert [tabisun.owner(chain, i) for i in range(3)] == [plain.owner(chain, i) for i in range(3)] == [0, 0, 0]
    for bad in (dict(CFG["layers"][3], weights_of=1), dict(CFG["layers"][3], weights_of=9), dict(CFG["layers"][3], weights_of=3)):
        with pytest.raises(ValueError):
            tabisun.plan(dict(CFG, layers=CFG["layers"][:3] + [bad]), tabisun.random_tensors(CFG, 1))


def test_plan_refuses_what_does_not_fit():
    t = tabisun.random_tensors(CFG, 1)
    for layer, key, val in ((0, "dim", 7), (0, "kv_heads", 3), (1, "vdim", 9), (2, "rot_dim", 2), (2, "vdim", 8)):
        wrong = copy.deepcopy(CFG)
        wrong["layers"] = wrong["layers"][:3]
        wrong["layers"][layer]["mixer"][key] = val
        with pytest.raises(ValueError):
            tabisun.plan(wrong, t)
    short = dict(t)
    del short["l2.mix.sink"]
    with pytest.raises(KeyError):
        tabisun.plan(CFG, short)
    for key, val in (("type", "linear"), ("mlp", {"ff": 14, "kind": "moe"})):
        other = copy.deepcopy(CFG)
        other["layers"] = other["layers"][:3]
        other["layers"][1][key] = val
        with pytest.raises(ValueError):
            tabisun.plan(other, t)


def test_registry_finds_the_family(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    container.write_tensors(str(tmp_path / "model.safetensors"), tabisun.random_tensors(CFG, 2))
    assert registry.architecture_of(str(tmp_path)) == "Tabisun"
    registry._defaults()
    assert registry.SEQ_LOADERS["Tabisun"] is tabisun.load
    back, _ = container.read_tensors(str(tmp_path / "model.safetensors"))
    assert back["head"].shape == (53, 24)


def test_records_match_the_header():
    """Every field the header adds for this family is in the ctypes mirror, in the header's order."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    text = open(os.path.join(root, "include", "calm_b200_seq.h")).read()
    body = text[text.index("struct SeqLayer {"):text.index("struct SeqModel {")]
    tail = ["glu_rows", "maps", "diff_lambda", "diff_mul", "v_from_k", "softcap", "rot_pairs", "rot_kind", "rot_low", "rot_high", "gate_channels"]
    names, mnames = [n for n, _ in seqlib.SeqLayer._fields_], [n for n, _ in seqlib.SeqModel._fields_]
    assert names[names.index(tail[0]):][:len(tail)] == tail
    at = [min(body.index(x) for x in (" " + n + ";", " " + n + ",") if x in body[body.index("glu_rows;") - 1:]) for n in tail]
    assert at == sorted(at)
    model = text[text.index("struct SeqModel {"):]
    assert mnames[mnames.index("res_gate"):][:2] == ["res_gate", "logit_cap"] and model.index("res_gate;") < model.index("logit_cap;")


def test_plain_statement_is_causal_and_chunks_bound_the_attention():
    t = as_f64(tabisun.random_tensors(CFG, 3))
    rng = np.random.default_rng(0)
    a = [int(x) for x in rng.integers(0, 53, 30)]
    b = a[:20] + [int(x) for x in rng.integers(0, 53, 10)]
    la, lb = plain.forward(CFG, t, a), plain.forward(CFG, t, b)
    assert np.allclose(la[:20], lb[:20], atol=1e-12) and not np.allclose(la[20:], lb[20:])
    assert np.abs(la).max() < 9.0
    h = rng.normal(size=(12, 24))
    h2 = h.copy()
    h2[3] += rng.normal(size=24)
    o1, o2 = plain.differential_attention(t, "l0.mix.", DIFF, h, 1e-5), plain.differential_attention(t, "l0.mix.", DIFF, h2, 1e-5)
    assert not np.allclose(o1[4], o2[4]) and np.allclose(o1[5:], o2[5:], atol=1e-12) and np.allclose(o1[:3], o2[:3], atol=1e-12)
    for mix, args in ((plain.capped_attention, ("l1.mix.", CAP)), (plain.latent_attention, ("l2.mix.", LAT))):
        o1, o2 = mix(t, *args, h, 1e-5), mix(t, *args, h2, 1e-5)
        assert np.allclose(o1[:3], o2[:3], atol=1e-12) and not np.allclose(o1[11], o2[11], atol=1e-6)


def test_frequencies_by_hand():
    f = plain.frequencies_by_wavelength(8, 10000.0, {"factor": 8.0, "original": 400, "low": 1.0, "high": 4.0})
    # wavelengths 6.3, 62.8, 628, 6283 against 100 (kept below) and 400 (divided above)
    assert np.allclose(f, [1.0, 0.1, 0.01 / 8, 0.001 / 8])
    f = plain.frequencies_by_wavelength(4, 100.0, {"factor": 4.0, "original": 20.0 * math.pi * 2.5, "low": 1.0, "high": 4.0})
    s = (2.5 - 1.0) / 3.0  # pair 1: f = 0.1, two and a half waves in the original context
    assert np.allclose(f, [1.0, (1 - s) * 0.1 / 4 + s * 0.1])
    f, mag = plain.frequencies_by_ramp(8, 10000.0, {"factor": 4.0, "original": 2000.0, "fast": 32.0, "slow": 1.0})
    # turns(pair): 318, 31.8, 3.18, 0.318; the pair index of 32 turns is 0.997 -> lo 0, that of one turn 2.50 -> hi 3
    r = [0.0, 1 / 3, 2 / 3, 1.0]
    assert np.allclose(f, [10.0 ** -i * (x / 4 + 1 - x) for i, x in enumerate(r)]) and abs(mag - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    v = np.zeros((3, 1, 5))
    v[:, 0, 0], v[:, 0, 4] = 1.0, 7.0
    assert np.allclose(plain.turn(v, [1.0, 0.1], 1.0, True)[2, 0], [math.cos(2.0), math.sin(2.0), 0, 0, 7.0])
    assert np.allclose(plain.turn(v, [1.0, 0.1], 2.0, False)[2, 0], [2 * math.cos(2.0), 0, 2 * math.sin(2.0), 0, 7.0])


def test_softmax_details_by_hand():
    q, k, v = np.array([[1.0], [2.0]]), np.array([[1.0], [3.0]]), np.array([[1.0], [5.0]])
    w = np.exp([4.0 * math.tanh(1.0 / 4.0), 4.0 * math.tanh(3.0 / 4.0)])  # scores 1 and 3 under a cap of 4 (scale 1/2)
    assert np.allclose(plain.softmax_values(q, k, v, 0.5, cap=4.0)[1], (w @ v) / w.sum())
    w = np.exp([1.0, 3.0])
    assert np.allclose(plain.softmax_values(q, k, v, 0.5, sink=2.0)[1], (w @ v) / (w.sum() + math.exp(2.0)))  # not scaled, no value
    assert np.allclose(plain.softmax_values(q, k, v, 0.5, size=1), v)


def test_post_norm_block_by_hand():
    """One layer: x + LN(mixer(x)), the mixer reading x itself, the feed-forward likewise, then the final norm, the head and the cap."""
    cfg = dict(CFG, layers=CFG["layers"][:1])
    t = as_f64(tabisun.random_tensors(cfg, 5))
    toks = [3, 9, 27, 1, 4, 4, 30]

    def ln(y, w):
        d = y - y.mean(-1, keepdims=True)
        return d / np.sqrt((d ** 2).mean(-1, keepdims=True) + 1e-5) * w

    x = t["embed"][toks]
    x = x + ln(plain.differential_attention(t, "l0.mix.", DIFF, x, 1e-5), t["l0.norm1"])
    g = x @ t["l0.mlp.gate"].T
    x = x + ln((g / (1 + np.exp(-g)) * (x @ t["l0.mlp.up"].T)) @ t["l0.mlp.down"].T, t["l0.norm2"])
    assert np.allclose(plain.forward(cfg, t, toks), 9.0 * np.tanh(ln(x, t["final.norm"]) @ t["head"].T / 9.0))


def test_first_token_of_a_chunk_by_hand():
    """Its own key alone is visible: both maps return its value, and the difference is normed away but for its sign."""
    t = as_f64(tabisun.random_tensors(CFG, 6))
    h = np.random.default_rng(1).normal(size=(11, 24))
    v = (h @ t["l0.mix.v"].T).reshape(11, 2, 10)
    lam = math.exp((t["l0.mix.lq1"] * t["l0.mix.lk1"]).sum()) - math.exp((t["l0.mix.lq2"] * t["l0.mix.lk2"]).sum()) + 0.25
    for p in (0, 5, 10):
        o = (1 - lam) * v[p]
        o = np.repeat(o / np.sqrt((o * o).mean(-1, keepdims=True) + 1e-5) * 0.75, 2, 0)  # heads 0, 1 read value head 0
        assert np.allclose(plain.differential_attention(t, "l0.mix.", DIFF, h, 1e-5)[p], o.reshape(-1) @ t["l0.mix.o"].T)
