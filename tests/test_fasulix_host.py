"""Host-side tests of the Fasulix family (no GPU): the loader's plan, the registry, and properties of the plain statement that
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
import fasulix_plain as plain  # noqa: E402

from calm_b200 import container, fasulix, registry, seqlib  # noqa: E402

MOE = {"kind": "moe", "expert": {"ff": 12, "limit": 0.8}, "router": {"experts": 3, "top": 2}}
FULL = {"heads": 3, "dim": 6, "rot_dim": 4, "vdim": 5, "q_rank": 10, "kv_rank": 14, "scale": 0.4, "rot": {"dims": 4, "base": 100.0}}
WIN = dict(FULL, heads=2, vdim=7, mask={"size": 5})
CFG = {"architecture": "Fasulix", "norm": {"eps": 1e-5}, "vocab": 53, "width": 24,
       "layers": [{"type": "mingru", "mixer": {"width": 20}, "mlp": MOE}, {"type": "latent_attention", "mixer": FULL, "mlp": None},
                  {"type": "latent_attention_2", "mixer": WIN, "mlp": {"kind": "moe", "expert": {"ff": 6, "limit": 2.0}, "router": {"experts": 2, "top": 1}}},
                  {"type": "latent_attention_2", "mixer": dict(WIN, kv_from=1, mask={"size": 9}), "mlp": MOE}]}


def as_f64(t):
    return {k: v.float().numpy().astype(np.float64) for k, v in t.items()}


def test_plan_binds_every_size_from_the_config():
    t = fasulix.random_tensors(CFG, 1)
    head, layers, up = fasulix.plan(CFG, t)
    assert head["block"] == seqlib.BLOCK_SANDWICH and head["norm_kind"] == seqlib.NORM_RMS and head["norm_offset"] == 0.0 and head["res_gate"] == 1
    assert head["head"] == head["embed"] == "embed" and head["eps"] == 1e-5
    a, b, c, d = layers
    # the residual gate's rows lead the input matrix of every sublayer, with their bias
    assert a["type"] == seqlib.SEQ_MINGRU and a["dim"] == a["vdim"] == 20 and a["heads"] == 1
    assert up[a["w_in"]].shape == (24 + 60, 24) and torch.equal(up[a["w_in"]][:24], t["l0.rg1"]) and torch.equal(up[a["w_in"]][44:64], t["l0.mix.x"])
    assert torch.equal(up[a["b_in"]][24:44], t["l0.mix.z.b"]) and torch.equal(up[a["b_in"]][44:64], t["l0.mix.x.b"]) and not up[a["b_in"]][64:].any()
    assert a["ff_kind"] == seqlib.FF_MOE and a["route_mode"] == 1 and a["expert_act"] == 2 and a["limit"] == 0.8 and a["experts"] == 3 and a["top"] == 2
    assert up[a["w_router"]].shape == (27, 24) and torch.equal(up[a["w_router"]][24:], t["l0.mlp.router"]) and torch.equal(up[a["b_router"]][:24], t["l0.rg2.b"]) and not up[a["b_router"]][24:].any()
    assert up[a["w_gate_up"]].shape == (3 * 24, 24) and torch.equal(up[a["w_gate_up"]][24:48:2], t["l0.mlp.e1.gate"]) and torch.equal(up[a["w_gate_up"]][25:48:2], t["l0.mlp.e1.up"])
    assert up[a["w_down"]].shape == (72, 12) and up[a["dwa"]].shape == (2,)
    assert b["type"] == seqlib.SEQ_LATENT and b["no_gate"] == 1 and b["rot_dims"] == 4 and b["rot_base"] == 100.0 and "window" not in b and up[b["sink"]].shape == (3,)
    assert up[b["w_in"]].shape == (24 + 10 + 18, 24) and "ff" not in b and "norm2" not in b and up[b["dwa"]].shape == (3,)
    # the query projection: every head's rotated rows first, then every head's unrotated rows
    assert torch.equal(up[b["w_uq"]][:4], t["l1.mix.uq"][6:10]) and torch.equal(up[b["w_uq"]][12:18], t["l1.mix.uq"][:6]) and torch.equal(up[b["w_uq"]][8:12], t["l1.mix.uq"][26:])
    assert torch.equal(up[b["w_ukT"]][1], t["l1.mix.uk"][6:12].T)
    assert c["window"] == 5 and "sink" not in c and "kv_shared" not in c and c["limit"] == 2.0
    assert d["window"] == 9 and d["kv_shared"] == 2 and "dkv_norm" not in d and up[d["w_in"]].shape == (24 + 10, 24) and up[d["dwa"]].shape == (5,)


def test_plan_refuses_what_does_not_fit():
    t = fasulix.random_tensors(CFG, 1)
    for path, val in ((("mixer", "heads"), 4), (("mixer", "kv_rank"), 13), (("mixer", "rot", "dims"), 2)):
        wrong = copy.deepcopy(CFG)
        at = wrong["layers"][1]
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = val
        with pytest.raises(ValueError):
            fasulix.plan(wrong, t)
    for name in ("l1.mix.sink", "l0.rg1.b", "l3.dwa", "l2.norm2b", "l2.mix.dkv.norm"):
        short = dict(t)
        del short[name]
        with pytest.raises(KeyError):
            fasulix.plan(CFG, short)
    for src in (3, 4, 0, -1):  # itself, a later layer, a layer without latents, none
        wrong = copy.deepcopy(CFG)
        wrong["layers"][3]["mixer"]["kv_from"] = src
        with pytest.raises(ValueError):
            fasulix.plan(wrong, t)
    wrong = copy.deepcopy(CFG)
    wrong["layers"][0]["type"] = "attention"
    with pytest.raises(ValueError):
        fasulix.plan(wrong, t)
    wrong = copy.deepcopy(CFG)
    wrong["layers"][0]["mlp"]["kind"] = "dense"
    with pytest.raises(ValueError):
        fasulix.plan(wrong, t)


def test_registry_finds_the_family(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    container.write_tensors(str(tmp_path / "model.safetensors"), fasulix.random_tensors(CFG, 2))
    assert registry.architecture_of(str(tmp_path)) == "Fasulix"
    registry._defaults()
    assert registry.SEQ_LOADERS["Fasulix"] is fasulix.load
    back, _ = container.read_tensors(str(tmp_path / "model.safetensors"))
    assert back["l3.dwa"].shape == (5,) and "l3.mix.dkv" not in back and "l1.rg2" not in back and "head" not in back


def test_records_match_the_header():
    """Every field the header adds for this family is in the ctypes mirror, in the header's order."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    text = open(os.path.join(root, "include", "calm_b200_seq.h")).read()
    body = text[text.index("struct SeqLayer {"):text.index("struct SeqModel {")]
    names = [n for n, _ in seqlib.SeqLayer._fields_]
    tail = ["kv_shared", "dwa", "w_rg2", "b_rg2", "glu_rows"]
    assert names[names.index(tail[0]):][:len(tail)] == tail
    at = [body.index((" " if n in ("kv_shared", "glu_rows") else "* ") + n + ";") for n in tail]
    assert at == sorted(at)
    mnames = [n for n, _ in seqlib.SeqModel._fields_]
    assert mnames[mnames.index("logit_scale"):][:2] == ["logit_scale", "res_gate"]
    model = text[text.index("struct SeqModel {"):]
    assert model.index("logit_scale;") < model.index("res_gate;")


def test_plain_statement_is_causal_and_the_window_bounds_the_attention():
    t = as_f64(fasulix.random_tensors(CFG, 3))
    rng = np.random.default_rng(0)
    a = [int(x) for x in rng.integers(0, 53, 30)]
    b = a[:20] + [int(x) for x in rng.integers(0, 53, 10)]
    la, lb = plain.forward(CFG, t, a), plain.forward(CFG, t, b)
    assert np.allclose(la[:20], lb[:20], atol=1e-12) and not np.allclose(la[20:], lb[20:])
    # the attention alone: a change at position 3 reaches position 7 (window of 5) and no further; the shared latents alike
    h = rng.normal(size=(12, 24))
    h2 = h.copy()
    h2[3] += 1.0
    o1, o2 = (plain.latent_attention(t, "l2.mix.", WIN, v, plain.latent_of(t, "l2.mix.", WIN, v, 1e-5), 1e-5) for v in (h, h2))
    assert not np.allclose(o1[7], o2[7]) and np.allclose(o1[8:], o2[8:], atol=1e-12) and np.allclose(o1[:3], o2[:3], atol=1e-12)
    assert [j for j in range(12) if plain.sees(8, j, 5)] == [4, 5, 6, 7, 8] and [j for j in range(4) if plain.sees(2, j, 0)] == [0, 1, 2]
    # the recurrence remembers across it
    r1, r2 = plain.min_gru(t, "l0.mix.", {"width": 20}, h), plain.min_gru(t, "l0.mix.", {"width": 20}, h2)
    assert np.allclose(r1[:3], r2[:3], atol=1e-12) and not np.allclose(r1[4], r2[4])


def test_recurrence_rotation_and_expert_by_hand():
    t = {"m.z": np.zeros((2, 2)), "m.z.b": np.array([0.0, math.log(3.0)]), "m.x": np.eye(2), "m.x.b": np.zeros(2), "m.g": np.zeros((2, 2)), "m.o": np.eye(2)}
    t["m.g"][:] = 1.0
    h = np.array([[1.0, -2.0], [3.0, 0.0]])
    s = lambda v: 1 / (1 + math.exp(-v))  # noqa: E731
    S1 = [0.5 * 1.5, 0.75 * s(-2.0)]
    S2 = [0.5 * S1[0] + 0.5 * 3.5, 0.25 * S1[1] + 0.75 * 0.5]
    want = np.array([S1, S2]) * np.array([[-1 * s(-1)], [3 * s(3)]])
    assert np.allclose(plain.min_gru(t, "m.", {"width": 2}, h), want)
    v = np.zeros((3, 1, 4))
    v[:, 0, 0] = 1.0  # channels 0 and 1 turn together, channels 2 and 3 by position * 100^(-2/4)
    v[:, 0, 3] = 1.0
    assert np.allclose(plain.rotate(v, 100.0)[2, 0], [math.cos(2.0), math.sin(2.0), -math.sin(0.2), math.cos(0.2)])
    e = {"e.gate": np.array([[5.0]]), "e.up": np.array([[-9.0]]), "e.down": np.array([[2.0]])}
    assert np.allclose(plain.expert(e, "e.", np.ones((1, 1)), 0.5), 2.0 * 0.5 * s(1.702 * 0.5) * (1.0 - 0.5))
    assert np.allclose(plain.expert(e, "e.", -np.ones((1, 1)), 0.5), 2.0 * -5.0 * s(1.702 * -5.0) * (1.0 + 0.5))  # the gate has no lower bound


def test_router_weights_are_scores_over_all_experts_and_ties_go_low():
    w = {"f.router": np.array([[0.0], [2.0], [2.0], [1.0]])}
    for e in range(4):
        w.update({f"f.e{e}.gate": np.ones((1, 1)), f"f.e{e}.up": np.zeros((1, 1)), f"f.e{e}.down": np.array([[10.0 ** e]])})
    y = plain.routed(w, "f.", {"router": {"experts": 4, "top": 1}, "expert": {"limit": 9.0}}, np.ones((1, 1)))
    z = np.exp([0.0, 2.0, 2.0, 1.0])
    assert np.allclose(y, z[1] / z.sum() * 10.0 / (1 + math.exp(-1.702)))


def test_one_layer_by_hand():
    """Norms around the sublayer, the gate read from the sublayer's input, the depth average over the embedding rows and the layer's result."""
    cfg = copy.deepcopy(CFG)
    cfg["layers"] = cfg["layers"][:1]
    cfg["layers"][0]["mlp"] = None
    t = as_f64(fasulix.random_tensors(cfg, 5))
    toks = [3, 9, 27, 1, 4, 4, 30]
    rms = lambda v, w: v / np.sqrt((v * v).mean(-1, keepdims=True) + 1e-5) * t[w]  # noqa: E731
    x = t["embed"][toks]
    h = rms(x, "l0.norm1")
    y = plain.min_gru(t, "l0.mix.", {"width": 20}, h) / (1 + np.exp(-(h @ t["l0.rg1"].T + t["l0.rg1.b"])))
    x1 = x + rms(y, "l0.norm1b")
    x2 = t["l0.dwa"][0] * x + t["l0.dwa"][1] * x1
    assert np.allclose(plain.forward(cfg, t, toks), rms(x2, "final.norm") @ t["embed"].T)
