"""Tabisun: a decoder whose config.json lists its layers.  A sublayer reads the residual stream itself and its output comes back
through a layer norm (weight, no bias), x <- x + norm1(mixer(x)), x <- x + norm2(feed-forward(x)).  A layer may use the tensors of
another one (weights_of) with a cache of its own.  Mixers: differential attention inside chunks of positions, without rotation
("attention"); grouped-query attention whose values are the projected keys, with neighbouring channels rotated together, frequencies
rescaled by wavelength and a soft cap on the scores ("attention_2"); latent attention with queries straight from the input, a rotated key
part shared by the heads, a sink and a gate per output channel ("latent_attention").  The first two norm every head's queries and keys.
Feed-forward: down(silu(gate) * up).  The logits come from a matrix of their own and are soft-capped.

This module is the host side, like the other families' modules: it reads config.json, checks every tensor's shape, stacks what reads
the same input into one matrix and binds everything in the records of seqlib.  Kernels, cache and state live in libcalm_b200_seq.so;
every size and constant comes from the config or a tensor's shape."""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Tuple

import torch

from . import container, seqlib

ARCHITECTURE = "Tabisun"


def owner(cfg: dict, i: int) -> int:
    """the layer whose tensors layer i uses"""
    layers, seen = cfg["layers"], {i}
    while layers[i].get("weights_of") is not None:
        j = int(layers[i]["weights_of"])
        if not 0 <= j < len(layers) or j in seen:
            raise ValueError(f"layer {i}: weights_of {j} names no layer with tensors")
        if any(layers[j].get(k) != layers[i].get(k) for k in ("type", "mixer", "mlp")):
            raise ValueError(f"layer {i} uses the tensors of layer {j} but differs from it")
        seen.add(j)
        i = j
    return i


def neighbours(rows: torch.Tensor) -> torch.Tensor:
    """[..., P, width] rows whose channels i and i + P/2 turn together -> the order in which the runtime turns 2i and 2i + 1 together.  Queries
    and keys are reordered alike, which their products do not see."""
    half = rows.shape[-2] // 2
    return torch.stack([rows[..., :half, :], rows[..., half:, :]], -2).reshape(rows.shape)


def plan(cfg: dict, tensors: Dict[str, torch.Tensor]) -> Tuple[dict, List[dict], Dict[str, torch.Tensor]]:
    """config + checkpoint tensors -> (model head, layer records, tensors to upload)."""
    if cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config")
    width, vocab = int(cfg["width"]), int(cfg["vocab"])
    up: Dict[str, torch.Tensor] = {}

    def need(name: str, shape) -> str:
        if name not in tensors:
            raise KeyError(f"checkpoint lacks tensor {name}")
        t = tensors[name]
        if list(t.shape) != list(shape):
            raise ValueError(f"tensor {name} has shape {list(t.shape)}, the config asks for {list(shape)}")
        up[name] = t if t.dtype == torch.bfloat16 else t.to(torch.bfloat16)
        return name

    def take(name: str, shape) -> torch.Tensor:
        return up.pop(need(name, shape))

    def put(name: str, parts: List[torch.Tensor]) -> str:
        up[name] = torch.cat(parts, 0).contiguous()
        return name

    def grouped(m: str, mx: dict) -> dict:
        H, G, D, Dv = int(mx["heads"]), int(mx.get("kv_heads", mx["heads"])), int(mx["dim"]), int(mx["vdim"])
        if G < 1 or H % G:
            raise ValueError(f"{m}: {H} heads do not share {G} key heads evenly")
        return {"type": seqlib.SEQ_GQA, "heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "taps": 1, "scale": float(mx["scale"]), "qk_per_head": 1, "no_gate": 1, "scores_f32": 1,
                "q_norm": need(m + "q.norm", [D]), "k_norm": need(m + "k.norm", [D]), "w_o": need(m + "o", [width, H * Dv])}

    def differential(m: str, mx: dict) -> dict:
        rec = grouped(m, mx)
        H, G, D, Dv = rec["heads"], rec["kv_heads"], rec["dim"], rec["vdim"]
        # a key head has two maps; the queries of the heads that share a map of it stand side by side: [key head][map][head of the group]
        q = take(m + "q", [H * 2 * D, width]).reshape(G, H // G, 2, D, width).transpose(1, 2).reshape(H * 2 * D, width)
        rec["w_in"] = put(m + "in", [q, take(m + "k", [G * 2 * D, width]), take(m + "v", [G * Dv, width])])
        l1, k1, l2, k2 = (take(m + n, [D]).double() for n in ("lq1", "lk1", "lq2", "lk2"))
        diff = float(mx["diff"])
        rec.update(maps=2, diff_lambda=math.exp(float((l1 * k1).sum())) - math.exp(float((l2 * k2).sum())) + diff, diff_mul=1.0 - diff, chunk=int((mx.get("mask") or {}).get("size", 0)))
        return rec

    def capped(m: str, mx: dict) -> dict:
        rec = grouped(m, mx)
        H, G, D = rec["heads"], rec["kv_heads"], rec["dim"]
        if rec["vdim"] != D:
            raise ValueError(f"{m}: values taken from the keys are {D} wide, vdim says {rec['vdim']}")
        rot = mx.get("rot") or {}
        rec["w_in"] = put(m + "in", [take(m + "q", [H * D, width]), take(m + "k", [G * D, width])])
        rec.update(v_from_k=1, softcap=float(mx.get("softcap") or 0.0), rot_pairs=1, rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)))
        sc = rot.get("scaling")
        if sc:
            rec.update(rot_kind=1, rot_factor=float(sc["factor"]), rot_original=float(sc["original"]), rot_low=float(sc["low"]), rot_high=float(sc["high"]))
        return rec

    def latent(m: str, mx: dict) -> dict:
        H, D, P, Dv, R = (int(mx[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        rot = mx["rot"]
        if int(rot["dims"]) != P:
            raise ValueError(f"{m}: rot.dims {rot['dims']} is not rot_dim {P}")
        rec = {"type": seqlib.SEQ_LATENT, "heads": H, "kv_heads": 1, "dim": D, "vdim": Dv, "taps": 1, "q_rank": 0, "kv_rank": R, "scale": float(mx["scale"]),
               "rot_dims": P, "rot_base": float(rot["base"]), "gate_channels": 1, "scores_f32": 1}
        sc = rot.get("scaling")
        if sc:
            rec.update(rot_factor=float(sc["factor"]), rot_original=float(sc["original"]), rot_fast=float(sc["fast"]), rot_slow=float(sc["slow"]))
        q = take(m + "q", [H * (D + P), width]).reshape(H, D + P, width)  # head by head [unrotated, rotated]
        down = take(m + "dkv", [R + P, width])
        rec["w_in"] = put(m + "in", [neighbours(q[:, D:]).reshape(H * P, width), down[:R], neighbours(down[R:]), take(m + "g", [H * Dv, width]), q[:, :D].reshape(H * D, width)])
        rec["dkv_norm"], rec["w_uv"], rec["sink"] = need(m + "dkv.norm", [R]), need(m + "uv", [H * Dv, R]), need(m + "sink", [H])
        up[m + "ukT"] = take(m + "uk", [H * D, R]).reshape(H, D, R).transpose(1, 2).contiguous()  # per head [kv_rank, dim]: the key side folded into the query
        rec["w_ukT"], rec["w_o"] = m + "ukT", need(m + "o", [width, H * Dv])
        return rec

    mixers = {"attention": differential, "attention_2": capped, "latent_attention": latent}

    def layer(i: int) -> dict:
        lc, p = cfg["layers"][i], f"l{i}."
        if lc["type"] not in mixers:
            raise ValueError(f"layer {i}: unknown mixer {lc['type']}")
        rec = mixers[lc["type"]](p + "mix.", lc["mixer"])
        rec["norm1"] = need(p + "norm1", [width])
        ml = lc.get("mlp")
        if ml:
            if ml["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {ml['kind']} is not part of this design")
            f, ff = p + "mlp.", int(ml["ff"])
            gate, upr = take(f + "gate", [ff, width]), take(f + "up", [ff, width])
            up[f + "gate_up"] = torch.stack([gate, upr], 1).reshape(2 * ff, width).contiguous()  # alternating rows: the unit is formed in the product's epilogue
            rec.update(ff=ff, ff_kind=seqlib.FF_GATED, ff_act=seqlib.ACT_SILU, glu_rows=1, w_gate_up=f + "gate_up", w_down=need(f + "down", [width, ff]), norm2=need(p + "norm2", [width]))
        return rec

    own: Dict[int, dict] = {}
    for i in range(len(cfg["layers"])):
        j = owner(cfg, i)
        if j not in own:
            own[j] = layer(j)
    # layers that share tensors are records of their own with the same tensor names (uploaded once), so each has its own cache
    layers = [dict(own[owner(cfg, i)]) for i in range(len(cfg["layers"]))]
    head = {"vocab": vocab, "width": width, "eps": float(cfg["norm"]["eps"]), "embed": need("embed", [vocab, width]), "head": need("head", [vocab, width]),
            "final_norm": need("final.norm", [width]), "norm_kind": seqlib.NORM_LN, "norm_offset": 0.0, "block": seqlib.BLOCK_POST,
            "logit_cap": float(cfg.get("logit_softcap") or 0.0)}
    return head, layers, up


def load(folder: str, dtype: str = "bfloat16", max_tokens: int = 4096, max_seqs: int = 64, page: int = 16) -> seqlib.SeqDeviceModel:
    """config.json + model.safetensors of `folder` onto the GPU."""
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    tensors, _ = container.read_tensors(os.path.join(folder, "model.safetensors"))
    return from_tensors(cfg, tensors, dtype, max_tokens, max_seqs, page)


def from_tensors(cfg: dict, tensors: Dict[str, torch.Tensor], dtype: str = "bfloat16", max_tokens: int = 4096, max_seqs: int = 64, page: int = 16):
    if dtype not in ("bfloat16", "float32"):
        raise ValueError("dtype must be bfloat16 or float32")
    head, layers, up = plan(cfg, tensors)
    return seqlib.SeqDeviceModel(head, layers, up, exact=dtype == "float32", max_tokens=max_tokens, max_seqs=max_seqs, page=page)


# ---------------------------------------------------------------- synthetic checkpoints (tests, bench)

def tensor_shapes(cfg: dict) -> Dict[str, list]:
    W, out = int(cfg["width"]), {}
    out["embed"] = [cfg["vocab"], W]
    for i, lc in enumerate(cfg["layers"]):
        if lc.get("weights_of") is not None:
            continue
        p, mx = f"l{i}.", lc["mixer"]
        m, H, D, Dv = p + "mix.", mx["heads"], mx["dim"], mx["vdim"]
        G = mx.get("kv_heads", H)
        out[p + "norm1"] = [W]
        if lc["type"] == "latent_attention":
            P, R = mx["rot_dim"], mx["kv_rank"]
            out.update({m + "q": [H * (D + P), W], m + "dkv": [R + P, W], m + "dkv.norm": [R], m + "uk": [H * D, R], m + "uv": [H * Dv, R], m + "sink": [H], m + "g": [H * Dv, W]})
        else:
            maps = 2 if lc["type"] == "attention" else 1
            out.update({m + "q": [H * maps * D, W], m + "k": [G * maps * D, W], m + "q.norm": [D], m + "k.norm": [D]})
            if maps == 2:
                out[m + "v"] = [G * Dv, W]
                out.update({m + n: [D] for n in ("lq1", "lk1", "lq2", "lk2")})
        out[m + "o"] = [W, H * Dv]
        if lc.get("mlp"):
            f, ff = p + "mlp.", lc["mlp"]["ff"]
            out.update({p + "norm2": [W], f + "gate": [ff, W], f + "up": [ff, W], f + "down": [W, ff]})
    out.update({"final.norm": [W], "head": [cfg["vocab"], W]})
    return out


def random_tensors(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Seeded bf16 weights with magnitudes that keep every mechanism active (gates open, two maps that differ, scores and logits that
    reach into their soft caps)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm", "norm1", "norm2"):
            t = (0.5 if leaf in ("norm1", "norm2") else 1.0) * (1.0 + 0.2 * torch.randn(shape, generator=g))
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            t = torch.randn(shape, generator=g) * (0.7 / shape[-1] ** 0.25)
        elif leaf == "embed":
            t = torch.randn(shape, generator=g) * 0.7
        elif leaf == "sink":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * (1.2 / math.sqrt(shape[-1]))
        out[name] = t.to(torch.bfloat16)
    return out
