"""Fasulix: a decoder whose config.json lists its layers.  Every sublayer has the model's RMS norm before and after it and a sigmoid
gate per column, read from the sublayer's own input, on its output; after a layer the stream becomes a learned weighted sum of the
embedding rows and everything the layers so far handed on (depth average).  Mixers: a gated recurrence per channel whose gates read
only the current token ("mingru"), latent attention with a rotated key part shared by the heads and a sink in the softmax
("latent_attention"), and the same under a sliding window without a sink ("latent_attention_2"), where a layer may also read the
latents an earlier layer caches instead of making its own (kv_from).  Feed-forward: routed clamped gated units weighted by a softmax
over all experts.  The logits come from the embedding table.

This module is the host side, like vimulorn.py, bovinex.py, zazilix.py and sopepel.py: it reads config.json, checks every tensor's
shape, stacks what reads the same input into one matrix and binds everything in the records of seqlib.  Kernels, cache and state live
in libcalm_b200_seq.so; every size and constant comes from the config or a tensor's shape."""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Tuple

import torch

from . import container, seqlib

ARCHITECTURE = "Fasulix"
LATENT = ("latent_attention", "latent_attention_2")


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

    def stack(name: str, parts: List[str]) -> str:
        up[name] = torch.cat([up.pop(p) for p in parts], 0).contiguous()
        return name

    def biases(name: str, parts: List[Tuple[str, int]]) -> str:
        """the stacked matrix's bias: a tensor's values, or zeros for rows without one"""
        up[name] = torch.cat([up.pop(need(b, [n])) if b else torch.zeros(n, dtype=torch.bfloat16) for b, n in parts], 0).contiguous()
        return name

    def recurrence(p: str, mx: dict) -> dict:
        m, D = p + "mix.", int(mx["width"])
        rec = {"type": seqlib.SEQ_MINGRU, "heads": 1, "kv_heads": 1, "dim": D, "vdim": D, "taps": 1}
        # the residual gate's rows lead: everything that reads the normed input is one product
        rec["w_in"] = stack(m + "in", [need(p + "rg1", [width, width])] + [need(m + n, [D, width]) for n in ("z", "x", "g")])
        rec["b_in"] = biases(m + "in.b", [(p + "rg1.b", width), (m + "z.b", D), (m + "x.b", D), ("", D)])
        rec["w_o"] = need(m + "o", [width, D])
        return rec

    def latent(i: int, p: str, kind: str, mx: dict) -> dict:
        m = p + "mix."
        H, D, P, Dv, Rq, Rk = (int(mx[k]) for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
        rot, src = mx["rot"], mx.get("kv_from")
        if int(rot["dims"]) != P:
            raise ValueError(f"layer {i}: rot.dims {rot['dims']} is not rot_dim {P}")
        rec = {"type": seqlib.SEQ_LATENT, "heads": H, "kv_heads": 1, "dim": D, "vdim": Dv, "taps": 1, "q_rank": Rq, "kv_rank": Rk, "scale": float(mx["scale"]),
               "rot_dims": P, "rot_base": float(rot["base"]), "no_gate": 1, "scores_f32": 1}
        rows, out_rows = [need(p + "rg1", [width, width]), need(m + "dq", [Rq, width])], Rq
        if src is None:
            rows.append(need(m + "dkv", [Rk + P, width]))
            rec["dkv_norm"], out_rows = need(m + "dkv.norm", [Rk]), Rq + Rk + P
        else:
            src = int(src)
            if not 0 <= src < i or cfg["layers"][src]["type"] not in LATENT or cfg["layers"][src]["mixer"].get("kv_from") is not None:
                raise ValueError(f"layer {i}: kv_from {src} is not an earlier layer with a latent of its own")
            rec["kv_shared"] = src + 1
        rec["w_in"] = stack(m + "in", rows)
        rec["b_in"] = biases(m + "in.b", [(p + "rg1.b", width), ("", out_rows)])
        rec["dq_norm"] = need(m + "dq.norm", [Rq])
        uq = up.pop(need(m + "uq", [H * (D + P), Rq])).reshape(H, D + P, Rq)  # head by head [unrotated, rotated] -> all rotated rows, then all unrotated ones
        up[m + "uq"] = torch.cat([uq[:, D:].reshape(H * P, Rq), uq[:, :D].reshape(H * D, Rq)], 0).contiguous()
        rec["w_uq"], rec["w_uv"] = m + "uq", need(m + "uv", [H * Dv, Rk])
        uk = up.pop(need(m + "uk", [H * D, Rk]))
        up[m + "ukT"] = uk.reshape(H, D, Rk).transpose(1, 2).contiguous()  # per head [kv_rank, dim]: the key side folded into the query
        rec["w_ukT"] = m + "ukT"
        if kind == "latent_attention":
            rec["sink"] = need(m + "sink", [H])
        else:
            rec["window"] = int(mx["mask"]["size"])
        rec["w_o"] = need(m + "o", [width, H * Dv])
        return rec

    layers = []
    for i, lc in enumerate(cfg["layers"]):
        p, mx, kind = f"l{i}.", lc["mixer"], lc["type"]
        if kind == "mingru":
            rec = recurrence(p, mx)
        elif kind in LATENT:
            rec = latent(i, p, kind, mx)
        else:
            raise ValueError(f"layer {i}: unknown mixer {kind}")
        rec["norm1"], rec["norm1b"] = need(p + "norm1", [width]), need(p + "norm1b", [width])
        rec["dwa"] = need(p + "dwa", [i + 2])
        ml = lc.get("mlp")
        if ml:
            if ml["kind"] != "moe":
                raise ValueError(f"layer {i}: feed-forward kind {ml['kind']} is not part of this design")
            f = p + "mlp."
            ff, E, top = int(ml["expert"]["ff"]), int(ml["router"]["experts"]), int(ml["router"]["top"])
            rec.update(ff=ff, ff_kind=seqlib.FF_MOE, experts=E, top=top, route_mode=1, route_scale=1.0, expert_act=2, limit=float(ml["expert"]["limit"]),
                       norm2=need(p + "norm2", [width]), norm2b=need(p + "norm2b", [width]))
            rec["w_router"] = stack(f + "in", [need(p + "rg2", [width, width]), need(f + "router", [E, width])])
            rec["b_router"] = biases(f + "in.b", [(p + "rg2.b", width), ("", E)])
            # experts side by side, [experts][gate and up rows alternating] and [experts][down]: one grouped product serves all of them, and the unit is
            # formed in its epilogue
            rec["glu_rows"] = 1
            pairs = [torch.stack([up.pop(need(f + f"e{e}.{n}", [ff, width])) for n in ("gate", "up")], 1).reshape(2 * ff, width) for e in range(E)]
            up[f + "gate_ups"] = torch.cat(pairs, 0).contiguous()
            rec["w_gate_up"] = f + "gate_ups"
            rec["w_down"] = stack(f + "downs", [need(f + f"e{e}.down", [width, ff]) for e in range(E)])
        layers.append(rec)
    head = {"vocab": vocab, "width": width, "eps": float(cfg["norm"]["eps"]), "embed": need("embed", [vocab, width]), "head": "embed",
            "final_norm": need("final.norm", [width]), "norm_kind": seqlib.NORM_RMS, "norm_offset": 0.0, "block": seqlib.BLOCK_SANDWICH, "res_gate": 1}
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
        p, mx = f"l{i}.", lc["mixer"]
        m = p + "mix."
        out.update({p + "norm1": [W], p + "norm1b": [W], p + "rg1": [W, W], p + "rg1.b": [W], p + "dwa": [i + 2]})
        if lc["type"] == "mingru":
            D = mx["width"]
            out.update({m + "z": [D, W], m + "z.b": [D], m + "x": [D, W], m + "x.b": [D], m + "g": [D, W], m + "o": [W, D]})
        else:
            H, D, P, Dv, Rq, Rk = (mx[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
            out.update({m + "dq": [Rq, W], m + "dq.norm": [Rq], m + "uq": [H * (D + P), Rq], m + "uk": [H * D, Rk], m + "uv": [H * Dv, Rk], m + "o": [W, H * Dv]})
            if mx.get("kv_from") is None:
                out.update({m + "dkv": [Rk + P, W], m + "dkv.norm": [Rk]})
            if lc["type"] == "latent_attention":
                out[m + "sink"] = [H]
        if lc.get("mlp"):
            f, ff, E = p + "mlp.", lc["mlp"]["expert"]["ff"], lc["mlp"]["router"]["experts"]
            out.update({p + "norm2": [W], p + "norm2b": [W], p + "rg2": [W, W], p + "rg2.b": [W], f + "router": [E, W]})
            for e in range(E):
                out.update({f + f"e{e}.gate": [ff, W], f + f"e{e}.up": [ff, W], f + f"e{e}.down": [W, ff]})
    out["final.norm"] = [W]
    return out


def random_tensors(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Seeded bf16 weights with magnitudes that keep every mechanism active (gates open, states that remember, clamps that are met,
    router choices spread over the experts, depth averages in which every earlier stream counts)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm", "norm1", "norm2", "norm1b", "norm2b"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "dwa":
            t = 0.3 * torch.randn(shape, generator=g)
            t[-1] += 1.0
        elif name.endswith(".z.b"):
            t = -1.0 + 1.5 * torch.randn(shape, generator=g)
        elif leaf == "b":
            t = 0.5 * torch.randn(shape, generator=g)
        elif leaf in ("embed", "sink"):
            t = torch.randn(shape, generator=g)
        elif leaf == "router":
            t = torch.randn(shape, generator=g) * (2.0 / math.sqrt(shape[-1]))
        else:
            t = torch.randn(shape, generator=g) * (1.2 / math.sqrt(shape[-1]))
        out[name] = t.to(torch.bfloat16)
    return out
