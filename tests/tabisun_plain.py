"""Plain float64 statement of the Tabisun design, one function per mechanism, token loops and no cache: the slow oracle the
runtime is compared with.  It shares no code with calm_b200 (numpy only; tensors come in as float64 arrays).

Notation: x [T, width] is one sequence's residual stream; a sublayer reads x itself and its output y comes back through a layer norm,
x <- x + LN(y).  p is the position of a token (0 for the first)."""
from __future__ import annotations

import math
from typing import Dict, List

import numpy as np

# mechanisms a test can leave out (or read wrongly) to show that the comparison would notice
KNOBS = {"center": True, "chunk_shift": 0, "diff": True, "head_norm": True, "values_are_raw_keys": True, "interleaved": True, "wavelengths": True, "cap": True,
         "halves": True, "yarn": True, "magnitude": True, "sink": True, "gate": True, "logit_cap": True, "maps_by_head": True, "one_minus": True}


def layer_norm(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    d = x - x.mean(-1, keepdims=True) if KNOBS["center"] else x
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w


def rms_norm(x: np.ndarray, w, eps: float) -> np.ndarray:
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def soft_cap(z, cap: float):
    return cap * np.tanh(z / cap)


def frequencies_by_wavelength(dims: int, base: float, sc: dict | None) -> List[float]:
    """angle per position of every pair; waves longer than original/low turn `factor` times slower, those shorter than original/high keep
    their speed, a linear blend between"""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc and KNOBS["wavelengths"]:
            wave, orig, low, high, fac = 2.0 * math.pi / f, float(sc["original"]), float(sc["low"]), float(sc["high"]), float(sc["factor"])
            if wave > orig / low:
                f = f / fac
            elif wave >= orig / high:
                s = (orig / wave - low) / (high - low)
                f = (1.0 - s) * f / fac + s * f
        out.append(f)
    return out


def frequencies_by_ramp(dims: int, base: float, sc: dict | None):
    """(angle per position of every pair, factor on cos and sin): a ramp over the pair index between the pairs that turn `fast` and `slow`
    times in the original context"""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0
    orig, fac = float(sc["original"]), float(sc["factor"])
    at = lambda t: dims * math.log(orig / (2.0 * math.pi * t)) / (2.0 * math.log(base))  # noqa: E731
    lo, hi = max(math.floor(at(float(sc["fast"]))), 0), min(math.ceil(at(float(sc["slow"]))), dims - 1)
    if KNOBS["yarn"]:
        for i in range(dims // 2):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f[i] = f[i] / fac * ramp + f[i] * (1.0 - ramp)
    return f, (0.1 * math.log(fac) + 1.0 if KNOBS["magnitude"] else 1.0)


def turn(v: np.ndarray, freq: List[float], mag: float, interleaved: bool) -> np.ndarray:
    """v [T, heads, dim]: the first 2 len(freq) channels turn by the position; pair i is (2i, 2i+1) or (i, i + len(freq))"""
    out, n = v.copy(), len(freq)
    for p in range(v.shape[0]):
        for i, f in enumerate(freq):
            a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + n)
            c, s = mag * math.cos(p * f), mag * math.sin(p * f)
            out[p, :, a], out[p, :, b] = v[p, :, a] * c - v[p, :, b] * s, v[p, :, b] * c + v[p, :, a] * s
    return out


def sees(i: int, j: int, size: int) -> bool:
    """query position i sees key position j: causal, and (with a chunk size) in the same chunk counted from position 0"""
    return j <= i and (size <= 0 or (i + KNOBS["chunk_shift"]) // size == (j + KNOBS["chunk_shift"]) // size)


def softmax_values(q: np.ndarray, k: np.ndarray, v: np.ndarray, scale: float, size: int = 0, cap: float = 0.0, sink: float | None = None) -> np.ndarray:
    """one head: q, k [T, d], v [T, dv] -> [T, dv]; `sink` joins the denominator only"""
    out = np.zeros((q.shape[0], v.shape[1]))
    for i in range(q.shape[0]):
        js = [j for j in range(i + 1) if sees(i, j, size)]
        s = (k[js] @ q[i]) * scale
        if cap > 0:
            s = soft_cap(s, cap)
        top = max(s.max(), sink if sink is not None else -math.inf)
        w = np.exp(s - top)
        out[i] = (w @ v[js]) / (w.sum() + (math.exp(sink - top) if sink is not None else 0.0))
    return out


def differential_attention(t, m: str, mx: dict, h: np.ndarray, eps: float) -> np.ndarray:
    H, G, D, Dv = int(mx["heads"]), int(mx["kv_heads"]), int(mx["dim"]), int(mx["vdim"])
    T, size, scale, diff = h.shape[0], int(mx["mask"]["size"]), float(mx["scale"]), float(mx["diff"])
    shape = lambda z, n: z.reshape(T, n, 2, D) if KNOBS["maps_by_head"] else z.reshape(T, 2, n, D).transpose(0, 2, 1, 3)  # noqa: E731
    q = rms_norm(shape(h @ t[m + "q"].T, H), t[m + "q.norm"], eps)
    k = rms_norm(shape(h @ t[m + "k"].T, G), t[m + "k.norm"], eps)
    v = (h @ t[m + "v"].T).reshape(T, G, Dv)
    lam = math.exp((t[m + "lq1"] * t[m + "lk1"]).sum()) - math.exp((t[m + "lq2"] * t[m + "lk2"]).sum()) + diff
    out = np.zeros((T, H, Dv))
    for a in range(H):
        g = a // (H // G)
        o = softmax_values(q[:, a, 0], k[:, g, 0], v[:, g], scale, size)
        if KNOBS["diff"]:
            o = o - lam * softmax_values(q[:, a, 1], k[:, g, 1], v[:, g], scale, size)
        if KNOBS["head_norm"]:
            o = rms_norm(o, 1.0, eps)
        out[:, a] = o * ((1.0 - diff) if KNOBS["one_minus"] else 1.0)
    return out.reshape(T, H * Dv) @ t[m + "o"].T


def capped_attention(t, m: str, mx: dict, h: np.ndarray, eps: float) -> np.ndarray:
    """the values are the keys as projected, before norm and rotation"""
    H, G, D = int(mx["heads"]), int(mx["kv_heads"]), int(mx["dim"])
    T, rot = h.shape[0], mx["rot"]
    q, raw = (h @ t[m + "q"].T).reshape(T, H, D), (h @ t[m + "k"].T).reshape(T, G, D)
    q, k = rms_norm(q, t[m + "q.norm"], eps), rms_norm(raw, t[m + "k.norm"], eps)
    v = raw if KNOBS["values_are_raw_keys"] else k
    f = frequencies_by_wavelength(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
    q, k = turn(q, f, 1.0, KNOBS["interleaved"]), turn(k, f, 1.0, KNOBS["interleaved"])
    cap = float(mx["softcap"]) if KNOBS["cap"] else 0.0
    out = np.stack([softmax_values(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], float(mx["scale"]), cap=cap) for a in range(H)], 1)
    return out.reshape(T, H * D) @ t[m + "o"].T


def latent_attention(t, m: str, mx: dict, h: np.ndarray, eps: float) -> np.ndarray:
    H, D, P, Dv, R = (int(mx[n]) for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    T, rot = h.shape[0], mx["rot"]
    f, mag = frequencies_by_ramp(P, float(rot["base"]), rot.get("scaling"))
    q = (h @ t[m + "q"].T).reshape(T, H, D + P)
    down = h @ t[m + "dkv"].T
    c = rms_norm(down[:, :R], t[m + "dkv.norm"], eps)
    kr = turn(down[:, None, R:], f, mag, not KNOBS["halves"])[:, 0]
    qr = turn(q[:, :, D:], f, mag, not KNOBS["halves"])
    ku, v = (c @ t[m + "uk"].T).reshape(T, H, D), (c @ t[m + "uv"].T).reshape(T, H, Dv)
    out = np.zeros((T, H, Dv))
    for a in range(H):
        out[:, a] = softmax_values(np.concatenate([q[:, a, :D], qr[:, a]], 1), np.concatenate([ku[:, a], kr], 1), v[:, a], float(mx["scale"]),
                                   sink=float(t[m + "sink"][a]) if KNOBS["sink"] else None)
    out = out.reshape(T, H * Dv)
    if KNOBS["gate"]:
        out = out * sigmoid(h @ t[m + "g"].T)
    return out @ t[m + "o"].T


MIXERS = {"attention": differential_attention, "attention_2": capped_attention, "latent_attention": latent_attention}


def dense_unit(t, f: str, h: np.ndarray) -> np.ndarray:
    return (silu(h @ t[f + "gate"].T) * (h @ t[f + "up"].T)) @ t[f + "down"].T


def owner(cfg: dict, i: int) -> int:
    """the layer whose tensors layer i uses"""
    while cfg["layers"][i].get("weights_of") is not None:
        i = int(cfg["layers"][i]["weights_of"])
    return i


def forward(cfg: dict, t: Dict[str, np.ndarray], toks: List[int], layers_out: list | None = None) -> np.ndarray:
    """logits [T, vocab] of one sequence"""
    eps = float(cfg["norm"]["eps"])
    x = t["embed"][list(toks)]
    for i, lc in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."
        x = x + layer_norm(MIXERS[lc["type"]](t, p + "mix.", lc["mixer"], x, eps), t[p + "norm1"], eps)
        if lc.get("mlp"):
            x = x + layer_norm(dense_unit(t, p + "mlp.", x), t[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    logits = layer_norm(x, t["final.norm"], eps) @ t["head"].T
    return soft_cap(logits, float(cfg["logit_softcap"])) if KNOBS["logit_cap"] else logits
