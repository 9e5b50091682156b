"""Plain float64 statement of the Fasulix design, one function per mechanism, token loops and no cache: the slow oracle the
runtime is compared with.  It shares no code with calm_b200 (numpy only; tensors come in as float64 arrays).

Notation: x [T, width] is one sequence's residual stream, X_k the stream a layer hands on before depth averaging (X_0 the embedding
rows); a sublayer reads h = norm(x) and its output y comes back gated and normed, x <- x + norm'(sigmoid(R h + r) * y).  p is the
position of a token (0 for the first)."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import numpy as np

# mechanisms a test can leave out (or read wrongly) to show that the comparison would notice
KNOBS = {"gate": True, "depth": True, "sink": True, "window_shift": 0, "interleaved": True, "renormalise": False, "half": True, "plus_one": True, "share_rotated": True}
# router margins of the last forward(): per routed layer, per token, the gap between the last chosen score and the best one left out
MARGINS: List[np.ndarray] = []


def rms_norm(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def min_gru(t, m: str, mx: dict, h: np.ndarray) -> np.ndarray:
    """per channel S <- (1 - z) S + z c, with gate z and candidate c read from the current token alone; read out through a SiLU gate"""
    z = sigmoid(h @ t[m + "z"].T + t[m + "z.b"])
    u = h @ t[m + "x"].T + t[m + "x.b"]
    c = np.where(u >= 0, u + (0.5 if KNOBS["half"] else 0.0), sigmoid(u))
    S, out = np.zeros(int(mx["width"])), []
    for i in range(h.shape[0]):
        S = (1.0 - z[i]) * S + z[i] * c[i]
        out.append(S)
    return (np.stack(out) * silu(h @ t[m + "g"].T)) @ t[m + "o"].T


def rotate(v: np.ndarray, base: float) -> np.ndarray:
    """v [T, heads, dims]: channels 2i and 2i+1 turn together by p * base^(-2i/dims)"""
    dims = v.shape[-1]
    out = np.empty_like(v)
    for p in range(v.shape[0]):
        for i in range(dims // 2):
            a = p * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            j, k = (2 * i, 2 * i + 1) if KNOBS["interleaved"] else (i, i + dims // 2)
            out[p, :, j], out[p, :, k] = v[p, :, j] * c - v[p, :, k] * s, v[p, :, k] * c + v[p, :, j] * s
    return out


def sees(i: int, j: int, size: int) -> bool:
    """query position i sees key position j: causal, and (with a window) among the last `size` positions, its own included"""
    return j <= i and (size <= 0 or i - j < size + KNOBS["window_shift"])


def latent_of(t, m: str, mx: dict, h: np.ndarray, eps: float):
    """what a layer caches: the normed latent [T, kv_rank] and the rotated key part [T, rot_dim] that all heads share"""
    R = int(mx["kv_rank"])
    d = h @ t[m + "dkv"].T
    return rms_norm(d[:, :R], t[m + "dkv.norm"], eps), rotate(d[:, None, R:], float(mx["rot"]["base"]))[:, 0]


def latent_attention(t, m: str, mx: dict, h: np.ndarray, cached, eps: float) -> np.ndarray:
    H, D, P, Dv = int(mx["heads"]), int(mx["dim"]), int(mx["rot_dim"]), int(mx["vdim"])
    T, size = h.shape[0], int((mx.get("mask") or {}).get("size", 0))
    c, kr = cached
    q = (rms_norm(h @ t[m + "dq"].T, t[m + "dq.norm"], eps) @ t[m + "uq"].T).reshape(T, H, D + P)
    qu, qr = q[:, :, :D], rotate(q[:, :, D:], float(mx["rot"]["base"]))
    ku, v = (c @ t[m + "uk"].T).reshape(T, H, D), (c @ t[m + "uv"].T).reshape(T, H, Dv)
    sink = t[m + "sink"] if (m + "sink") in t and KNOBS["sink"] else None
    out = np.zeros((T, H, Dv))
    for i in range(T):
        js = [j for j in range(T) if sees(i, j, size)]
        for a in range(H):
            s = np.array([(qu[i, a] @ ku[j, a] + qr[i, a] @ kr[j]) * float(mx["scale"]) for j in js])
            top = max(s.max(), sink[a]) if sink is not None else s.max()
            e = np.exp(s - top)
            out[i, a] = (e / (e.sum() + (math.exp(sink[a] - top) if sink is not None else 0.0))) @ v[js, a]
    return out.reshape(T, H * Dv) @ t[m + "o"].T


def expert(t, f: str, h: np.ndarray, limit: float) -> np.ndarray:
    g, u = np.minimum(h @ t[f + "gate"].T, limit), np.clip(h @ t[f + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + (1.0 if KNOBS["plus_one"] else 0.0))) @ t[f + "down"].T


def routed(t, f: str, ml: dict, h: np.ndarray) -> np.ndarray:
    E, top, limit = int(ml["router"]["experts"]), int(ml["router"]["top"]), float(ml["expert"]["limit"])
    z = h @ t[f + "router"].T
    out, margins = np.zeros_like(h), []
    for n in range(h.shape[0]):
        e = np.exp(z[n] - z[n].max())
        s = e / e.sum()
        order = sorted(range(E), key=lambda k: (-s[k], k))
        chosen = order[:top]
        total = s[chosen].sum() if KNOBS["renormalise"] else 1.0
        for k in chosen:
            out[n] += s[k] / total * expert(t, f"{f}e{k}.", h[n], limit)
        margins.append(z[n][order[top - 1]] - z[n][order[top]] if top < E else np.inf)
    MARGINS.append(np.array(margins))
    return out


def gated(t, g: str, h: np.ndarray, y: np.ndarray) -> np.ndarray:
    """a sublayer's output times a sigmoid read from the sublayer's own input"""
    return y * sigmoid(h @ t[g].T + t[g + ".b"]) if KNOBS["gate"] else y


def forward(cfg: dict, t: Dict[str, np.ndarray], toks: List[int], trace: Optional[list] = None) -> np.ndarray:
    """logits [T, vocab] of one sequence; `trace` collects the stream after every layer (depth averaged)"""
    eps = float(cfg["norm"]["eps"])
    x = t["embed"][toks]
    X, cached = [x], {}
    for i, lc in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", lc["mixer"]
        h = rms_norm(x, t[p + "norm1"], eps)
        if lc["type"] == "mingru":
            y = min_gru(t, p + "mix.", mx, h)
        else:
            src = mx.get("kv_from")
            cached[i] = latent_of(t, p + "mix.", mx, h, eps) if src is None else cached[src]
            if src is not None and not KNOBS["share_rotated"]:
                cached[i] = (cached[src][0], np.zeros_like(cached[src][1]))
            y = latent_attention(t, p + "mix.", mx, h, cached[i], eps)
        x = x + rms_norm(gated(t, p + "rg1", h, y), t[p + "norm1b"], eps)
        if lc.get("mlp"):
            h = rms_norm(x, t[p + "norm2"], eps)
            x = x + rms_norm(gated(t, p + "rg2", h, routed(t, p + "mlp.", lc["mlp"], h)), t[p + "norm2b"], eps)
        X.append(x)
        if KNOBS["depth"]:
            x = sum(w * Xk for w, Xk in zip(t[p + "dwa"], X))
        if trace is not None:
            trace.append(x)
    return rms_norm(x, t["final.norm"], eps) @ t["embed"].T
