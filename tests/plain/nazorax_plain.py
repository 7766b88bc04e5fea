"""A plain, slow implementation of the Nazorax design from its equations: one function per
mechanism, float64 on the CPU, one sequence at a time, attention as whole matrices.  It shares
no code with the engine; the tests hold the engine to it.

Notation: T tokens of one sequence at positions 0..T-1, h [T, width] a layer's normed input,
w a dict of float64 tensors by checkpoint name, p the name prefix of the part at hand, mx a
mixer's dict of sizes from the configuration.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64
GATE_SLOPE = 1.702
UP_SHIFT = 1.0


# ----------------------------------------------------------------------- small pieces
def silu(z):
    return z * torch.sigmoid(z)


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def tanh_norm(x, w, name):
    """No statistic of the row: tanh(alpha x) weight + bias, alpha one number."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def linear(x, w, name):
    """W x (+ b where the checkpoint has a bias of that name)."""
    y = x @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


def frequencies(rot) -> (List[float], float):
    """One frequency per pair, and the factor on cosines and sines."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def index_of(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(index_of(sc["fast"])), 0)
    hi = min(math.ceil(index_of(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1.0 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x, rot):
    """x [T, heads, d]: the pair (i, i + dims/2) of every head's first ``dims`` sizes turns by
    position times the pair's frequency."""
    T, dims = x.shape[0], rot["dims"]
    f, mag = frequencies(rot)
    half = dims // 2
    ang = torch.arange(T, dtype=F64)[:, None, None] * torch.tensor(f, dtype=F64)[None, None, :]
    c, s = torch.cos(ang) * mag, torch.sin(ang) * mag
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def softmax_attention(q, k, v, scale, window: Optional[int] = None, sinks=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads key head h // (H / G);
    position i sees j <= i (and i - j < window when there is one).  ``sinks``: one logit per
    query head that joins the denominator and has no value."""
    T, H, _ = q.shape
    G = k.shape[1]
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = dist >= 0
    if window is not None:
        seen = seen & (dist < window)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        if sinks is not None:
            s = torch.cat([s, sinks[h].expand(T, 1)], dim=1)
        out[:, h] = torch.softmax(s, dim=-1)[:, :T] @ v[:, g]
    return out


# ----------------------------------------------------------------------- mixers
def windowed_attention(h, w, p, mx):
    T, H, G, d, dv = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = linear(h, w, p + "q").view(T, H, d)
    k = linear(h, w, p + "k").view(T, G, d)
    v = linear(h, w, p + "v").view(T, G, dv)
    q, k = rotate_halves(q, mx["rot"]), rotate_halves(k, mx["rot"])
    o = softmax_attention(q, k, v, mx["scale"], (mx.get("mask") or {}).get("size"))
    return linear(o.reshape(T, H * dv), w, p + "o")


def latent_attention(h, w, p, mx, eps):
    """Keys and values expanded from the latent, head by head."""
    T, H, d, dr, dv, r = (h.shape[0], mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"],
                          mx["kv_rank"])
    q = linear(h, w, p + "q").view(T, H, d + dr)
    down = linear(h, w, p + "dkv")
    c = rms_norm(down[:, :r], w[p + "dkv.norm"], eps)
    shared = rotate_halves(down[:, None, r:], mx["rot"])
    q = torch.cat([q[..., :d], rotate_halves(q[..., d:], mx["rot"])], dim=-1)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, d), shared.expand(T, H, dr)], dim=-1)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    o = softmax_attention(q, k, v, mx["scale"], None, w[p + "sink"])
    return linear(o.reshape(T, H * dv), w, p + "o")


# ----------------------------------------------------------------------- feed-forwards
def dense(h, w, p):
    return linear(silu(linear(h, w, p + "gate")) * linear(h, w, p + "up"), w, p + "down")


def expert(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(GATE_SLOPE * g) * (u + UP_SHIFT)) @ w[p + "down"].T


def mixture(h, w, p, mlp):
    T, E, top = h.shape[0], mlp["router"]["experts"], mlp["router"]["top"]
    z = h @ w[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(T):
        best = sorted(range(E), key=lambda e: (-float(z[t, e]), e))[:top]
        probs = torch.softmax(z[t, best], dim=0)
        for e, pr in zip(best, probs):
            out[t] += pr * expert(h[t:t + 1], w, f"{p}e{e}.", mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        out = out + expert(h, w, p + "shared.", mlp["shared"]["limit"])
    return out


# ----------------------------------------------------------------------- the model
def layer_order(raw) -> List[tuple]:
    """(layer, opens a pass) of every layer run."""
    n, lp = len(raw["layers"]), raw.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    run = list(range(lp["start"], lp["stop"]))
    out = [(i, False) for i in range(lp["start"])]
    for _ in range(lp["times"]):
        out += [(i, i == run[0]) for i in run]
    return out + [(i, False) for i in range(lp["stop"], n)]


def forward(raw: dict, weights: Dict[str, torch.Tensor], tokens: List[int],
            layer_outputs: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = raw["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    x0 = x.clone()
    for i, opens in layer_order(raw):
        entry, p = raw["layers"][i], f"l{i}."
        if opens:
            x = torch.cat([x, x0], dim=-1) @ w["loop.in"].T
        h = tanh_norm(x, w, p + "norm1")
        mx = entry["mixer"]
        if entry["type"] == "attention":
            y = windowed_attention(h, w, p + "mix.", mx)
        else:
            y = latent_attention(h, w, p + "mix.", mx, eps)
        mlp = entry.get("mlp")
        if mlp is not None:
            y = y + (dense(h, w, p + "mlp.") if mlp["kind"] == "dense"
                     else mixture(h, w, p + "mlp.", mlp))
        x = x + y
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return tanh_norm(x, w, "final.norm") @ w["head"].T
