"""A plain, slow implementation of the Pabelix design from its equations: one function per
mechanism, float64 on the CPU, one sequence at a time, attention as whole matrices.  It shares
no code with the engine; the tests hold the engine to it.

Notation: T tokens of one sequence at positions 0..T-1, h [T, width] a sublayer's normed
input, w a dict of float64 tensors by checkpoint name, p the name prefix of the part at hand,
mx a mixer's dict of sizes from the configuration.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


# ----------------------------------------------------------------------- small pieces
def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * (1 + weight): the weight holds the deviation from one."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * (1.0 + weight)


def position_vectors(T: int, width: int):
    """[T, width]: at position p entry 2i is the sine and entry 2i + 1 the cosine of
    p * 10000^(-2i / width)."""
    out = torch.zeros(T, width, dtype=F64)
    for c in range(width):
        f = 10000.0 ** (-(c - c % 2) / width)
        ang = torch.arange(T, dtype=F64) * f
        out[:, c] = torch.sin(ang) if c % 2 == 0 else torch.cos(ang)
    return out


def query_temperature(T: int, temp: Optional[dict]):
    """[T]: 1 + coef ln(floor((p + 1) / every) + 1) at position p."""
    if not temp:
        return torch.ones(T, dtype=F64)
    return torch.tensor([1.0 + temp["coef"] * math.log((p + 1) // temp["every"] + 1)
                         for p in range(T)], dtype=F64)


def softmax_map(q, k, v, scale):
    """One causal attention map of one head: q, k [T, d], v [T, dv]; position i sees j <= i."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    s = s.masked_fill(torch.triu(torch.ones(T, T, dtype=torch.bool), 1), -math.inf)
    return torch.softmax(s, dim=-1) @ v


def mix_weight(w, p: str, diff: float):
    """The one number by which the second map's output counts against the first's."""
    one = torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum())
    two = torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum())
    return one - two + diff


def combine_maps(a1, a2, lam, diff: float, eps: float):
    """a1 - lam a2, divided by its root mean square over the head's values, times 1 - diff."""
    o = a1 - lam * a2
    return o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * (1.0 - diff)


# ------------------------------------------------------------------------------ mixer
def project_kv(h, w, p: str, mx: dict):
    """(k [T, G, 2, dim], v [T, G, vdim]): what a layer keeps of its tokens."""
    T, G = h.shape[0], mx["kv_heads"]
    k = (h @ w[p + "k"].T).view(T, G, 2, mx["dim"])
    v = (h @ w[p + "v"].T).view(T, G, mx["vdim"])
    return k, v


def differential_attention(h, w, p: str, mx: dict, eps: float, kv):
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    k, v = kv
    q = (h @ w[p + "q"].T).view(T, H, 2, d) * query_temperature(T, mx.get("q_temp"))[:, None, None, None]
    lam = mix_weight(w, p, mx["diff"])
    out = torch.zeros(T, H, dv, dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        a1 = softmax_map(q[:, hd, 0], k[:, g, 0], v[:, g], mx["scale"])
        a2 = softmax_map(q[:, hd, 1], k[:, g, 1], v[:, g], mx["scale"])
        out[:, hd] = combine_maps(a1, a2, lam, mx["diff"], eps)
    out = out.reshape(T, H * dv) * torch.sigmoid(h @ w[p + "g"].T)
    return out @ w[p + "o"].T


# ---------------------------------------------------------------------- feed-forward
def clamped_mlp(h, w, p: str, limit: float):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def expert(h, w, p: str):
    z = h @ w[p + "gate"].T
    return (z * torch.sigmoid(z) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p: str, router: dict):
    """(ids [T, top], weights [T, top]): sigmoid scores; a group of neighbours counts by the
    sum of its two largest scores; the weights are the chosen experts' scores as they are."""
    s = torch.sigmoid(h @ w[p + "router"].T)
    choice = s.clone()
    n = s.shape[1]
    groups = router.get("groups")
    if groups and groups["count"] > 1:
        per = n // groups["count"]
        best = s.view(-1, groups["count"], per).topk(min(2, per), dim=-1).values.sum(-1)
        kept = best.topk(groups["keep"], dim=-1).indices
        allowed = torch.zeros_like(best, dtype=torch.bool).scatter_(1, kept, True)
        choice = choice.masked_fill(~allowed.repeat_interleave(per, dim=1), -math.inf)
    ids = choice.topk(router["top"], dim=-1).indices
    return ids, s.gather(1, ids)


def mixture_of_experts(h, w, p: str, mlp: dict):
    ids, wts = route(h, w, p, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t].tolist(), wts[t]):
            out[t] += a * expert(h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


def feed_forward(h, w, p: str, mlp: dict):
    if mlp["kind"] == "dense":
        return clamped_mlp(h, w, p, mlp["limit"])
    return mixture_of_experts(h, w, p, mlp)


# ------------------------------------------------------------------------- the model
def forward(raw: dict, weights: Dict[str, torch.Tensor], tokens: List[int],
            layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one sequence."""
    w = {n: t.to(F64) for n, t in weights.items()}
    eps = raw["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    x = x + position_vectors(len(tokens), raw["width"])
    kept = {}
    for i, layer in enumerate(raw["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        h = rms_norm(x, w[p + "norm1"], eps)
        if mx.get("kv_from") is None:
            kept[i] = project_kv(h, w, p + "mix.", mx)
            kv = kept[i]
        else:
            kv = kept[mx["kv_from"]]
        y = differential_attention(h, w, p + "mix.", mx, eps, kv)
        x = x + rms_norm(y, w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"])
            x = x + rms_norm(y, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T
