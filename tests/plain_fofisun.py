"""A plain, slow statement of the Fofisun decoder: one function per mechanism, float64 on the CPU, whole sequences, no
cache and no batching. It shares no code with ``hi_b200``; the tests hold the engine against it.

A model is ``(config, tensors)``: the dict that config.json holds and a dict name -> float64 tensor.
Notation: T tokens, W the model width; a linear map stored [out, in] acts as ``x @ M.T``.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def rms_norm(x: torch.Tensor, weight: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis, times ``weight``."""
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The model's norm: its weight is stored around zero and acts as 1 + w."""
    return rms_norm(x, 1.0 + w, eps)


def gelu(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


# ----------------------------------------------------------------------------- embedding
def position_vectors(n: int, width: int) -> torch.Tensor:
    """[n, width]: column 2i is sin(p f_i), column 2i + 1 cos(p f_i), f_i = 10000^(-2i / width)."""
    out = torch.zeros(n, width, dtype=F64)
    p = torch.arange(n, dtype=F64)
    for c in range(width):
        f = 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.sin(p * f) if c % 2 == 0 else torch.cos(p * f)
    return out


def embedding(tokens: List[int], w: Dict[str, torch.Tensor]) -> torch.Tensor:
    table = w["embed"]
    return table[torch.tensor(tokens, dtype=torch.long)] + position_vectors(len(tokens), table.shape[1])


# ----------------------------------------------------------------------------- differential attention
def short_convolution(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """u [T, C], taps [C, K]: y_t = sum_j taps[:, j] u_(t - K + 1 + j), zeros before the start."""
    t, k = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(k - 1, u.shape[1], dtype=u.dtype), u])
    y = torch.zeros_like(u)
    for j in range(k):
        y = y + padded[j: j + t] * taps[:, j]
    return y


def visible(t: int, mask: Optional[dict]) -> torch.Tensor:
    """[T, T] bool: query i may read key j."""
    out = torch.zeros(t, t, dtype=torch.bool)
    for i in range(t):
        for j in range(i + 1):
            out[i, j] = mask is None or i - j < mask["size"] or j < mask.get("keep_first", 0)
    return out


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, see: torch.Tensor) -> torch.Tensor:
    """One map: q, k [T, d], v [T, dv]."""
    s = (q @ k.T) * scale
    s = torch.where(see, s, torch.full_like(s, -math.inf))
    p = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return (p / p.sum(dim=-1, keepdim=True)) @ v


def map_factor(m: dict, w: Dict[str, torch.Tensor], pre: str) -> float:
    """What the second map is multiplied by: one number for the layer."""
    one = math.exp(float((w[f"{pre}.lq1"] * w[f"{pre}.lk1"]).sum()))
    two = math.exp(float((w[f"{pre}.lq2"] * w[f"{pre}.lk2"]).sum()))
    return one - two + m["diff"]


def attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], pre: str, eps: float) -> torch.Tensor:
    t, heads, groups, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    u = {n: h @ w[f"{pre}.{n}"].T for n in "qkv"}
    if m.get("conv"):
        u = {n: short_convolution(x, w[f"{pre}.{n}.conv"]) for n, x in u.items()}
    q = rms_norm(u["q"].view(t, heads, 2, dim), w[f"{pre}.q.norm"], eps)
    k = rms_norm(u["k"].view(t, groups, 2, dim), w[f"{pre}.k.norm"], eps)
    v = u["v"].view(t, groups, vdim)
    see, lam = visible(t, m.get("mask")), map_factor(m, w, pre)
    rows = []
    for a in range(heads):
        b = a // (heads // groups)
        a1 = softmax_attention(q[:, a, 0], k[:, b, 0], v[:, b], m["scale"], see)
        a2 = softmax_attention(q[:, a, 1], k[:, b, 1], v[:, b], m["scale"], see)
        rows.append(rms_norm(a1 - lam * a2, None, eps) * (1.0 - m["diff"]))
    gate = torch.sigmoid(h @ w[f"{pre}.g"].T)
    return (torch.cat(rows, dim=-1) * gate) @ w[f"{pre}.o"].T


# ----------------------------------------------------------------------------- feed-forward
def clamped_unit(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[f"{pre}.gate"].T, max=limit)
    u = torch.clamp(h @ w[f"{pre}.up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[f"{pre}.down"].T


def router_choice(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], pre: str):
    """(ids [T, top], logits [T, experts]): the experts with the largest logits."""
    z = h @ w[f"{pre}.router"].T + w[f"{pre}.router.b"]
    return torch.topk(z, mlp["router"]["top"], dim=-1).indices, z


def mixture(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], pre: str, forced_ids=None) -> torch.Tensor:
    ids, z = router_choice(h, mlp, w, pre)
    if forced_ids is not None:
        ids = forced_ids
    chosen = torch.gather(z, 1, ids)
    weight = torch.softmax(chosen, dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for r in range(ids.shape[1]):
            out[t] += weight[t, r] * clamped_unit(h[t: t + 1], w, f"{pre}.e{int(ids[t, r])}", mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        share = torch.sigmoid(h @ w[f"{pre}.shared.sg"].T)
        out = out + share * clamped_unit(h, w, f"{pre}.shared", mlp["shared"]["limit"])
    return out


def feed_forward(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], pre: str, forced_ids=None) -> torch.Tensor:
    if mlp["kind"] == "dense":
        return gelu(h @ w[f"{pre}.up"].T) @ w[f"{pre}.down"].T
    return mixture(h, mlp, w, pre, forced_ids)


# ----------------------------------------------------------------------------- the model
def layer_order(cfg: dict) -> List[int]:
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    order = list(range(loop["start"]))
    for _ in range(loop["times"]):
        order += list(range(loop["start"], loop["stop"]))
    return order + list(range(loop["stop"], n))


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], forced: Optional[dict] = None,
            streams: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab]. ``forced`` {"l<i>.mlp" ("run<n>/l<i>.mlp" for the n-th
    repetition): ids [T, top]} replaces the routers' choices; ``streams`` collects
    the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x = embedding(tokens, w)
    runs: Dict[int, int] = {}
    for i in layer_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}"
        runs[i] = runs.get(i, -1) + 1
        y = attention(layer_norm(x, w[f"{p}.norm1"], eps), layer["mixer"], w, f"{p}.mix", eps)
        x = x + layer_norm(y, w[f"{p}.norm1b"], eps)
        if layer["mlp"] is not None:
            y = feed_forward(layer_norm(x, w[f"{p}.norm2"], eps), layer["mlp"], w, f"{p}.mlp",
                             None if forced is None else forced.get((f"run{runs[i]}/" if runs[i] else "") + f"{p}.mlp"))
            x = x + layer_norm(y, w[f"{p}.norm2b"], eps)
        if streams is not None:
            streams.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T
