"""A plain, slow statement of the Darotar decoder: one function per mechanism, float64 on the CPU, whole sequences, no
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


# ----------------------------------------------------------------------------- rotation
def frequencies(rot: dict) -> List[float]:
    """base^(-2i / dims) of every pair, divided by the factor of a linear scaling where there is one."""
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    return [rot["base"] ** (-2.0 * i / rot["dims"]) / factor for i in range(rot["dims"] // 2)]


def rotate(x: torch.Tensor, rot: dict, neighbours: bool) -> torch.Tensor:
    """x [T, heads, d], row t at position t: the first ``dims`` dims turn in pairs, (2i, 2i + 1) with ``neighbours``,
    else (i, i + dims/2); the others pass."""
    y, dims = x.clone(), rot["dims"]
    p = torch.arange(x.shape[0], dtype=x.dtype)[:, None]
    for i, f in enumerate(frequencies(rot)):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + dims // 2)
        u, v = x[..., a], x[..., b]
        y[..., a] = u * torch.cos(p * f) - v * torch.sin(p * f)
        y[..., b] = v * torch.cos(p * f) + u * torch.sin(p * f)
    return y


# ----------------------------------------------------------------------------- softmax
def visible(t: int, window: Optional[int]) -> torch.Tensor:
    """[T, T] bool: query i may read key j."""
    out = torch.zeros(t, t, dtype=torch.bool)
    for i in range(t):
        for j in range(i + 1):
            out[i, j] = window is None or i - j < window
    return out


def softmax_weights(scores: torch.Tensor, see: torch.Tensor, sink: Optional[float] = None) -> torch.Tensor:
    """exp(score) over their sum and exp(``sink``)."""
    s = torch.where(see, scores, torch.full_like(scores, -math.inf))
    top = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=sink)
    e = torch.exp(s - top)
    total = e.sum(dim=-1, keepdim=True)
    return e / (total if sink is None else total + torch.exp(sink - top))


# ----------------------------------------------------------------------------- mixers
def attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], pre: str, eps: float) -> torch.Tensor:
    """Keys and values are one projection: the key is normed after its rotation, the value is the projection itself."""
    t, heads, groups, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[f"{pre}.q"].T).view(t, heads, dim)
    v = (h @ w[f"{pre}.k"].T).view(t, groups, dim)
    q = rms_norm(rotate(q, m["rot"], True), None, eps)
    k = rms_norm(rotate(v, m["rot"], True), None, eps)
    see = visible(t, (m.get("mask") or {}).get("size"))
    rows = []
    for a in range(heads):
        b = a // (heads // groups)
        rows.append(softmax_weights((q[:, a] @ k[:, b].T) * m["scale"], see) @ v[:, b])
    return torch.cat(rows, dim=-1) @ w[f"{pre}.o"].T


def latents(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], pre: str, eps: float):
    """(latent [T, rank], rotated key part [T, rot_dim]) of every token."""
    y = h @ w[f"{pre}.dkv"].T
    c = rms_norm(y[:, : m["kv_rank"]], w[f"{pre}.dkv.norm"], eps)
    return c, rotate(y[:, None, m["kv_rank"]:], m["rot"], False)[:, 0]


def latent_attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], pre: str, eps: float, rows) -> torch.Tensor:
    """``rows``: this layer's or another layer's :func:`latents`."""
    t, heads, dim, rot_dim, vdim = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, k_rot = rows
    q = (rms_norm(h @ w[f"{pre}.dq"].T, w[f"{pre}.dq.norm"], eps) @ w[f"{pre}.uq"].T).view(t, heads, dim + rot_dim)
    q_rot = rotate(q[:, :, dim:], m["rot"], False)
    k = (c @ w[f"{pre}.uk"].T).view(t, heads, dim)
    v = (c @ w[f"{pre}.uv"].T).view(t, heads, vdim)
    see, out = visible(t, None), []
    for a in range(heads):
        s = (q[:, a, :dim] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"]
        out.append(softmax_weights(s, see, w[f"{pre}.sink"][a]) @ v[:, a])
    return (torch.cat(out, dim=-1) * torch.sigmoid(h @ w[f"{pre}.g"].T)) @ w[f"{pre}.o"].T


# ----------------------------------------------------------------------------- feed-forward
def silu_unit(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str) -> torch.Tensor:
    g = h @ w[f"{pre}.gate"].T
    return (g * torch.sigmoid(g) * (h @ w[f"{pre}.up"].T)) @ w[f"{pre}.down"].T


def router_choice(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], pre: str):
    """(ids [T, top], scores [T, experts]): the experts with the largest scores."""
    s = torch.sigmoid(h @ w[f"{pre}.router"].T)
    return torch.topk(s, mlp["router"]["top"], dim=-1).indices, s


def mixture(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], pre: str, forced_ids=None) -> torch.Tensor:
    """A chosen expert's score multiplies what the expert reads."""
    ids, s = router_choice(h, mlp, w, pre)
    if forced_ids is not None:
        ids = forced_ids
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in ids[t].tolist():
            out[t] += silu_unit(s[t, e] * h[t: t + 1], w, f"{pre}.e{e}")[0]
    return out


# ----------------------------------------------------------------------------- the model
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], forced: Optional[dict] = None,
            streams: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab]. ``forced`` {"l<i>.mlp": ids [T, top]} replaces the routers' choices; ``streams`` collects
    the residual stream after every layer."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        if layer["type"] == "attention":
            y = attention(x, m, w, f"{p}.mix", eps)
        else:
            if m.get("kv_from") is None:
                kept[i] = latents(x, m, w, f"{p}.mix", eps)
            y = latent_attention(x, m, w, f"{p}.mix", eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        x = x + mult * rms_norm(y, w[f"{p}.norm1"], eps)
        if layer["mlp"] is not None:
            y = mixture(x, layer["mlp"], w, f"{p}.mlp", None if forced is None else forced.get(f"{p}.mlp"))
            x = x + mult * rms_norm(y, w[f"{p}.norm2"], eps)
        if streams is not None:
            streams.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
