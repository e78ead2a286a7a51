"""Small Darotar configurations of the tests and a writer of weights with activations of order one everywhere (fan-in
scaled matrices, norm weights around one, routers with clear choices, sinks of the size of the scores), so that a
mechanism that is left out or misplaced moves the logits."""
from __future__ import annotations

import copy
import math
from typing import Dict, Optional

import torch


def attention(heads, kv_heads, dim, scale, base, dims=None, factor=None, window=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
         "rot": {"base": base, "dims": dim if dims is None else dims}}
    if factor is not None:
        m["rot"]["scaling"] = {"factor": factor}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def config(vocab, width, eps, layers, mult=0.6):
    return {"architecture": "Darotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


# windows shorter than the prompts and no multiple of a page of 16, partial rotation, latents of layer 0 read by two later
# layers with other heads and query sizes, a layer between that has latents of its own, one and several experts a token
DA_A = config(131, 64, 1e-5, [
    latent(4, 16, 8, 12, 24, 20, 0.3, 5000.0, mlp=moe(8, 1, 24)),
    attention(4, 2, 16, 0.2, 1000.0, factor=2.5, window=40, mlp=moe(6, 2, 16)),
    latent(2, 24, 8, 20, 24, 12, 0.25, 5000.0, kv_from=0),
    attention(3, 1, 16, 0.25, 300.0, dims=8, window=23, mlp=moe(4, 1, 32)),
    latent(4, 16, 4, 16, 32, 24, 0.3, 100.0, mlp=moe(5, 3, 16)),
    latent(6, 8, 8, 8, 24, 28, 0.4, 5000.0, kv_from=0, mlp=moe(8, 1, 24)),
])
# rows of 128 and 64 for the tensor-core kernels in bfloat16, more query heads on the shared row than a row tile of 16,
# windows over several key tiles
DA_B = config(200, 128, 1e-6, [
    attention(4, 2, 64, 0.1, 40000.0, factor=8.0, window=150, mlp=moe(4, 1, 64)),
    latent(20, 32, 32, 32, 96, 64, 0.125, 10000.0, mlp=moe(8, 2, 64)),
    attention(2, 1, 128, 0.06, 20000.0, dims=32, window=70, mlp=moe(4, 1, 64)),
    latent(8, 64, 32, 48, 96, 40, 0.1, 10000.0, kv_from=1, mlp=moe(4, 1, 128)),
], mult=0.45)
# what a configuration may leave out: no window, no scaling, no feed-forward, a factor of one; one head of everything
DA_C = config(64, 48, 1e-5, [
    attention(2, 2, 16, 0.3, 700.0),
    latent(1, 8, 8, 8, 16, 16, 0.4, 900.0, mlp=moe(1, 1, 24)),
    attention(1, 1, 24, 0.25, 60.0, dims=2, window=1, mlp=moe(3, 3, 12)),
], mult=1.0)
# sizes that no kernel's wide path takes: width, head sizes, ranks, experts, feed-forward and vocabulary that are no
# multiples of four or sixteen
DA_D = config(77, 51, 3e-4, [
    attention(3, 1, 10, 0.35, 50.0, dims=6, factor=0.5, window=9, mlp=moe(5, 3, 14)),
    latent(3, 7, 6, 5, 18, 11, 0.4, 30.0, mlp=moe(7, 1, 10)),
    latent(5, 9, 6, 11, 18, 13, 0.3, 30.0, kv_from=1, mlp=moe(3, 2, 9)),
    attention(6, 2, 22, 0.2, 80.0, dims=22, window=16),
], mult=0.8)
# rows longer than the tensor-core kernels take, more than eight experts a token
DA_E = config(150, 64, 1e-5, [
    latent(2, 40, 40, 30, 180, 70, 0.15, 2000.0, mlp=moe(12, 9, 8)),
    attention(2, 1, 272, 0.02, 3000.0, dims=100, factor=3.0, window=50, mlp=moe(4, 2, 16)),
    attention(4, 2, 112, 0.06, 3000.0, window=33),
    latent(3, 16, 40, 64, 180, 33, 0.2, 2000.0, kv_from=0, mlp=moe(10, 10, 8)),
])

CONFIGS = {"A": DA_A, "B": DA_B, "C": DA_C, "D": DA_D, "E": DA_E}


def peaked(cfg: dict, factor: float) -> dict:
    """The same model with the scale of every softmax multiplied: nearly all weight then lies on one key, so a key
    that is lost, doubled or shifted shows in the logits."""
    out = copy.deepcopy(cfg)
    for layer in out["layers"]:
        layer["mixer"]["scale"] *= factor
    return out


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """All tensors of a model, float32 values that bfloat16 holds exactly."""
    g = torch.Generator().manual_seed(seed)
    w: Dict[str, torch.Tensor] = {}
    width = cfg["width"]

    def mat(name, rows, cols, gain=1.0):
        w[name] = torch.randn(rows, cols, generator=g) * (gain / math.sqrt(cols))

    def vec(name, n, mean=0.0, std=1.0):
        w[name] = mean + std * torch.randn(n, generator=g)

    w["embed"] = torch.randn(cfg["vocab"], width, generator=g)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}", layer["mixer"], layer["mlp"]
        for n in ("norm1",) + (("norm2",) if mlp else ()):
            vec(f"{p}.{n}", width, 1.0, 0.3)
        if layer["type"] == "attention":
            mat(f"{p}.mix.q", m["heads"] * m["dim"], width, 1.5)
            mat(f"{p}.mix.k", m["kv_heads"] * m["dim"], width, 1.5)
            mat(f"{p}.mix.o", width, m["heads"] * m["dim"], 1.5)
        else:
            mat(f"{p}.mix.dq", m["q_rank"], width, 1.5)
            vec(f"{p}.mix.dq.norm", m["q_rank"], 1.0, 0.3)
            mat(f"{p}.mix.uq", m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.5)
            if m.get("kv_from") is None:
                mat(f"{p}.mix.dkv", m["kv_rank"] + m["rot_dim"], width, 1.5)
                vec(f"{p}.mix.dkv.norm", m["kv_rank"], 1.0, 0.3)
            mat(f"{p}.mix.uk", m["heads"] * m["dim"], m["kv_rank"], 1.5)
            mat(f"{p}.mix.uv", m["heads"] * m["vdim"], m["kv_rank"], 1.5)
            vec(f"{p}.mix.sink", m["heads"], 2.0, 1.5)
            mat(f"{p}.mix.g", m["heads"] * m["vdim"], width, 1.5)
            mat(f"{p}.mix.o", width, m["heads"] * m["vdim"], 1.5)
        if mlp is None:
            continue
        mat(f"{p}.mlp.router", mlp["router"]["experts"], width, 2.0)
        for j in range(mlp["router"]["experts"]):
            mat(f"{p}.mlp.e{j}.gate", mlp["expert"]["ff"], width, 1.5)
            mat(f"{p}.mlp.e{j}.up", mlp["expert"]["ff"], width, 1.5)
            mat(f"{p}.mlp.e{j}.down", width, mlp["expert"]["ff"], 1.5)
    vec("final.norm", width, 1.0, 0.3)
    mat("head", cfg["vocab"], width, 3.0)
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in w.items()}


def write_model(path: str, cfg: dict, seed: int, weights: Optional[Dict[str, torch.Tensor]] = None) -> Dict[str, torch.Tensor]:
    """A model folder (config.json + model.safetensors in bfloat16) with :func:`make_weights` (or the given
    weights); returns the weights."""
    import json
    import os

    from safetensors.torch import save_file

    weights = make_weights(cfg, seed) if weights is None else weights
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return weights


def plain_logits(cfg: dict, weights: Dict[str, torch.Tensor], tokens, forced=None) -> torch.Tensor:
    """Logits [T, vocab] of the plain model in float64."""
    import plain_darotar as plain

    return plain.forward(cfg, {k: v.double() for k, v in weights.items()}, list(tokens), forced=forced)
