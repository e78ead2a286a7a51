"""Small Fofisun configurations of the tests and a writer of weights with activations of order one everywhere (fan-in
scaled matrices, norm weights around zero as the model stores them, routers with clear choices, a second map that
matters), so that a mechanism that is left out or misplaced moves the logits."""
from __future__ import annotations

import copy
import math
from typing import Dict, Optional

import torch


def attention(heads, kv_heads, dim, vdim, scale, diff, conv=None, window=None, keep=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if conv is not None:
        m["conv"] = conv
    if window is not None:
        m["mask"] = {"size": window}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    return {"type": "attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, shared=None, shared_limit=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared is not None:
        m["shared"] = {"ff": shared, "limit": limit if shared_limit is None else shared_limit}
    return m


def config(vocab, width, eps, layers, loop=None):
    cfg = {"architecture": "Fofisun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# windows shorter than the prompts with kept first tokens (fewer and more than a page of 16), both feed-forwards, two
# layers that run twice
FO_A = config(131, 64, 1e-5, [
    attention(4, 2, 16, 24, 0.3, 0.2, conv=3, window=40, keep=5, mlp=dense(96)),
    attention(2, 1, 16, 32, 0.3, 0.4, conv=4, window=23, keep=19, mlp=moe(8, 2, 24, 1.2, shared=32, shared_limit=0.9)),
    attention(4, 2, 16, 24, 0.3, 0.2, conv=3, window=40, keep=5, mlp=moe(6, 3, 16, 0.8)),
    attention(3, 3, 8, 16, 0.5, 0.6, conv=2, mlp=dense(40)),
], loop=(1, 3, 2))
# rows of 128 for the tensor-core kernels in bfloat16, many query heads on one key head (more than a row tile of 16 by
# two maps), windows over several key tiles, kept tokens over more than one of them
FO_B = config(200, 128, 1e-6, [
    attention(4, 2, 64, 128, 0.125, 0.35, conv=4, window=150, keep=70, mlp=moe(4, 1, 64, 2.0, shared=48, shared_limit=1.5)),
    attention(12, 1, 32, 64, 0.2, 0.5, conv=4, window=97, keep=1, mlp=dense(128)),
    attention(2, 1, 64, 64, 0.125, 0.3, conv=4, mlp=moe(4, 2, 64, 1.0)),
])
# what a configuration may leave out: no window, no kept tokens, no convolution, no feed-forward, no shared expert, no loop
FO_C = config(64, 48, 1e-5, [
    attention(3, 1, 8, 12, 0.4, 0.1, mlp=moe(3, 3, 20, 1.0)),
    attention(2, 2, 16, 16, 0.25, 0.7, conv=1, window=30),
    attention(1, 1, 24, 8, 0.3, 0.0, conv=4, window=12, keep=0, mlp=dense(30)),
])
# sizes that no kernel's wide path takes: width, head sizes, experts, feed-forward and vocabulary that are no multiples
# of four or sixteen, value heads of another size than two key maps, five taps, a window of one page and of one token,
# kept tokens beyond the whole prompt, a loop over the first layer alone
FO_D = config(77, 51, 1e-5, [
    attention(3, 1, 10, 6, 0.4, 0.25, conv=5, window=16, keep=3, mlp=moe(5, 3, 14, 1.1, shared=10, shared_limit=0.7)),
    attention(6, 2, 6, 22, 0.5, 0.15, conv=2, window=1, keep=2, mlp=dense(33)),
    attention(2, 2, 7, 9, 0.5, 0.55, conv=3, window=9, keep=500, mlp=moe(7, 1, 10, 0.6, shared=22)),
], loop=(0, 1, 3))
# rows longer than the tensor-core kernels take, more than eight experts a token, a loop over every layer
FO_E = config(150, 64, 3e-4, [
    attention(2, 1, 112, 40, 0.1, 0.3, conv=4, window=50, keep=20, mlp=moe(12, 9, 8, 1.3, shared=16)),
    attention(2, 2, 20, 300, 0.25, 0.45, conv=4, window=33, keep=4, mlp=dense(64)),
], loop=(0, 2, 2))

CONFIGS = {"A": FO_A, "B": FO_B, "C": FO_C, "D": FO_D, "E": FO_E}


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

    def unit(name, ff):
        mat(name + ".gate", ff, width, 1.5)
        mat(name + ".up", ff, width, 1.5)
        mat(name + ".down", width, ff, 1.5)

    w["embed"] = torch.randn(cfg["vocab"], width, generator=g)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}", layer["mixer"], layer["mlp"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp else ()):
            vec(f"{p}.{n}", width, 0.0, 0.3)
        rows = {"q": m["heads"] * 2 * m["dim"], "k": m["kv_heads"] * 2 * m["dim"], "v": m["kv_heads"] * m["vdim"]}
        for n, r in rows.items():
            mat(f"{p}.mix.{n}", r, width, 1.5)
            if m.get("conv"):
                w[f"{p}.mix.{n}.conv"] = 0.6 * torch.randn(r, m["conv"], generator=g)
        vec(f"{p}.mix.q.norm", m["dim"], 1.0, 0.4)
        vec(f"{p}.mix.k.norm", m["dim"], 1.0, 0.4)
        for n in ("lq1", "lk1", "lq2", "lk2"):
            vec(f"{p}.mix.{n}", m["dim"], 0.0, 0.5 / math.sqrt(m["dim"]))
        mat(f"{p}.mix.g", m["heads"] * m["vdim"], width, 1.5)
        mat(f"{p}.mix.o", width, m["heads"] * m["vdim"], 2.0)
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            mat(f"{p}.mlp.up", mlp["ff"], width, 1.5)
            mat(f"{p}.mlp.down", width, mlp["ff"], 1.5)
            continue
        mat(f"{p}.mlp.router", mlp["router"]["experts"], width, 2.0)
        vec(f"{p}.mlp.router.b", mlp["router"]["experts"], 0.0, 1.0)
        for j in range(mlp["router"]["experts"]):
            unit(f"{p}.mlp.e{j}", mlp["expert"]["ff"])
        if mlp.get("shared"):
            unit(f"{p}.mlp.shared", mlp["shared"]["ff"])
            mat(f"{p}.mlp.shared.sg", 1, width, 1.5)
    vec("final.norm", width, 0.0, 0.3)
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
    import plain_fofisun as plain

    return plain.forward(cfg, {k: v.double() for k, v in weights.items()}, list(tokens), forced=forced)
