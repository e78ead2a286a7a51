"""Typed configuration of the Darotar decoder: a norm on every sub-layer's output only, two kinds of mixer (windowed
attention whose values are its keys, and latent attention with a learned sink, an output gate and latents that layers may
share), and routed experts as feed-forward.

config.json keys: ``architecture`` ("Darotar"), ``vocab``, ``width``, ``norm.eps``, ``residual_mult`` (default 1), and
``layers``: a list of ``{"type": "attention" | "latent_attention", "mixer": {...}, "mlp": {...} | null}``.

Mixer keys.
  attention         ``heads, kv_heads, dim, vdim`` (``vdim`` = ``dim``: the values are the projected keys), ``scale``,
                    ``rot`` = ``{base, dims, scaling?}`` with ``scaling`` = ``{factor}``, ``mask.size`` (optional: a query
                    reads itself and the ``size - 1`` tokens before it)
  latent_attention  ``heads, dim, rot_dim, vdim, kv_rank, q_rank, scale``, ``rot`` (``rot.dims`` = ``rot_dim``), optional
                    ``kv_from`` (an earlier latent_attention layer whose latents this one reads)
mlp keys: ``kind`` ("moe"), ``router`` = ``{experts, top}``, ``expert`` = ``{ff}``.

Where ``q_rank`` is absent, the checkpoint's ``l<i>.mix.dq`` [q_rank, width] gives it (:func:`sizes_from_tensors`).
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, get_key, token_ids

MIXERS = ("attention", "latent_attention")


@dataclass(frozen=True)
class DarotarRotation:
    base: float
    dims: int
    factor: Optional[float] = None       # every frequency is divided by it


@dataclass(frozen=True)
class DarotarAttention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot: DarotarRotation
    window: Optional[int] = None


@dataclass(frozen=True)
class DarotarLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: DarotarRotation
    q_rank: Optional[int] = None
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class DarotarMoe:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class DarotarLayer:
    kind: str
    mixer: Any                        # DarotarAttention | DarotarLatent
    mlp: Optional[DarotarMoe]         # None: the layer has no feed-forward


@dataclass(frozen=True)
class DarotarConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[DarotarLayer, ...]
    residual_mult: float = 1.0
    eos_token_ids: Tuple[int, ...] = ()
    architectures: Tuple[str, ...] = ("Darotar",)

    @staticmethod
    def from_json(raw: Dict[str, Any], generation: Optional[Dict[str, Any]] = None) -> "DarotarConfig":
        def obj(parent, key, where, required=True):
            value = parent.get(key)
            if value is None and not required:
                return None
            if not isinstance(value, dict):
                raise ConfigError(f"config.json: required key '{where}' is missing or not an object")
            return value

        def need(parent, key, typ, where):
            try:
                return get_key(parent, key, typ, required=True)
            except ConfigError as e:
                raise ConfigError(str(e).replace("key '", f"key '{where}.")) from None

        def sizes(parent, keys, where):
            values = [need(parent, k, int, where) for k in keys]
            if min(values) <= 0:
                raise ConfigError(f"config.json: {where}: {', '.join(keys)} must be positive")
            return values

        def rotation(parent, where, head_dim):
            r, rw = obj(parent, "rot", f"{where}.rot"), f"{where}.rot"
            base, dims = need(r, "base", float, rw), need(r, "dims", int, rw)
            if dims <= 0 or dims % 2 or dims > head_dim or not base > 0.0:
                raise ConfigError(f"config.json: {rw}.dims must be even and at most {head_dim}, base positive")
            scaling, factor = obj(r, "scaling", f"{rw}.scaling", required=False), None
            if scaling:
                factor = need(scaling, "factor", float, f"{rw}.scaling")
                if not factor > 0:
                    raise ConfigError(f"config.json: {rw}.scaling.factor must be positive")
            return DarotarRotation(base, dims, factor)

        def attention(m, where):
            heads, kv_heads, dim = sizes(m, ("heads", "kv_heads", "dim"), where)
            if heads % kv_heads:
                raise ConfigError(f"config.json: {where}: heads must be a multiple of kv_heads")
            if get_key(m, "vdim", int, default=dim) != dim:
                raise ConfigError(f"config.json: {where}.vdim must equal dim (the values are the keys)")
            mask, window = obj(m, "mask", f"{where}.mask", required=False), None
            if mask:
                (window,) = sizes(mask, ("size",), f"{where}.mask")
            return DarotarAttention(heads, kv_heads, dim, need(m, "scale", float, where), rotation(m, where, dim), window)

        def latent(m, where, i, layers):
            heads, dim, rot_dim, vdim, kv_rank = sizes(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank"), where)
            q_rank = get_key(m, "q_rank", int)
            if q_rank is not None and q_rank < 1:
                raise ConfigError(f"config.json: {where}.q_rank must be positive")
            rot = rotation(m, where, rot_dim)
            if rot.dims != rot_dim:
                raise ConfigError(f"config.json: {where}.rot.dims must equal rot_dim (the whole rotated part turns)")
            kv_from = get_key(m, "kv_from", int)
            mixer = DarotarLatent(heads, dim, rot_dim, vdim, kv_rank, need(m, "scale", float, where), rot, q_rank, kv_from)
            if kv_from is not None:
                source = layers[kv_from] if 0 <= kv_from < i else None
                if source is None or source.kind != "latent_attention" or source.mixer.kv_from is not None:
                    raise ConfigError(f"config.json: {where}.kv_from must name an earlier latent_attention layer with latents of its own")
                if (source.mixer.kv_rank, source.mixer.rot_dim, source.mixer.rot) != (kv_rank, rot_dim, rot):
                    raise ConfigError(f"config.json: {where}.kv_from: kv_rank, rot_dim and rot must equal those of layer {kv_from}")
            return mixer

        def experts(mlp, where):
            if mlp is None:
                return None
            if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
                raise ConfigError(f"config.json: {where}.kind must be 'moe' (or mlp null)")
            n, top = sizes(obj(mlp, "router", f"{where}.router"), ("experts", "top"), f"{where}.router")
            if top > n:
                raise ConfigError(f"config.json: {where}.router.top is larger than the number of experts")
            (ff,) = sizes(obj(mlp, "expert", f"{where}.expert"), ("ff",), f"{where}.expert")
            return DarotarMoe(n, top, ff)

        vocab = get_key(raw, "vocab", int, required=True)
        width = get_key(raw, "width", int, required=True)
        if vocab <= 0 or width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        eps = need(obj(raw, "norm", "norm"), "eps", float, "norm")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]"
            if not isinstance(entry, dict) or not isinstance(entry.get("mixer"), dict):
                raise ConfigError(f"config.json: {where} needs 'type' and a 'mixer' object")
            kind = entry.get("type")
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}.type is {kind!r}; known mixers: {MIXERS}")
            m, mw = entry["mixer"], f"{where}.mixer"
            mixer = attention(m, mw) if kind == "attention" else latent(m, mw, i, layers)
            layers.append(DarotarLayer(kind, mixer, experts(entry.get("mlp"), f"{where}.mlp")))
        eos = token_ids(raw, "eos_token_id") or (token_ids(generation, "eos_token_id") if generation else [])
        return DarotarConfig(vocab=vocab, width=width, eps=eps, layers=tuple(layers),
                             residual_mult=get_key(raw, "residual_mult", float, default=1.0), eos_token_ids=tuple(eos))


def sizes_from_tensors(cfg: DarotarConfig, shapes: Dict[str, tuple]) -> DarotarConfig:
    """The query latents' sizes that config.json does not hold, read off ``l<i>.mix.dq`` ([q_rank, width])."""
    layers = list(cfg.layers)
    for i, layer in enumerate(layers):
        dq = shapes.get(f"l{i}.mix.dq")
        if layer.kind == "latent_attention" and layer.mixer.q_rank is None and dq:
            layers[i] = replace(layer, mixer=replace(layer.mixer, q_rank=int(dq[0])))
    return replace(cfg, layers=tuple(layers))
