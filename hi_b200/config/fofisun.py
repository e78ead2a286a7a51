"""Typed configuration of the Fofisun decoder: a norm before and after every sub-layer, differential attention behind short
convolutions, a dense or a mixture-of-experts feed-forward, and a range of layers that may run several times.

config.json keys: ``architecture`` ("Fofisun"), ``vocab``, ``width``, ``norm.eps``, optionally ``loop`` =
``{start, stop, times}`` (layers start .. stop - 1 run ``times`` times in a row), and ``layers``: a list of
``{"type": "attention", "mixer": {...}, "mlp": {...} | null}``.

Mixer keys: ``heads, kv_heads, dim, vdim``, ``diff`` (the constant of the second map's factor), ``scale`` (of the scores),
``conv`` (taps; optional), ``mask`` = ``{size, keep_first?}`` (optional: a query reads itself, the ``size - 1`` tokens
before it and the first ``keep_first`` of the sequence).
mlp keys: ``kind`` = "dense": ``ff``; "moe": ``router`` = ``{experts, top}``, ``expert`` = ``{ff, limit}``, optional
``shared`` = ``{ff, limit}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, get_key, token_ids


@dataclass(frozen=True)
class FofisunAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    diff: float
    scale: float
    conv: Optional[int] = None
    window: Optional[int] = None
    keep_first: int = 0


@dataclass(frozen=True)
class FofisunDense:
    ff: int


@dataclass(frozen=True)
class FofisunMoe:
    experts: int
    top: int
    ff: int
    limit: float
    shared_ff: Optional[int] = None
    shared_limit: Optional[float] = None


@dataclass(frozen=True)
class FofisunLayer:
    mixer: FofisunAttention
    mlp: Any                          # FofisunDense | FofisunMoe | None


@dataclass(frozen=True)
class FofisunLoop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class FofisunConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[FofisunLayer, ...]
    loop: Optional[FofisunLoop] = None
    eos_token_ids: Tuple[int, ...] = ()
    architectures: Tuple[str, ...] = ("Fofisun",)

    @staticmethod
    def from_json(raw: Dict[str, Any], generation: Optional[Dict[str, Any]] = None) -> "FofisunConfig":
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

        def unit(parent, where):
            (ff,) = sizes(parent, ("ff",), where)
            limit = need(parent, "limit", float, where)
            if not limit > 0:
                raise ConfigError(f"config.json: {where}.limit must be positive")
            return ff, limit

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
            if entry.get("type") != "attention":
                raise ConfigError(f"config.json: {where}.type is {entry.get('type')!r}; known mixers: ('attention',)")
            m, mw = entry["mixer"], f"{where}.mixer"
            heads, kv_heads, dim, vdim = sizes(m, ("heads", "kv_heads", "dim", "vdim"), mw)
            if heads % kv_heads:
                raise ConfigError(f"config.json: {mw}: heads must be a multiple of kv_heads")
            conv = get_key(m, "conv", int)
            if conv is not None and conv < 1:
                raise ConfigError(f"config.json: {mw}.conv must be at least one tap")
            scale = get_key(m, "scale", float)
            mask, window, keep = obj(m, "mask", f"{mw}.mask", required=False), None, 0
            if mask:
                (window,) = sizes(mask, ("size",), f"{mw}.mask")
                keep = get_key(mask, "keep_first", int, default=0)
                if keep < 0:
                    raise ConfigError(f"config.json: {mw}.mask.keep_first must not be negative")
            mixer = FofisunAttention(heads, kv_heads, dim, vdim, need(m, "diff", float, mw),
                                     dim ** -0.5 if scale is None else scale, conv, window, keep)
            mlp_raw, mlp, lw = entry.get("mlp"), None, f"{where}.mlp"
            if mlp_raw is not None:
                if not isinstance(mlp_raw, dict) or mlp_raw.get("kind") not in ("dense", "moe"):
                    raise ConfigError(f"config.json: {lw}.kind must be 'dense' or 'moe' (or mlp null)")
                if mlp_raw["kind"] == "dense":
                    mlp = FofisunDense(*sizes(mlp_raw, ("ff",), lw))
                else:
                    experts, top = sizes(obj(mlp_raw, "router", f"{lw}.router"), ("experts", "top"), f"{lw}.router")
                    if top > experts:
                        raise ConfigError(f"config.json: {lw}.router.top is larger than the number of experts")
                    ff, limit = unit(obj(mlp_raw, "expert", f"{lw}.expert"), f"{lw}.expert")
                    shared = obj(mlp_raw, "shared", f"{lw}.shared", required=False)
                    shared_ff, shared_limit = unit(shared, f"{lw}.shared") if shared else (None, None)
                    mlp = FofisunMoe(experts, top, ff, limit, shared_ff, shared_limit)
            layers.append(FofisunLayer(mixer, mlp))
        loop_raw, loop = obj(raw, "loop", "loop", required=False), None
        if loop_raw:
            start, stop, times = (need(loop_raw, k, int, "loop") for k in ("start", "stop", "times"))
            if not 0 <= start < stop <= len(layers) or times < 1:
                raise ConfigError("config.json: loop needs 0 <= start < stop <= number of layers and times >= 1")
            loop = FofisunLoop(start, stop, times)
        eos = token_ids(raw, "eos_token_id") or (token_ids(generation, "eos_token_id") if generation else [])
        return FofisunConfig(vocab=vocab, width=width, eps=eps, layers=tuple(layers), loop=loop, eos_token_ids=tuple(eos))
