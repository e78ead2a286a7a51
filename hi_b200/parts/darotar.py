"""Darotar as data: its configuration turned into a ModelSpec of registered parts.

Every layer is a ``normed_output`` block (the sub-layers read the stream itself; an RMS norm and a constant factor on what
they return). The mixer is ``attention`` whose values are the projected keys (interleaved rotation with a linear scaling,
a weightless norm of q and k after it, a sliding window) or ``latent_attention`` (query latent, shared rotated key part,
learned sink, an output gate per element); a latent layer with ``kv_from`` reads the cache slot of the layer it names. The
feed-forward is ``routed_experts`` with sigmoid scores on the experts' inputs.
Checkpoint names: ``embed``, ``head``, ``final.norm``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.router``,
``l<i>.mlp.e<j>.{gate,up,down}``.
"""
from __future__ import annotations

from typing import Optional

from ..config.darotar import DarotarConfig
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _scaling(rot) -> Optional[dict]:
    return None if rot.factor is None else {"factor": rot.factor}


def _mixer(cfg: DarotarConfig, layer) -> PartSpec:
    m, w, eps = layer.mixer, cfg.width, cfg.eps
    if layer.kind == "attention":
        rope = PartSpec("rope", {"head_dim": m.dim, "theta": m.rot.base, "rot_dim": m.rot.dims, "interleaved": True,
                                 "exact": True, "scaling": _scaling(m.rot)})
        return PartSpec("attention", {
            "name": "mix", "hidden_size": w, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
            "window": ("sliding", m.window) if m.window else None, "position": rope, "qk_norm": True, "qk_norm_eps": eps,
            "scale": m.scale, "names": "short", "values": "keys"})
    if m.q_rank is None:
        raise ValueError("latent_attention: q_rank is neither in config.json nor in the checkpoint's shapes")
    return PartSpec("latent_attention", {
        "name": "mix", "hidden_size": w, "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
        "q_rank": m.q_rank, "rot_dim": m.rot_dim, "rot_base": m.rot.base, "rot_scaling": _scaling(m.rot), "scale": m.scale,
        "eps": eps, "own_latents": m.kv_from is None, "gate": "element", "sink": True})


def build_darotar_spec(cfg: DarotarConfig) -> ModelSpec:
    w = cfg.width

    def norm(name):
        return PartSpec("rmsnorm", {"name": name, "size": w, "eps": cfg.eps, "tensor": "bare"})

    layers, schedule = [], []
    for i, l in enumerate(cfg.layers):
        source = getattr(l.mixer, "kv_from", None)
        schedule.append(ScheduleEntry(layer=i, cache=i if source is None else source, writes_cache=source is None))
        ffn = None if l.mlp is None else PartSpec("routed_experts", {
            "name": "mlp", "hidden_size": w, "num_experts": l.mlp.experts, "top_k": l.mlp.top, "intermediate_size": l.mlp.ff,
            "shared_expert": False, "score": "sigmoid", "renormalize": False, "scale": "input", "names": "per_expert"})
        layers.append(LayerSpec(prefix=f"l{i}", mixer=_mixer(cfg, l), feed_forward=ffn, norm_mixer=norm("norm1"),
                                norm_feed_forward=norm("norm2") if ffn is not None else None,
                                arrangement=PartSpec("normed_output", {"mult": cfg.residual_mult})))
    return ModelSpec(
        hidden_size=w, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"name": "embed", "vocab_size": cfg.vocab, "hidden_size": w}),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"name": "head", "vocab_size": cfg.vocab, "hidden_size": w, "tensor": "head"}),
        eos_token_ids=cfg.eos_token_ids, max_position_embeddings=None)


def normalize_darotar_tensor_name(name: str) -> Optional[str]:
    """The parts ask for the checkpoint's own names, but for the embedding table (``embed`` is the
    token-embedding part's ``embed.weight``)."""
    return "embed.weight" if name == "embed" else name
