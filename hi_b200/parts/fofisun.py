"""Fofisun as data: its configuration turned into a ModelSpec of registered parts.

Every layer is a ``sandwich`` block (an RMS norm, its weight stored around zero, before and after each sub-layer). The
mixer is ``attention`` with two maps a head over the same values (differential attention), short convolutions on q, k and
v, weighted q/k norms, no rotation, a sliding window that keeps the first tokens, and an output gate. The feed-forward is
``dense_mlp`` with the exact gelu or ``routed_experts`` with clamped units, a router bias, weights that are the softmax
over the chosen logits, and a gated shared expert. The embedding adds a sinusoidal vector of the position. A range of
layers may run several times: every run is a schedule entry with a cache slot of its own.
Checkpoint names: ``embed``, ``head``, ``final.norm``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

from typing import Optional

from ..config.fofisun import FofisunConfig, FofisunDense
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

SINUSOID_BASE = 10000.0


def _feed_forward(w: int, mlp) -> Optional[PartSpec]:
    if mlp is None:
        return None
    if isinstance(mlp, FofisunDense):
        return PartSpec("dense_mlp", {"name": "mlp", "hidden_size": w, "intermediate_size": mlp.ff, "activation": "gelu"})
    return PartSpec("routed_experts", {
        "name": "mlp", "hidden_size": w, "num_experts": mlp.experts, "top_k": mlp.top, "intermediate_size": mlp.ff,
        "activation": "clamped", "limit": mlp.limit, "score": "softmax", "renormalize": True, "scale": "output",
        "router_bias": True, "names": "per_expert", "shared_expert": mlp.shared_ff is not None,
        "shared_intermediate_size": mlp.shared_ff, "shared_limit": mlp.shared_limit,
        "shared_gate": mlp.shared_ff is not None})


def build_fofisun_spec(cfg: FofisunConfig) -> ModelSpec:
    w = cfg.width

    def norm(name):
        return PartSpec("rmsnorm", {"name": name, "size": w, "eps": cfg.eps, "tensor": "bare", "one_plus": True})

    layers = []
    for i, l in enumerate(cfg.layers):
        m, ffn = l.mixer, _feed_forward(w, l.mlp)
        window = None if m.window is None else ("sliding", m.window, m.keep_first)
        mixer = PartSpec("attention", {
            "name": "mix", "hidden_size": w, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
            "value_dim": m.vdim, "window": window, "qk_norm_weighted": True, "qk_norm_eps": cfg.eps, "scale": m.scale,
            "names": "short", "conv": m.conv, "differential": m.diff, "output_gate": True})
        block = PartSpec("sandwich", {"hidden_size": w, "eps": cfg.eps, "one_plus": True, "feed_forward": ffn is not None})
        layers.append(LayerSpec(prefix=f"l{i}", mixer=mixer, feed_forward=ffn, norm_mixer=norm("norm1"),
                                norm_feed_forward=norm("norm2") if ffn is not None else None, arrangement=block))
    order = list(range(len(layers)))
    if cfg.loop is not None:
        lo, hi = cfg.loop.start, cfg.loop.stop
        order = order[:lo] + order[lo:hi] * cfg.loop.times + order[hi:]
    return ModelSpec(
        hidden_size=w, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"name": "embed", "vocab_size": cfg.vocab, "hidden_size": w,
                                               "sinusoid": SINUSOID_BASE}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(layer=l, cache=run) for run, l in enumerate(order)),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"name": "head", "vocab_size": cfg.vocab, "hidden_size": w, "tensor": "head"}),
        eos_token_ids=cfg.eos_token_ids, max_position_embeddings=None)


def normalize_fofisun_tensor_name(name: str) -> Optional[str]:
    """The parts ask for the checkpoint's own names, but for the embedding table (``embed`` is the
    token-embedding part's ``embed.weight``)."""
    return "embed.weight" if name == "embed" else name
