"""A decoder assembled from a :class:`ModelSpec`: embedding, a schedule of layers, final norm, head."""
from __future__ import annotations

from typing import Callable, Dict, List, Optional

import torch

from . import attention as _attention  # noqa: F401  (registers the parts)
from . import basic as _basic          # noqa: F401
from . import delta_rule as _delta     # noqa: F401
from . import feed_forward as _ffn     # noqa: F401
from . import gla as _gla              # noqa: F401
from . import latent_attention as _latent  # noqa: F401
from . import mamba2 as _mamba2         # noqa: F401
from . import mlstm as _mlstm          # noqa: F401
from . import pair as _pair            # noqa: F401
from .context import CacheView, StepContext
from .registry import BuildEnv, build
from .spec import CacheSpec, ModelSpec, PartSpec, TensorSpec


class Layer:
    """The parts of one layer, built from its :class:`LayerSpec`."""

    def __init__(self, spec, env: BuildEnv):
        self.spec = spec

        def sub(part_spec):
            name = part_spec.params.get("name")
            return f"{spec.prefix}.{name}" if name else spec.prefix

        self.norm_mixer = build("norm", spec.norm_mixer, env, sub(spec.norm_mixer))
        self.mixer = build("mixer", spec.mixer, env, sub(spec.mixer))
        self.norm_feed_forward = self.feed_forward = None
        if spec.feed_forward is not None:
            if spec.norm_feed_forward is not None:       # None: the block's two sub-layers share one norm
                self.norm_feed_forward = build("norm", spec.norm_feed_forward, env, sub(spec.norm_feed_forward))
            self.feed_forward = build("feed_forward", spec.feed_forward, env, sub(spec.feed_forward))
        arrangement = spec.arrangement if isinstance(spec.arrangement, PartSpec) else PartSpec(spec.arrangement)
        self.arrangement = build("arrangement", arrangement, env, spec.prefix)

    def parts(self):
        """The layer's parts that may hold tensors (the arrangement last: most have none)."""
        parts = [self.norm_mixer, self.mixer, self.norm_feed_forward, self.feed_forward, self.arrangement]
        return [p for p in parts if p is not None]


class Model:
    def __init__(self, spec: ModelSpec, dtype: torch.dtype, device):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype} is not supported (bfloat16 or float32)")
        self.spec, self.dtype, self.device = spec, dtype, torch.device(device)
        self.env = BuildEnv(dtype=dtype, device=self.device, hidden_size=spec.hidden_size)
        self.embedding = build("embedding", spec.embedding, self.env, spec.embedding.params.get("name", ""))
        self.layers = [Layer(ls, self.env) for ls in spec.layers]
        self.final_norm = build("norm", spec.final_norm, self.env, spec.final_norm.params.get("name", ""))
        self.head = build("head", spec.head, self.env, spec.head.params.get("name", ""))
        self.interludes = [build("interlude", ps, self.env, ps.params.get("name", "")) for ps in spec.interludes]
        for i, entry in enumerate(spec.schedule):
            if not 0 <= entry.layer < len(self.layers):
                raise ValueError(f"schedule entry {i} names layer {entry.layer}; the model has {len(self.layers)}")
            if entry.interlude is not None and not 0 <= entry.interlude < len(self.interludes):
                raise ValueError(f"schedule entry {i} names interlude {entry.interlude}; the model has {len(self.interludes)}")
        # cache slots: the spec of the mixer of the first entry that names the slot
        self.cache_specs: Dict[int, Optional[CacheSpec]] = {}
        for entry in spec.schedule:
            cs = self.layers[entry.layer].mixer.cache_spec()
            if entry.cache in self.cache_specs:
                if self.cache_specs[entry.cache] != cs:
                    raise ValueError(f"cache slot {entry.cache} is shared by mixers with different cache needs")
            else:
                self.cache_specs[entry.cache] = cs
        # fixed-size state of a block arrangement (what its layer keeps per request beside the mixer's), by cache slot
        self.block_state_sizes: Dict[int, int] = {}
        for entry in spec.schedule:
            size = int(self.layers[entry.layer].arrangement.state_size())
            if size and entry.writes_cache:
                self.block_state_sizes[entry.cache] = size
        writers = {e.cache for e in spec.schedule if e.writes_cache}
        for slot in self.cache_specs:
            if slot not in writers:
                raise ValueError(f"cache slot {slot} is read but no schedule entry writes it")
        self.loaded = False
        self.graph_safe = all(getattr(p, "graph_safe", False) for p in self.all_parts())

    # ---- weights
    def all_parts(self):
        parts = [self.embedding]
        for layer in self.layers:
            parts += layer.parts()
        return parts + self.interludes + [self.final_norm, self.head]

    def tensor_specs(self) -> List[TensorSpec]:
        specs: List[TensorSpec] = []
        for part in self.all_parts():
            specs += part.tensor_specs()
        return specs

    def load(self, fetch: Callable[[str], Optional[torch.Tensor]]) -> None:
        for part in self.all_parts():
            part.load(fetch)
        self.loaded = True

    # ---- one step
    def forward(self, ctx: StepContext, caches: Dict[int, CacheView], logit_rows: Optional[torch.Tensor]):
        """Run the step's tokens through the schedule; float32 logits [len(logit_rows), V]
        (None when no logits are wanted: the final norm and the head are then skipped)."""
        if not self.loaded:
            raise RuntimeError("model weights are not loaded")
        ctx.scratch = {}
        residual = self.embedding.forward(ctx.tokens, ctx.positions) if getattr(self.embedding, "needs_positions", False) \
            else self.embedding.forward(ctx.tokens)
        if any(getattr(p, "needs_embedding_output", False) for p in self.interludes):
            ctx.scratch["embedding_output"] = residual.clone()       # the stream is summed into in place
        pending, tap, runs = None, ctx.tap, {}
        for entry in self.spec.schedule:
            layer = self.layers[entry.layer]
            # what the parts of a layer report from its second run on carries the run's number
            n = runs[entry.layer] = runs.get(entry.layer, -1) + 1
            ctx.run_prefix = f"run{n}/" if n else ""
            if tap is not None:
                ctx.tap = tap if not n else (lambda name, t, prefix=ctx.run_prefix: tap(prefix + name, t))
            view = caches[entry.cache]
            if view.writes != entry.writes_cache:
                view = CacheView(group=view.group, k_pages=view.k_pages, v_pages=view.v_pages, state=view.state,
                                 writes=entry.writes_cache, slot=view.slot, block_state=view.block_state)
            if entry.interlude is not None:
                residual, pending = self.interludes[entry.interlude].forward(residual, pending, ctx, entry.interlude_arg)
            residual, pending = layer.arrangement.forward(layer, residual, pending, ctx, view)
        ctx.tap, ctx.run_prefix = tap, ""
        if logit_rows is None or logit_rows.numel() == 0:
            return None
        z = self.final_norm.forward(residual, pending, logit_rows)
        return self.head.forward(z, self.embedding)
