"""The attention mixer: grouped-query attention over a paged cache, global or windowed."""
from __future__ import annotations

from typing import Optional

import numpy as np
import torch

from ..kernels import ops
from .basic import Part
from .linear import linear
from .registry import build, register
from .spec import CacheSpec, PartSpec, TensorSpec


DIFF_TC_MIN_TOKENS = 64      # new tokens of a request from which differential attention takes the tcgen05 kernel (its
                             # tile is 64 tokens by two maps)


def _key_splits(ctx, nh: int, chunk: int, sliding: int, single: bool, device) -> int:
    """Portions far into long contexts on a layer that sees every key: all blocks of the
    tensor-core prefill kernel then have about the same many key tiles, and a partly filled
    last round of blocks is worth splitting the keys for (ops.prefill_key_splits)."""
    if chunk or sliding:
        return 1
    portions = [(s, n) for s, n in zip(ctx.start_pos, ctx.n_new) if n > 1 or not single]
    if not portions:
        return 1
    shortest, longest_new = min(s for s, _n in portions), max(n for _s, n in portions)
    if shortest < 2 * longest_new:
        return 1
    blocks = nh * sum(-(-n // ops.PREFILL_TC_MIN_TOKENS) for _s, n in portions)
    return ops.prefill_key_splits(blocks, shortest // 64, ops.sm_count(device))


def attend_over_pages(q, k_pages, v_pages, block_table, ctx, nh: int, nkv: int, hd: int, chunk: int, sliding: int,
                      scale: float, sink: bool = False, softcap: float = 0.0, slopes=None, sink_values=None, keep: int = 0):
    """softmax(q k^T scale + mask) v for the step's tokens over the paged keys and values that are in
    the cache already, by the kernel that fits the step: single decoded tokens, portions of prompts
    (with single tokens of other requests beside them), or the general kernel for what those refuse
    (float32, other head sizes). ``q`` [N, nh, hd] -> [N, nh, hd]. Every mixer whose scores are dot
    products over paged rows comes through here; ``k_pages`` and ``v_pages`` may be the same pool.
    ``sink``: the softmax's denominator has one more term of score 0 (it has no value); ``sink_values``
    (float32 [nh]): of the head's own score instead. ``softcap`` > 0: scores become softcap tanh(score / softcap);
    ``slopes`` (float32 [nh]): slopes[head] * (distance to the key) is taken off after the cap.
    ``keep``: first tokens of a request that a sliding window keeps."""
    positions = ctx.positions
    decode_ok = ops.decode_attention_supported(q.dtype, nh, nkv, hd)

    def decode(rows_q, seq, pos, longest):
        return ops.decode_attention(rows_q, k_pages, v_pages, block_table, seq, pos, chunk, sliding, scale, longest,
                                    sink=sink, softcap=softcap, slopes=slopes, sink_values=sink_values, keep=keep)

    if ctx.max_new == 1 and decode_ok:
        # every token of the step is one request's decoded token: the tensor-core kernel
        return decode(q, ctx.seq_of_token, positions, ctx.max_context)
    # at least a tile of new tokens somewhere: the tcgen05 kernel; short portions: mma.sync
    tc = ctx.max_new >= ops.PREFILL_TC_MIN_TOKENS and ops.prefill_attention_tc_supported(q.dtype, nh, nkv, hd, ctx.page_size)
    if ctx.max_new > 1 and ops.prefill_attention_supported(q.dtype, nh, nkv, hd):
        # portions of prompts (single tokens of other requests ride along as one-row tiles)
        single = ctx.decode_rows is not None and decode_ok
        if tc:
            o = ops.prefill_attention_tc(q, k_pages, v_pages, block_table, ctx.cu_seqlens, positions,
                                         ctx.n_seqs, ctx.max_new, chunk, sliding, scale, skip_single=single,
                                         key_splits=_key_splits(ctx, nh, chunk, sliding, single, q.device), sink=sink,
                                         softcap=softcap, slopes=slopes, sink_values=sink_values, keep=keep)
        else:
            o = ops.prefill_attention(q, k_pages, v_pages, block_table, ctx.cu_seqlens, positions,
                                      ctx.n_seqs, ctx.max_new, chunk, sliding, scale, skip_single=single, sink=sink,
                                      softcap=softcap, slopes=slopes, sink_values=sink_values, keep=keep)
        if single:
            # single tokens beside portions: their long key ranges go through the split decode kernel
            rows = ctx.decode_rows
            od = decode(q.index_select(0, rows), ctx.seq_of_token.index_select(0, rows), positions.index_select(0, rows),
                        ctx.decode_max_context)
            o.index_copy_(0, rows, od)
        return o
    return ops.paged_attention(q, k_pages, v_pages, block_table, ctx.seq_of_token, positions,
                               chunk, sliding, scale, ctx.max_context, sink=sink, softcap=softcap, slopes=slopes,
                               sink_values=sink_values, keep=keep)


def differential_attend_over_pages(q, k_pages, v_pages, block_table, ctx, chunk: int, sliding: int, keep: int, scale: float,
                                   lam: float, eps: float, mul: float, vdim: int, gate):
    """The two maps of every head (heads 2a and 2a + 1 of ``q`` [N, 2H, hd], both over the same cached rows), their
    difference a1 - lam a2 normed over the head's ``vdim`` values, times ``mul`` and the gate's sigmoid -> [N, H * vdim].
    The kernel is chosen by the step as in :func:`attend_over_pages`: from a tile of new tokens on the tcgen05 kernel,
    which takes both maps in one block and finishes the row itself; the other kernels leave their split partials in
    float32 and ``ops.diff_merge`` does the rest."""
    n, nh, hd = q.shape
    nkv, positions = k_pages.shape[1], ctx.positions
    finish = (lam, eps, mul, vdim, gate)
    decode_ok = ops.decode_attention_supported(q.dtype, nh, nkv, hd)

    def decode(rows_q, seq, pos, longest):
        return ops.decode_attention(rows_q, k_pages, v_pages, block_table, seq, pos, chunk, sliding, scale, longest,
                                    keep=keep, parts=True)

    def empty():
        return torch.empty((n, nh // 2 * vdim), dtype=q.dtype, device=q.device)

    if ctx.max_new == 1 and decode_ok:
        return ops.diff_merge(*decode(q, ctx.seq_of_token, positions, ctx.max_context), *finish, empty())
    if ctx.max_new > 1 and scale > 0 and ops.prefill_attention_supported(q.dtype, nh, nkv, hd):
        single = ctx.decode_rows is not None and decode_ok
        if ctx.max_new >= DIFF_TC_MIN_TOKENS and ops.prefill_attention_tc_supported(q.dtype, nh, nkv, hd, ctx.page_size):
            o = ops.diff_prefill_attention_tc(q, k_pages, v_pages, block_table, ctx.cu_seqlens, positions, ctx.n_seqs,
                                              ctx.max_new, chunk, sliding, keep, scale, *finish, skip_single=single)
        else:
            parts = ops.prefill_attention(q, k_pages, v_pages, block_table, ctx.cu_seqlens, positions, ctx.n_seqs,
                                          ctx.max_new, chunk, sliding, scale, skip_single=single, keep=keep, parts=True)
            o = ops.diff_merge(*parts, *finish, empty())
        if single:
            # single tokens beside portions (their rows of ``o`` are not written so far)
            rows = ctx.decode_rows
            parts = decode(q.index_select(0, rows), ctx.seq_of_token.index_select(0, rows), positions.index_select(0, rows),
                           ctx.decode_max_context)
            ops.diff_merge(*parts, *finish, o, rows=rows)
        return o
    parts = ops.paged_attention(q, k_pages, v_pages, block_table, ctx.seq_of_token, positions, chunk, sliding, scale,
                                ctx.max_context, keep=keep, parts=True)
    return ops.diff_merge(*parts, *finish, empty())


def sigmoid_attend_over_pages(q, k_pages, v_pages, block_table, ctx, nh: int, nkv: int, hd: int, chunk: int,
                              sliding: int, scale: float, head_bias, v_inv_freq, v_interleaved: bool):
    """sum_j sigmoid(q . k_j scale + head_bias) v_j over the keys each token may read, turned back by the token's
    position where the values are cached rotated, by the kernel that fits the step, as :func:`attend_over_pages`
    chooses for the softmax: the tensor-core decode kernel for single tokens, the tcgen05 kernel for portions of
    at least a tile of new tokens (single tokens beside them through the decode kernel), the general kernel for the
    rest (float32, other head sizes, short portions)."""
    positions = ctx.positions
    if ops.sigmoid_attention_tc_supported(q.dtype, nh, nkv, hd, ctx.page_size):
        if ctx.max_new == 1:
            return ops.sigmoid_decode_attention(q, k_pages, v_pages, block_table, ctx.seq_of_token, positions, chunk,
                                                sliding, scale, head_bias, ctx.max_context, v_inv_freq, v_interleaved)
        if ctx.max_new >= ops.PREFILL_TC_MIN_TOKENS:
            single = ctx.decode_rows is not None
            o = ops.sigmoid_prefill_attention_tc(q, k_pages, v_pages, block_table, ctx.cu_seqlens, positions, ctx.n_seqs,
                                                 ctx.max_new, chunk, sliding, scale, head_bias, skip_single=single,
                                                 v_inv_freq=v_inv_freq, v_interleaved=v_interleaved)
            if single:
                rows = ctx.decode_rows
                od = ops.sigmoid_decode_attention(q.index_select(0, rows), k_pages, v_pages, block_table,
                                                  ctx.seq_of_token.index_select(0, rows), positions.index_select(0, rows),
                                                  chunk, sliding, scale, head_bias, ctx.decode_max_context, v_inv_freq,
                                                  v_interleaved)
                o.index_copy_(0, rows, od)
            return o
    return ops.sigmoid_attention(q, k_pages, v_pages, block_table, ctx.seq_of_token, positions, chunk, sliding, scale,
                                 head_bias, ctx.max_context, v_inv_freq=v_inv_freq, v_interleaved=v_interleaved)


@register("mixer", "attention")
class AttentionMixer(Part):
    """q/k/v projections, position encoding or temperature, optional weightless q/k norm, cache
    append, softmax(q k^T scale + mask) v, output projection
    (Llama4Attention::forward, crates/hi-mlx/src/models.rs:5978-6052).

    params:
      ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``
      ``window``       None (every earlier key) | ("chunk", C) | ("sliding", W) | ("sliding", W, K): the last W tokens
                       and the first K of the request
      ``position``     PartSpec of the position family
      ``qk_norm``, ``qk_norm_eps``   weightless L2 norm of q and k after the rotation
      ``temperature``  None | (floor_scale, attn_scale): q *= 1 + attn_scale*ln(1 + floor((pos+1)/floor_scale))
      ``scale``        softmax scale; default head_dim ** -0.5 (models.rs:5963)
      ``bias``         the random-weights writer makes the projections' biases too: True (all four) or a
                       string of the projections that have one ("qkv")
      ``value_dim``    size of a value head where it differs from ``head_dim`` (the query/key size). Keys,
                       values and queries are then kept in rows of one padded size (the larger of the two,
                       rounded up to 16): the projections get zero rows, the output projection zero columns
      ``qk_norm_weighted``  the norm of q and k is an RMS norm BEFORE the rotation with a weight per dim,
                       ``<prefix>.q.norm`` / ``<prefix>.k.norm`` [head_dim], shared by the heads
      ``sink``         the softmax's denominator has one more term of score 0: exp(s_j) / (1 + sum exp(s_j));
                       "learned": the term's score is a number per head, ``<prefix>.sink`` [heads], that is not
                       scaled, capped or biased: exp(s_j) / (exp(sink_h) + sum exp(s_j))
      ``softcap``      None | c: the scaled score becomes c tanh(score / c)
      ``distance_bias``  None | e: slope_h * (i - j) is taken off the (capped) score of query i and key j,
                       slope_h = 2^(-e (h + 1) / heads) for head h = 0 .. heads - 1
      ``names``        "proj" (default): ``<prefix>.{q,k,v,o}_proj.weight`` / ``.bias``;
                       "short": ``<prefix>.{q,k,v,o}`` and ``<prefix>.{q,k,v,o}.b``
      ``weights``      "softmax" (default) | "sigmoid": the weight of a visible key is sigmoid(score + pb[head]),
                       ``<prefix>.pb`` [heads], and the weights are not normalised over the keys
      ``value_rotation``  None | {"base": b, "interleaved": bool}: the value of position j is cached rotated by j
                       over all its dims (pair m by j * b^(-2m / value_dim)) and each head's sum at position i is
                       turned back by i, so a value's weight in the output also depends on i - j
      ``conv``         None | K: every channel of q, k and v passes a causal convolution of K taps over time right
                       after the projection, y_t = sum_j taps[:, j] u_(t - K + 1 + j) (zeros before the start):
                       ``<prefix>.{q,k,v}.conv`` [channels, K]; the last K - 1 inputs are state of the request
      ``differential``  None | c: every query and key head has two maps of ``head_dim`` (a head's second map
                       follows its first in the projection's rows), each an attention of its own over the same values; their results a1, a2 give
                       o = a1 - lambda a2 with lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + c (one number a layer,
                       ``<prefix>.lq1|lk1|lq2|lk2`` [head_dim]), and o <- o / rms(o) (over the head's values, eps
                       ``qk_norm_eps``) * (1 - c)
      ``values``       "projected" (default) | "keys": there is no value projection; a key as projected, before norm and
                       rotation, is its value too (``value_dim`` is then ``head_dim``)
      ``output_gate``  the heads' results are multiplied element by element by sigmoid(W_g h), ``<prefix>.g``
                       [heads * value_dim, H], before the output projection
    tensors: the four projections (without ``v`` where the values are the keys), and each projection's bias where the checkpoint has one (a bias is
    used iff its tensor exists: crates/hi-mlx/src/models.rs:1808, 1843-1845).
    """

    graph_safe = True
    FUSED_DECODE = True      # decode steps: one launch for encoding, cache append, attention and merge

    def __init__(self, params, prefix, env):
        super().__init__(params, prefix, env)
        p = params
        self.hidden = int(p["hidden_size"])
        self.nh, self.nkv, self.hd = int(p["num_heads"]), int(p["num_kv_heads"]), int(p["head_dim"])
        if self.nh % self.nkv:
            raise ValueError(f"{prefix}: {self.nh} heads are not a multiple of {self.nkv} kv heads")
        self.dim, self.vdim = self.hd, int(p.get("value_dim") or self.hd)      # sizes as the checkpoint has them
        self.norm_weighted = bool(p.get("qk_norm_weighted", False))
        self.sink = bool(p.get("sink", False))
        self.learned_sink = p.get("sink") == "learned"
        self.softcap = float(p["softcap"]) if p.get("softcap") else 0.0
        self.distance_bias = float(p["distance_bias"]) if p.get("distance_bias") else None
        self.sink_values = self.slopes = None
        self.sigmoid = p.get("weights", "softmax") == "sigmoid"
        if p.get("weights", "softmax") not in ("softmax", "sigmoid") or (self.sigmoid and self.sink):
            raise ValueError(f"{prefix}: weights are 'softmax' or 'sigmoid' (which has no sink)")
        self.value_rotation = dict(p["value_rotation"]) if p.get("value_rotation") else None
        if self.value_rotation and not self.sigmoid:
            raise ValueError(f"{prefix}: rotated values are built for sigmoid weights only")
        if self.sigmoid and (self.softcap or self.distance_bias is not None):
            raise ValueError(f"{prefix}: a cap or a distance bias on the scores is built for softmax weights only")
        self.head_bias = self._v_table = None
        self.taps = int(p.get("conv") or 0)
        self.diff = float(p["differential"]) if p.get("differential") is not None else None
        self.gated = bool(p.get("output_gate", False))
        self.maps = 1 if self.diff is None else 2
        self.values_are_keys = p.get("values", "projected") == "keys"
        if p.get("values", "projected") not in ("projected", "keys"):
            raise ValueError(f"{prefix}: values are 'projected' or 'keys'")
        if self.values_are_keys and (self.vdim != self.dim or self.sigmoid or self.taps or self.diff is not None or p.get("output_gate")):
            raise ValueError(f"{prefix}: values that are the keys are built for softmax weights, one head size, no convolution, "
                             f"second map or output gate")
        # these work on the unpadded projection (ops.conv_qkv encodes and appends)
        self.unpadded = bool(self.taps) or self.diff is not None or self.gated
        if self.unpadded and (self.sigmoid or p.get("temperature") or (p.get("qk_norm") and not self.norm_weighted)):
            raise ValueError(f"{prefix}: a convolution, a second map or an output gate is built for softmax weights, without a "
                             f"query temperature or a norm after the rotation")
        if self.diff is not None and (self.sink or self.softcap or self.distance_bias is not None):
            raise ValueError(f"{prefix}: two maps are built for plain scores without a sink")
        self.conv_taps = None
        self.lam = 0.0
        self.short_names = p.get("names", "proj") == "short"
        if self.diff is not None:
            # a key row holds both maps; rows that the tensor-core kernels take where one is long enough
            self.hd = -(-max(2 * self.dim, self.vdim) // 16) * 16
            if env.dtype == torch.bfloat16:
                self.hd = next((r for r in ops.TC_ROW_LENGTHS if r >= self.hd), self.hd)
        elif self.dim != self.vdim or self.dim % 16:
            self.hd = -(-max(self.dim, self.vdim) // 16) * 16                  # rows of the cache and of q
        if self.hd > (1024 if self.hd != self.dim or self.norm_weighted or self.unpadded or self.values_are_keys else 256):
            raise ValueError(f"{prefix}: head size {self.hd} is not supported")
        self.window = tuple(p["window"]) if p.get("window") else None
        self.keep = int(self.window[2]) if self.window and len(self.window) > 2 else 0
        self.position = build("position", p.get("position") or PartSpec("none"), env, prefix)
        self.qk_norm = bool(p.get("qk_norm", False)) or self.norm_weighted
        self.qk_norm_eps = float(p.get("qk_norm_eps", 1e-6))
        self.temperature = tuple(p["temperature"]) if p.get("temperature") else None
        self.scale = float(p.get("scale") or self.dim ** -0.5)
        self.bias = p.get("bias", False)
        self.w_qnorm = self.w_knorm = None
        self.w_qkv: Optional[torch.Tensor] = None
        self.w_o: Optional[torch.Tensor] = None
        self.b_qkv: Optional[torch.Tensor] = None
        self.b_o: Optional[torch.Tensor] = None

    def cache_spec(self):
        state = (self.taps - 1) * self.channels if self.taps > 1 else 0
        return CacheSpec(kv_heads=self.nkv, head_dim=self.hd, window=self.window, state_shape=(state,) if state else ())

    @property
    def channels(self) -> int:
        """Columns of the unpadded projection that q, k and v take."""
        return (self.nh + self.nkv) * self.maps * self.dim + self.nkv * self.vdim

    def _name(self, proj: str, bias: bool = False) -> str:
        if self.short_names:
            return f"{self.prefix}.{proj}.b" if bias else f"{self.prefix}.{proj}"
        return f"{self.prefix}.{proj}_proj.bias" if bias else f"{self.prefix}.{proj}_proj.weight"

    def tensor_specs(self):
        h, nh, nkv = self.hidden, self.nh, self.nkv
        have = "qkvo" if self.bias is True else (self.bias or "")
        rows = {"q": nh * self.maps * self.dim, "k": nkv * self.maps * self.dim, "v": nkv * self.vdim, "o": h}
        names = "qko" if self.values_are_keys else "qkvo"
        specs = [TensorSpec(self._name(n), (rows[n], h) if n != "o" else (h, nh * self.vdim)) for n in names]
        # "absent": the random-weights writer leaves them out
        specs += [TensorSpec(self._name(n, bias=True), (rows[n],), init="normal" if n in have else "absent", optional=True)
                  for n in names]
        if self.norm_weighted:
            specs += [TensorSpec(f"{self.prefix}.{n}.norm", (self.dim,), init="ones") for n in "qk"]
        if self.sigmoid:
            specs.append(TensorSpec(f"{self.prefix}.pb", (self.nh,)))
        if self.learned_sink:
            specs.append(TensorSpec(f"{self.prefix}.sink", (self.nh,)))
        if self.taps:
            specs += [TensorSpec(f"{self.prefix}.{n}.conv", (rows[n], self.taps)) for n in "qkv"]
        if self.diff is not None:
            specs += [TensorSpec(f"{self.prefix}.{n}", (self.dim,)) for n in ("lq1", "lk1", "lq2", "lk2")]
        if self.gated:
            specs.append(TensorSpec(f"{self.prefix}.g", (nh * self.vdim, h)))
        return specs

    def _pad_heads(self, t, heads: int, size: int):
        """[heads * size, ...] -> [heads * hd, ...] with zero rows behind every head's own."""
        if t is None or size == self.hd:
            return t
        out = torch.zeros((heads, self.hd, *t.shape[1:]), dtype=t.dtype, device=t.device)
        out[:, :size] = t.view(heads, size, *t.shape[1:])
        return out.view(heads * self.hd, *t.shape[1:])

    def _load_unpadded(self, fetch):
        """One product for q, k, v and the gate, rows as the checkpoint has them."""
        rows = [fetch(self._name(n)) for n in "qkv"] + ([fetch(f"{self.prefix}.g")] if self.gated else [])
        if self.gated and self.channels % 8:         # the gate's rows start on 16 bytes
            rows.insert(3, torch.zeros((-self.channels % 8, self.hidden), dtype=rows[0].dtype, device=rows[0].device))
        self.gate_at = -(-self.channels // 8) * 8
        pad = -sum(t.shape[0] for t in rows) % 8
        if pad:
            rows.append(torch.zeros((pad, self.hidden), dtype=rows[0].dtype, device=rows[0].device))
        if len({t.dtype for t in rows}) > 1:
            rows = [t.float() for t in rows]
        self.w_qkv = torch.cat(rows, dim=0).contiguous()
        w_o = fetch(self._name("o"))
        if self.diff is None and not self.gated and self.vdim != self.hd:
            w_o = self._pad_heads(w_o.t().contiguous(), self.nh, self.vdim).t()
        self.w_o = w_o.contiguous()
        f32, dev = torch.float32, self.w_qkv.device
        biases = [fetch(self._name(n, bias=True)) for n in "qkv"]
        if any(b is not None for b in biases):
            full = torch.zeros(self.w_qkv.shape[0], dtype=self.w_qkv.dtype, device=dev)
            at = 0
            for b, t in zip(biases, rows):
                if b is not None:
                    full[at: at + b.numel()] = b.to(full.dtype)
                at += t.shape[0]
            self.b_qkv = full
        b_o = fetch(self._name("o", bias=True))
        self.b_o = None if b_o is None else b_o.to(self.w_o.dtype).contiguous()
        if self.norm_weighted:
            self.w_qnorm, self.w_knorm = (fetch(f"{self.prefix}.{n}.norm").to(f32).contiguous() for n in "qk")
        if self.taps:
            self.conv_taps = torch.cat([fetch(f"{self.prefix}.{n}.conv").to(f32) for n in "qkv"], dim=0).t().contiguous()      # [K, channels]
        if self.diff is not None:
            lq1, lk1, lq2, lk2 = (fetch(f"{self.prefix}.{n}").to(torch.float64) for n in ("lq1", "lk1", "lq2", "lk2"))
            self.lam = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + self.diff)
        self._load_score_tensors(fetch)

    def _load_score_tensors(self, fetch):
        if self.learned_sink:
            self.sink_values = fetch(f"{self.prefix}.sink").to(torch.float32).contiguous()
        if self.distance_bias is not None:
            slopes = [2.0 ** (-self.distance_bias * (h + 1) / self.nh) for h in range(self.nh)]
            self.slopes = torch.tensor(slopes, dtype=torch.float64).to(torch.float32).to(self.w_qkv.device)

    def load(self, fetch):
        if self.unpadded:
            return self._load_unpadded(fetch)
        names = "qk" if self.values_are_keys else "qkv"
        rows = [fetch(self._name(n)) for n in names]
        if len({t.dtype for t in rows}) > 1:
            rows = [t.float() for t in rows]
        sizes = ((self.nh, self.dim), (self.nkv, self.dim), (self.nkv, self.vdim))[: len(names)]
        self.w_qkv = torch.cat([self._pad_heads(t, *hs) for t, hs in zip(rows, sizes)], dim=0).contiguous()     # one product
        w_o = fetch(self._name("o"))
        if self.vdim != self.hd:
            w_o = self._pad_heads(w_o.t().contiguous(), self.nh, self.vdim).t()
        self.w_o = w_o.contiguous()
        biases = [fetch(self._name(n, bias=True)) for n in names]
        if any(b is not None for b in biases):          # a projection without one adds zeros
            biases = [torch.zeros(hs[0] * self.hd, dtype=self.w_qkv.dtype, device=self.w_qkv.device) if b is None
                      else self._pad_heads(b, *hs) for b, hs in zip(biases, sizes)]
            self.b_qkv = torch.cat([b.to(self.w_qkv.dtype) for b in biases]).contiguous()
        b_o = fetch(self._name("o", bias=True))
        self.b_o = None if b_o is None else b_o.to(self.w_o.dtype).contiguous()
        if self.norm_weighted:
            def weight(n):
                w = torch.zeros(self.hd, dtype=torch.float32, device=self.w_qkv.device)
                w[: self.dim] = fetch(f"{self.prefix}.{n}.norm").to(torch.float32)
                return w
            self.w_qnorm, self.w_knorm = weight("q"), weight("k")
        if self.sigmoid:
            self.head_bias = fetch(f"{self.prefix}.pb").to(torch.float32).contiguous()
        self._load_score_tensors(fetch)
        if self.value_rotation:
            if self.vdim % 2:
                raise ValueError(f"{self.prefix}: rotated values need an even value size")
            base = float(self.value_rotation["base"])
            table = np.array([base ** (-2.0 * m / self.vdim) for m in range(self.vdim // 2)], dtype=np.float64)
            self._v_table = torch.from_numpy(table.astype(np.float32)).to(self.w_qkv.device)

    def _forward_unpadded(self, normed, ctx, cache):
        if self.taps > 1 and (cache.state is None or not cache.writes):
            raise RuntimeError(f"{self.prefix}: a convolution over time needs a state slot of its own")
        proj = linear(normed, self.w_qkv, bias=self.b_qkv)
        table = self.position.rotary_table()
        if table is None and hasattr(self.position, "apply"):
            raise TypeError(f"{self.prefix}: position parts without a rotary table work on the padded projection only")
        inv_freq, interleaved = table if table is not None else (None, False)
        block_table = ctx.block_tables[cache.group]
        chunk = self.window[1] if self.window and self.window[0] == "chunk" else 0
        sliding = self.window[1] if self.window and self.window[0] == "sliding" else 0
        q = ops.conv_qkv(proj, self.conv_taps, cache.state, self.norm_weighted, self.qk_norm_eps, self.w_qnorm, self.w_knorm,
                         inv_freq, interleaved, float(getattr(self.position, "magnitude", 1.0)), ctx.positions,
                         ctx.seq_of_token, ctx.cu_seqlens, ctx.slots, block_table, cache.k_pages, cache.v_pages,
                         cache.writes, ctx.max_new == 1, self.nh, self.nkv, self.maps, self.dim, self.vdim)
        gate = proj[:, self.gate_at: self.gate_at + self.nh * self.vdim] if self.gated else None
        if self.diff is not None:
            o = differential_attend_over_pages(q, cache.k_pages, cache.v_pages, block_table, ctx, chunk, sliding, self.keep,
                                               self.scale, self.lam, self.qk_norm_eps, 1.0 - self.diff, self.vdim, gate)
            return linear(o, self.w_o, bias=self.b_o)
        o = attend_over_pages(q, cache.k_pages, cache.v_pages, block_table, ctx, self.nh, self.nkv, self.hd, chunk, sliding,
                              self.scale, sink=self.sink, softcap=self.softcap, slopes=self.slopes,
                              sink_values=self.sink_values, keep=self.keep)
        o = ops.gate_rows(o, gate, self.vdim) if gate is not None else o.view(o.shape[0], self.nh * self.hd)
        return linear(o, self.w_o, bias=self.b_o)

    def forward(self, normed, ctx, cache):
        if self.unpadded:
            return self._forward_unpadded(normed, ctx, cache)
        qkv = linear(normed, self.w_qkv, bias=self.b_qkv)
        positions = ctx.positions
        table = self.position.rotary_table()
        if table is None and hasattr(self.position, "apply"):
            # a position part without a rotary table encodes q and k itself
            if self.values_are_keys:
                raise TypeError(f"{self.prefix}: values that are the keys need a position part with a rotary table")
            n = qkv.shape[0]
            q, k, v = qkv.split([self.nh * self.hd, self.nkv * self.hd, self.nkv * self.hd], dim=1)
            q, k = self.position.apply(q.reshape(n, self.nh, self.hd), k.reshape(n, self.nkv, self.hd), positions)
            qkv = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v], dim=1).to(normed.dtype).contiguous()
        inv_freq, interleaved = table if table is not None else (None, False)
        block_table = ctx.block_tables[cache.group]
        chunk = self.window[1] if self.window and self.window[0] == "chunk" else 0
        sliding = self.window[1] if self.window and self.window[0] == "sliding" else 0
        rot_mul = float(getattr(self.position, "magnitude", 1.0))
        plain = not (self.norm_weighted or self.sink or self.hd != self.dim or rot_mul != 1.0)
        if self.sigmoid:
            v_inter = bool(self.value_rotation and self.value_rotation.get("interleaved", False))
            q = ops.qkv_post(qkv, self.nh, self.nkv, self.hd, positions, inv_freq, interleaved, self.qk_norm,
                             self.qk_norm_eps, self.temperature, ctx.seq_of_token, block_table, cache.k_pages,
                             cache.v_pages, ctx.page_size, cache.writes, q_norm_weight=self.w_qnorm,
                             k_norm_weight=self.w_knorm, norm_first=self.norm_weighted,
                             norm_dim=0 if plain else self.dim, rot_mul=rot_mul, v_inv_freq=self._v_table,
                             v_interleaved=v_inter)
            o = sigmoid_attend_over_pages(q, cache.k_pages, cache.v_pages, block_table, ctx, self.nh, self.nkv, self.hd,
                                          chunk, sliding, self.scale, self.head_bias, self._v_table, v_inter)
            return linear(o.view(o.shape[0], self.nh * self.hd), self.w_o, bias=self.b_o)
        extras = self.keep > 0 or bool(self.softcap) or self.slopes is not None or self.sink_values is not None
        if self.hd == self.dim and ctx.max_new == 1 and cache.writes and self.FUSED_DECODE and qkv.dtype == torch.bfloat16 \
                and not extras:
            # a step of single decoded tokens: encoding, cache append, attention and the merge of its
            # splits in one launch, where the kernel takes the shapes
            o = ops.decode_attention_fused(qkv, self.nh, self.nkv, self.hd, positions, inv_freq, interleaved, self.qk_norm,
                                           self.qk_norm_eps, self.temperature, ctx.seq_of_token, block_table,
                                           cache.k_pages, cache.v_pages, chunk, sliding, self.scale, ctx.max_context,
                                           q_norm_weight=self.w_qnorm, k_norm_weight=self.w_knorm,
                                           norm_first=self.norm_weighted, rot_mul=rot_mul, sink=self.sink,
                                           values_are_keys=self.values_are_keys)
            if o is not None:
                return linear(o.view(o.shape[0], self.nh * self.hd), self.w_o, bias=self.b_o)
        q = ops.qkv_post(qkv, self.nh, self.nkv, self.hd, positions, inv_freq, interleaved, self.qk_norm,
                         self.qk_norm_eps, self.temperature, ctx.seq_of_token, block_table, cache.k_pages,
                         cache.v_pages, ctx.page_size, cache.writes, q_norm_weight=self.w_qnorm,
                         k_norm_weight=self.w_knorm, norm_first=self.norm_weighted,
                         norm_dim=0 if plain else self.dim, rot_mul=rot_mul, values_are_keys=self.values_are_keys)
        o = attend_over_pages(q, cache.k_pages, cache.v_pages, block_table, ctx, self.nh, self.nkv, self.hd, chunk,
                              sliding, self.scale, sink=self.sink, softcap=self.softcap, slopes=self.slopes,
                              sink_values=self.sink_values, keep=self.keep)
        return linear(o.view(o.shape[0], self.nh * self.hd), self.w_o, bias=self.b_o)
