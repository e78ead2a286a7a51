"""Darotar without a GPU: the plain implementation's mechanisms against closed forms and against each other, the
configuration reader, and the ModelSpec the builder makes (parts, cache slots that layers share, tensor names)."""
import copy
import math

import pytest
import torch

import plain_darotar as plain
from darotar_configs import CONFIGS, DA_A, DA_B, DA_C, DA_D, attention, config, latent, make_weights, moe, plain_logits, write_model

F64 = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


def _one_layer(layer, width=24, **kw):
    cfg = config(19, width, 1e-5, [layer], **kw)
    return cfg, {k: v.double() for k, v in make_weights(cfg, 3).items()}


# --------------------------------------------------------------------------- mechanisms of the plain model
def test_rotation_pairs_and_scaling():
    rot = {"base": 100.0, "dims": 6}
    x = rnd(12, 2, 9, seed=1)
    near, far = plain.rotate(x, rot, True), plain.rotate(x, rot, False)
    for y in (near, far):
        assert torch.equal(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])          # position 0; dims that pass
        assert torch.allclose(y.pow(2).sum(-1), x.pow(2).sum(-1))
    a = 7 * 100.0 ** (-4.0 / 6)                                                          # pair 2 at position 7
    assert torch.allclose(near[7, :, 4], x[7, :, 4] * math.cos(a) - x[7, :, 5] * math.sin(a))
    assert torch.allclose(near[7, :, 5], x[7, :, 5] * math.cos(a) + x[7, :, 4] * math.sin(a))
    assert torch.allclose(far[7, :, 2], x[7, :, 2] * math.cos(a) - x[7, :, 5] * math.sin(a))
    assert torch.allclose(far[7, :, 5], x[7, :, 5] * math.cos(a) + x[7, :, 2] * math.sin(a))
    slow = plain.rotate(x, {**rot, "scaling": {"factor": 3.0}}, True)
    assert torch.allclose(slow[9], plain.rotate(x[[0, 0, 0, 9]], rot, True)[3])          # position 9 turns as position 3
    # a product of two rotated rows depends on their distance only
    q, k = rnd(1, 1, 6, seed=2).expand(12, 1, 6), rnd(1, 1, 6, seed=3).expand(12, 1, 6)
    qr, kr = plain.rotate(q, rot, True)[:, 0], plain.rotate(k, rot, True)[:, 0]
    assert math.isclose(float(qr[9] @ kr[5]), float(qr[4] @ kr[0]))


def test_a_sink_takes_weight_and_has_no_value():
    s, see = rnd(5, 5, seed=4), plain.visible(5, None)
    p = plain.softmax_weights(s, see, torch.tensor(0.7, dtype=F64))
    want = torch.exp(s[3, :4]) / (torch.exp(s[3, :4]).sum() + math.exp(0.7))
    assert torch.allclose(p[3, :4], want) and float(p[3, 4]) == 0.0
    assert torch.allclose(plain.softmax_weights(s, see).sum(-1), torch.ones(5, dtype=F64))
    assert float(plain.softmax_weights(s, see, torch.tensor(500.0, dtype=F64)).max()) < 1e-200
    assert torch.allclose(plain.softmax_weights(s, see, torch.tensor(-500.0, dtype=F64)), plain.softmax_weights(s, see))


def test_the_window_counts_the_token_itself():
    see = plain.visible(12, 3)
    assert see[9].nonzero().flatten().tolist() == [7, 8, 9] and see[1].nonzero().flatten().tolist() == [0, 1]
    assert torch.equal(plain.visible(6, 1), torch.eye(6, dtype=torch.bool))
    assert bool(plain.visible(6, None)[5].all())


def test_attention_mechanisms_each_matter():
    cfg, w = _one_layer(attention(4, 2, 8, 0.5, 40.0, dims=6, factor=2.0, window=6))
    m, h = cfg["layers"][0]["mixer"], rnd(20, 24, seed=7)
    y = plain.attention(h, m, w, "l0.mix", 1e-5)
    h2 = h.clone()
    h2[9:] += 1.0
    assert torch.equal(plain.attention(h2, m, w, "l0.mix", 1e-5)[:9], y[:9])                       # causal
    h2 = h.clone()
    h2[8] += 1.0
    y2 = plain.attention(h2, m, w, "l0.mix", 1e-5)
    assert torch.equal(y2[14:], y[14:]) and not torch.allclose(y2[13], y[13])                      # the window's edge
    for change in ({"scale": 1.0}, {"mask": {"size": 7}}, {"mask": None}, {"rot": {**m["rot"], "dims": 8}},
                   {"rot": {**m["rot"], "base": 41.0}}, {"rot": {"base": 40.0, "dims": 6}}):
        assert not torch.allclose(plain.attention(h, {**m, **change}, w, "l0.mix", 1e-5)[12:], y[12:]), change
    w2 = {k: v * (3.0 if k.endswith(".q") else 1.0) for k, v in w.items()}
    assert torch.allclose(plain.attention(h, m, w2, "l0.mix", 0.0), plain.attention(h, m, w, "l0.mix", 0.0))     # q is normed


def test_values_are_the_keys_before_norm_and_rotation():
    """With a window of one token a row reads its own value alone: the key projection as it is."""
    cfg, w = _one_layer(attention(2, 1, 6, 0.5, 40.0, window=1))
    m, h = cfg["layers"][0]["mixer"], rnd(9, 24, seed=8)
    k = h @ w["l0.mix.k"].T
    assert torch.allclose(plain.attention(h, m, w, "l0.mix", 1e-5), torch.cat([k, k], dim=-1) @ w["l0.mix.o"].T)


def test_latent_attention_mechanisms_each_matter():
    cfg, w = _one_layer(latent(3, 8, 4, 6, 10, 9, 0.4, 50.0))
    m, h = cfg["layers"][0]["mixer"], rnd(15, 24, seed=9)
    rows = plain.latents(h, m, w, "l0.mix", 1e-5)
    y = plain.latent_attention(h, m, w, "l0.mix", 1e-5, rows)
    h2 = h.clone()
    h2[9:] += 1.0
    y2 = plain.latent_attention(h2, m, w, "l0.mix", 1e-5, plain.latents(h2, m, w, "l0.mix", 1e-5))
    assert torch.equal(y2[:9], y[:9])
    assert not torch.allclose(plain.latent_attention(h, {**m, "scale": 0.5}, w, "l0.mix", 1e-5, rows), y)
    for name in ("dq.norm", "uk", "uv", "g", "sink"):
        w2 = {**w, f"l0.mix.{name}": w[f"l0.mix.{name}"].flip(0) * 1.5}
        assert not torch.allclose(plain.latent_attention(h, m, w2, "l0.mix", 1e-5, rows), y), name
    # the latent is normed and the shared key part is not: it grows with its rows of the down projection
    w2 = {**w, "l0.mix.dkv": w["l0.mix.dkv"] * 2.0}
    c2, k2 = plain.latents(h, m, w2, "l0.mix", 0.0)
    c, k = plain.latents(h, m, w, "l0.mix", 0.0)
    assert torch.allclose(c2, c) and torch.allclose(k2, 2.0 * k)
    # a gate that is open everywhere leaves one half of the heads' results
    w2 = {**w, "l0.mix.g": torch.zeros_like(w["l0.mix.g"])}
    big = {**w, "l0.mix.g": torch.zeros_like(w["l0.mix.g"]), "l0.mix.o": w["l0.mix.o"] * 2.0}
    assert torch.allclose(2.0 * plain.latent_attention(h, m, w2, "l0.mix", 1e-5, rows),
                          plain.latent_attention(h, m, big, "l0.mix", 1e-5, rows))


def test_scores_scale_what_the_experts_read():
    cfg, w = _one_layer(attention(1, 1, 4, 0.5, 10.0, mlp=moe(4, 2, 10)))
    mlp, h = cfg["layers"][0]["mlp"], rnd(11, 24, seed=5)
    ids, s = plain.router_choice(h, mlp, w, "l0.mlp")
    assert torch.allclose(s, 1 / (1 + torch.exp(-(h @ w["l0.mlp.router"].T))))
    y, t = plain.mixture(h, mlp, w, "l0.mlp"), 6
    want = 0
    for e in ids[t].tolist():
        x = s[t, e] * h[t]
        g = w[f"l0.mlp.e{e}.gate"] @ x
        want = want + w[f"l0.mlp.e{e}.down"] @ (g / (1 + torch.exp(-g)) * (w[f"l0.mlp.e{e}.up"] @ x))
    assert torch.allclose(y[t], want)
    outside = sum(s[t, e] * plain.silu_unit(h[t: t + 1], w, f"l0.mlp.e{e}")[0] for e in ids[t].tolist())
    assert not torch.allclose(y[t], outside)
    assert sorted(ids[t].tolist()) == sorted(torch.topk(s[t], 2).indices.tolist())


def test_norms_act_on_what_the_sublayers_return():
    """A sub-layer's gain cancels in its norm (eps 0), the norms' weights and the factor do not; with both at zero the
    stream stays the embedding."""
    cfg = copy.deepcopy(DA_A)
    cfg["norm"]["eps"] = 1e-30
    w = {k: v.double() for k, v in make_weights(cfg, 1).items()}
    toks = [3, 5, 7, 9]
    ref = plain.forward(cfg, w, toks)
    w2 = {k: v * 5.0 if k.endswith(".mix.o") or k.endswith(".down") else v for k, v in w.items()}
    assert torch.allclose(plain.forward(cfg, w2, toks), ref, atol=1e-8)
    assert not torch.allclose(plain.forward({**cfg, "residual_mult": 0.5}, w, toks), ref)
    streams = []
    plain.forward({**cfg, "residual_mult": 0.0}, w, toks, streams=streams)
    assert len(streams) == 6 and all(torch.equal(s, w["embed"][toks]) for s in streams)
    halved = {k: v * 0.5 if k.endswith(".norm1") or k.endswith(".norm2") else v for k, v in w.items()}
    assert torch.allclose(plain.forward({**cfg, "residual_mult": 1.2}, halved, toks), ref, atol=1e-8)


def test_a_layer_that_reads_anothers_latents():
    """A reader whose own maps equal the source's reads the source's rows, not its own input's."""
    one = latent(2, 8, 4, 6, 10, 9, 0.4, 50.0)
    two = latent(2, 8, 4, 6, 10, 9, 0.4, 50.0, kv_from=0)
    cfg = config(19, 24, 1e-5, [one, two])
    w = {k: v.double() for k, v in make_weights(cfg, 3).items()}
    assert "l1.mix.dkv" not in w and "l1.mix.uk" in w
    toks = [1, 4, 2, 8, 5, 7]
    shared = plain.forward(cfg, w, toks)
    own = copy.deepcopy(cfg)
    del own["layers"][1]["mixer"]["kv_from"]
    w2 = {**w, "l1.mix.dkv": w["l0.mix.dkv"], "l1.mix.dkv.norm": w["l0.mix.dkv.norm"]}
    assert not torch.allclose(plain.forward(own, w2, toks), shared)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_a_longer_sequence_keeps_its_prefix(name):
    cfg = CONFIGS[name]
    w = make_weights(cfg, 7)
    toks = [(7 * i + 3) % cfg["vocab"] for i in range(26)]
    a, b = plain_logits(cfg, w, toks), plain_logits(cfg, w, toks[:19])
    assert torch.allclose(a[:19], b, atol=1e-9)
    assert float(a.std()) > 0.3


# --------------------------------------------------------------------------- configuration and ModelSpec
def test_reader_takes_every_size_from_the_configuration():
    from hi_b200.config.darotar import DarotarConfig

    c = DarotarConfig.from_json(DA_A)
    assert (c.vocab, c.width, c.eps, c.residual_mult) == (131, 64, 1e-5, 0.6)
    a, l = c.layers[1].mixer, c.layers[2].mixer
    assert (a.heads, a.kv_heads, a.dim, a.scale, a.window) == (4, 2, 16, 0.2, 40)
    assert (a.rot.base, a.rot.dims, a.rot.factor) == (1000.0, 16, 2.5)
    assert (l.heads, l.dim, l.rot_dim, l.vdim, l.kv_rank, l.q_rank, l.scale, l.kv_from) == (2, 24, 8, 20, 24, 12, 0.25, 0)
    assert (c.layers[1].mlp.experts, c.layers[1].mlp.top, c.layers[1].mlp.ff) == (6, 2, 16) and c.layers[2].mlp is None
    d = DarotarConfig.from_json({k: v for k, v in DA_C.items() if k != "residual_mult"})
    assert d.residual_mult == 1.0 and d.layers[0].mixer.window is None and d.layers[0].mixer.rot.factor is None


@pytest.mark.parametrize("path,value,names", [
    (("vocab",), None, "vocab"), (("norm", "eps"), None, "eps"), (("layers", 0, "type"), "mamba2", "type"),
    (("layers", 0, "mixer", "kv_rank"), None, "kv_rank"), (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 1, "mixer", "vdim"), 8, "vdim"), (("layers", 1, "mixer", "scale"), None, "scale"),
    (("layers", 1, "mixer", "mask", "size"), 0, "size"), (("layers", 1, "mixer", "rot", "dims"), 5, "dims"),
    (("layers", 1, "mixer", "rot", "scaling", "factor"), 0.0, "factor"), (("layers", 0, "mixer", "rot", "dims"), 4, "dims"),
    (("layers", 2, "mixer", "kv_from"), 1, "kv_from"), (("layers", 2, "mixer", "kv_from"), 4, "kv_from"),
    (("layers", 5, "mixer", "kv_from"), 2, "kv_from"), (("layers", 5, "mixer", "kv_from"), -1, "kv_from"),
    (("layers", 2, "mixer", "kv_rank"), 16, "kv_rank"), (("layers", 0, "mlp", "kind"), "dense", "kind"),
    (("layers", 1, "mlp", "router", "top"), 9, "top"), (("layers", 1, "mlp", "expert", "ff"), None, "ff"), (("layers",), [], "layers")])
def test_reader_names_what_is_wrong(path, value, names):
    from hi_b200.config.base import ConfigError
    from hi_b200.config.darotar import DarotarConfig

    cfg = copy.deepcopy(DA_A)
    node = cfg
    for key in path[:-1]:
        node = node[key]
    if value is None:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    with pytest.raises(ConfigError, match=names):
        DarotarConfig.from_json(cfg)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_spec_asks_for_exactly_the_checkpoints_tensors(name):
    from hi_b200.config.registry import lookup
    from hi_b200.parts.model import Model

    cfg = CONFIGS[name]
    arch = lookup(cfg)
    assert arch.name == "darotar"
    model = Model(arch.build_spec(arch.parse_config(cfg, None)), torch.float32, "cpu")
    want = {arch.normalize_tensor_name(k): tuple(v.shape) for k, v in make_weights(cfg, 1).items()}
    have = {s.name: tuple(s.shape) for s in model.tensor_specs() if not s.optional}
    assert set(want) - {"head"} == set(have)
    assert all(want[k] == have[k] for k in have)
    assert model.graph_safe


def test_layers_share_a_cache_slot():
    from hi_b200.config.registry import lookup
    from hi_b200.parts.model import Model

    arch = lookup(DA_A)
    spec = arch.build_spec(arch.parse_config(DA_A, None))
    assert [e.cache for e in spec.schedule] == [0, 1, 0, 3, 4, 0]
    assert [e.writes_cache for e in spec.schedule] == [True, True, False, True, True, False]
    cs = Model(spec, torch.float32, "cpu").cache_specs
    assert sorted(cs) == [0, 1, 3, 4]
    assert cs[1].window == ("sliding", 40) and cs[3].window == ("sliding", 23) and cs[0].window is None
    assert not cs[0].values and cs[1].values and (cs[1].kv_heads, cs[1].head_dim) == (2, 16)
    bf = Model(arch.build_spec(arch.parse_config(DA_B, None)), torch.bfloat16, "cpu").cache_specs
    assert bf[1].head_dim == 128                                   # rows that the tensor-core kernels take


def test_the_query_rank_may_come_from_the_checkpoint(tmp_path):
    from hi_b200.config.registry import load_architecture

    cfg = copy.deepcopy(DA_D)
    write_model(str(tmp_path), cfg, 3)
    for layer in cfg["layers"]:
        layer["mixer"].pop("q_rank", None)
    import json

    (tmp_path / "config.json").write_text(json.dumps(cfg))
    arch, parsed, _raw = load_architecture(str(tmp_path))
    assert [getattr(l.mixer, "q_rank", None) for l in parsed.layers] == [None, 11, 13, None]
    arch.build_spec(parsed)


def test_frequency_table_of_a_linear_scaling():
    from hi_b200.parts.basic import exact_inverse_frequencies

    t = exact_inverse_frequencies(12, 321.0, {"factor": 3.0})
    want = plain.frequencies({"base": 321.0, "dims": 12, "scaling": {"factor": 3.0}})
    assert t.dtype.name == "float32" and max(abs(float(a) / b - 1) for a, b in zip(t, want)) < 1e-7


def test_parts_refuse_what_is_not_built():
    from hi_b200.parts.registry import BuildEnv, build
    from hi_b200.parts.spec import PartSpec

    env = BuildEnv(dtype=torch.float32, device=torch.device("cpu"), hidden_size=32)
    base = {"hidden_size": 32, "num_heads": 2, "num_kv_heads": 1, "head_dim": 16, "values": "keys"}
    for bad in ({"value_dim": 8}, {"conv": 3}, {"weights": "sigmoid"}, {"differential": 0.3}, {"output_gate": True}, {"values": "queries"}):
        with pytest.raises(ValueError):
            build("mixer", PartSpec("attention", {**base, **bad}), env, "x")


def test_inspect_runs_without_a_gpu(tmp_path, capsys):
    from hi_b200.cli import main

    write_model(str(tmp_path / "m"), DA_D, 3)
    assert main(["inspect", str(tmp_path / "m")]) == 0
    text = capsys.readouterr().out
    assert "normed_output" in text and "latent_attention" in text and "routed_experts" in text
