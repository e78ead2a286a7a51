"""Fofisun without a GPU: the plain implementation's mechanisms against closed forms and against each other, the
configuration reader, the ModelSpec the builder makes (parts, cache needs, tensor names, the order of layers), and the
cache manager's windows that keep the first tokens."""
import copy
import math

import pytest
import torch

import plain_fofisun as plain
from fofisun_configs import CONFIGS, FO_A, FO_C, FO_D, attention, config, dense, make_weights, moe, plain_logits

F64 = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


def _one_layer(layer, width=24, **kw):
    cfg = config(19, width, 1e-5, [layer], **kw)
    return cfg, {k: v.double() for k, v in make_weights(cfg, 3).items()}


# --------------------------------------------------------------------------- mechanisms of the plain model
def test_position_vectors():
    p = plain.position_vectors(50, 12)
    assert torch.equal(p[0], torch.tensor([0.0, 1.0] * 6, dtype=F64))
    assert math.isclose(float(p[7, 4]), math.sin(7 * 10000.0 ** (-4 / 12))) and math.isclose(float(p[7, 5]), math.cos(7 * 10000.0 ** (-4 / 12)))
    assert torch.allclose(p[:, 0::2] ** 2 + p[:, 1::2] ** 2, torch.ones(50, 6, dtype=F64))
    assert plain.position_vectors(3, 7).shape == (3, 7)


def test_convolution_reads_the_past_only():
    u, taps = rnd(9, 5, seed=1), rnd(5, 4, seed=2)
    y = plain.short_convolution(u, taps)
    assert torch.allclose(y[0], taps[:, 3] * u[0])
    assert torch.allclose(y[5], taps[:, 0] * u[2] + taps[:, 1] * u[3] + taps[:, 2] * u[4] + taps[:, 3] * u[5])
    u2 = u.clone()
    u2[6:] += 1.0
    assert torch.equal(plain.short_convolution(u2, taps)[:6], y[:6])


def test_a_window_keeps_its_first_tokens():
    see = plain.visible(12, {"size": 3, "keep_first": 2})
    assert see[9].nonzero().flatten().tolist() == [0, 1, 7, 8, 9]
    assert see[1].nonzero().flatten().tolist() == [0, 1] and see[0].nonzero().flatten().tolist() == [0]
    assert see[3].nonzero().flatten().tolist() == [0, 1, 2, 3]
    assert torch.equal(plain.visible(12, {"size": 3})[9].nonzero().flatten(), torch.tensor([7, 8, 9]))
    assert bool(plain.visible(6, None)[5].all())


def test_attention_mechanisms_each_matter():
    cfg, w = _one_layer(attention(4, 2, 8, 6, 0.5, 0.3, conv=3, window=6, keep=2))
    m = cfg["layers"][0]["mixer"]
    h = rnd(20, 24, seed=7)
    y = plain.attention(h, m, w, "l0.mix", 1e-5)
    h2 = h.clone()
    h2[9:] += 1.0
    assert torch.equal(plain.attention(h2, m, w, "l0.mix", 1e-5)[:9], y[:9])                       # causal
    h2 = h.clone()
    h2[5:10] += 1.0       # outside the window of 14 and 2 positions of convolution behind it, not among the kept tokens
    y2 = plain.attention(h2, m, w, "l0.mix", 1e-5)
    assert torch.allclose(y2[17:], y[17:], atol=1e-12) and not torch.allclose(y2[16], y[16])
    h2 = h.clone()
    h2[1] += 1.0                                                                                    # a kept token
    assert not torch.allclose(plain.attention(h2, m, w, "l0.mix", 1e-5)[19], y[19])
    for change in ({"diff": 0.2}, {"scale": 1.0}, {"mask": {"size": 6, "keep_first": 1}}, {"mask": {"size": 7, "keep_first": 2}}):
        assert not torch.allclose(plain.attention(h, {**m, **change}, w, "l0.mix", 1e-5)[12:], y[12:])
    for name in ("q.norm", "k.norm", "q.conv", "k.conv", "v.conv", "g", "lq1", "lk2"):
        w2 = dict(w)
        w2[f"l0.mix.{name}"] = w[f"l0.mix.{name}"] * 1.5
        assert not torch.allclose(plain.attention(h, m, w2, "l0.mix", 1e-5), y), name


def test_the_second_map_is_taken_off():
    """With equal maps the difference is (1 - lambda) times one map; its norm leaves only the sign and the direction."""
    cfg, w = _one_layer(attention(1, 1, 4, 6, 0.5, 0.3))
    m = cfg["layers"][0]["mixer"]
    w = dict(w)
    for n in "qk":
        w[f"l0.mix.{n}"] = torch.cat([w[f"l0.mix.{n}"][:4]] * 2)
    h = rnd(9, 24, seed=4)
    w["l0.mix.g"] = torch.full_like(w["l0.mix.g"], 0.0)           # the gate is one half everywhere
    w["l0.mix.o"] = torch.eye(24, 6, dtype=F64)
    lam = plain.map_factor(m, w, "l0.mix")
    q = plain.rms_norm(h @ w["l0.mix.q"][:4].T, w["l0.mix.q.norm"], 1e-5)
    k = plain.rms_norm(h @ w["l0.mix.k"][:4].T, w["l0.mix.k.norm"], 1e-5)
    a = plain.softmax_attention(q, k, h @ w["l0.mix.v"].T, 0.5, plain.visible(9, None))
    want = plain.rms_norm((1 - lam) * a, None, 1e-5) * 0.7 * 0.5
    assert torch.allclose(plain.attention(h, m, w, "l0.mix", 1e-5)[:, :6], want, atol=1e-12)
    w["l0.mix.lq1"] = torch.zeros(4, dtype=F64)
    w["l0.mix.lq2"] = torch.zeros(4, dtype=F64)
    assert math.isclose(plain.map_factor(m, w, "l0.mix"), 0.3)    # e^0 - e^0 + diff


def test_clamped_unit_and_mixture():
    cfg, w = _one_layer(attention(1, 1, 4, 6, 0.5, 0.3, mlp=moe(4, 2, 10, 0.8, shared=6, shared_limit=0.5)))
    mlp = cfg["layers"][0]["mlp"]
    h = 3.0 * rnd(11, 24, seed=5)
    g, u = h @ w["l0.mlp.e1.gate"].T, h @ w["l0.mlp.e1.up"].T
    assert float(g.max()) > 0.8 and float(u.min()) < -0.8 < 0.8 < float(u.max())            # every limit is reached
    act = torch.minimum(g, torch.tensor(0.8, dtype=F64))
    act = act / (1 + torch.exp(-1.702 * act)) * (u.clamp(-0.8, 0.8) + 1)
    assert torch.allclose(plain.clamped_unit(h, w, "l0.mlp.e1", 0.8), act @ w["l0.mlp.e1.down"].T)
    ids, z = plain.router_choice(h, mlp, w, "l0.mlp")
    y = plain.mixture(h, mlp, w, "l0.mlp")
    t = 6
    a, b = (int(i) for i in ids[t])
    wa = float(1 / (1 + torch.exp(z[t, b] - z[t, a])))                                       # softmax over the two chosen
    want = wa * plain.clamped_unit(h[t: t + 1], w, f"l0.mlp.e{a}", 0.8) + (1 - wa) * plain.clamped_unit(h[t: t + 1], w, f"l0.mlp.e{b}", 0.8)
    share = 1 / (1 + torch.exp(-(h[t: t + 1] @ w["l0.mlp.shared.sg"].T)))
    want = want + share * plain.clamped_unit(h[t: t + 1], w, "l0.mlp.shared", 0.5)
    assert torch.allclose(y[t: t + 1], want)
    w2 = dict(w)
    w2["l0.mlp.router.b"] = w["l0.mlp.router.b"].flip(0) * 3
    assert not torch.equal(plain.router_choice(h, mlp, w2, "l0.mlp")[0], ids)


def test_gelu_is_the_exact_one():
    z = torch.tensor([-3.0, -0.5, 0.0, 0.7, 2.0], dtype=F64)
    phi = torch.distributions.Normal(0.0, 1.0).cdf(z)
    assert torch.allclose(plain.gelu(z), z * phi, atol=1e-7)


def test_norms_before_and_after_each_sublayer():
    """With every norm1b / norm2b weight at -1 the sub-layers' results vanish and the stream stays the embedding."""
    cfg, w = CONFIGS["A"], {k: v.double() for k, v in make_weights(CONFIGS["A"], 1).items()}
    toks = [3, 5, 7, 9]
    for i in range(len(cfg["layers"])):
        w[f"l{i}.norm1b"] = torch.full_like(w[f"l{i}.norm1b"], -1.0)
        if f"l{i}.norm2b" in w:
            w[f"l{i}.norm2b"] = torch.full_like(w[f"l{i}.norm2b"], -1.0)
    streams = []
    logits = plain.forward(cfg, w, toks, streams=streams)
    x = plain.embedding(toks, w)
    assert len(streams) == 6 and all(torch.equal(s, x) for s in streams)
    assert torch.allclose(logits, plain.layer_norm(x, w["final.norm"], 1e-5) @ w["head"].T)


def test_looped_layers_are_layers_written_out():
    cfg = CONFIGS["A"]
    w = make_weights(cfg, 2)
    assert plain.layer_order(cfg) == [0, 1, 2, 1, 2, 3]
    flat = {k: v for k, v in cfg.items() if k != "loop"}
    flat["layers"] = [cfg["layers"][i] for i in plain.layer_order(cfg)]
    w2 = {k: v for k, v in w.items() if not k.startswith("l")}
    for run, i in enumerate(plain.layer_order(cfg)):
        w2.update({f"l{run}." + k.split(".", 1)[1]: v for k, v in w.items() if k.startswith(f"l{i}.")})
    toks = list(range(20))
    assert torch.allclose(plain_logits(cfg, w, toks), plain_logits(flat, w2, toks))


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
    from hi_b200.config.fofisun import FofisunConfig

    c = FofisunConfig.from_json(FO_A)
    a = c.layers[1]
    assert (c.vocab, c.width, c.eps) == (131, 64, 1e-5) and (c.loop.start, c.loop.stop, c.loop.times) == (1, 3, 2)
    assert (a.mixer.heads, a.mixer.kv_heads, a.mixer.dim, a.mixer.vdim, a.mixer.scale, a.mixer.diff, a.mixer.conv, a.mixer.window,
            a.mixer.keep_first) == (2, 1, 16, 32, 0.3, 0.4, 4, 23, 19)
    assert (a.mlp.experts, a.mlp.top, a.mlp.ff, a.mlp.limit, a.mlp.shared_ff, a.mlp.shared_limit) == (8, 2, 24, 1.2, 32, 0.9)
    assert c.layers[0].mlp.ff == 96
    d = FofisunConfig.from_json(FO_C)
    assert d.loop is None and d.layers[0].mixer.conv is None and d.layers[0].mixer.window is None and d.layers[1].mlp is None
    assert d.layers[0].mlp.shared_ff is None and d.layers[2].mixer.diff == 0.0


@pytest.mark.parametrize("path,value,names", [
    (("vocab",), None, "vocab"), (("norm", "eps"), None, "eps"), (("layers", 0, "type"), "mamba2", "type"),
    (("layers", 0, "mixer", "heads"), None, "heads"), (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "diff"), None, "diff"), (("layers", 0, "mixer", "conv"), 0, "conv"),
    (("layers", 0, "mixer", "mask", "size"), 0, "size"), (("layers", 0, "mixer", "mask", "keep_first"), -1, "keep_first"),
    (("layers", 0, "mlp", "kind"), "swiglu", "kind"), (("layers", 1, "mlp", "expert", "limit"), None, "limit"),
    (("layers", 1, "mlp", "router", "top"), 9, "top"), (("layers", 1, "mlp", "shared", "ff"), None, "ff"),
    (("loop", "times"), 0, "loop"), (("loop", "stop"), 5, "loop"), (("layers",), [], "layers")])
def test_reader_names_what_is_wrong(path, value, names):
    from hi_b200.config.base import ConfigError
    from hi_b200.config.fofisun import FofisunConfig

    cfg = copy.deepcopy(FO_A)
    node = cfg
    for key in path[:-1]:
        node = node[key]
    if value is None:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    with pytest.raises(ConfigError, match=names):
        FofisunConfig.from_json(cfg)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_spec_asks_for_exactly_the_checkpoints_tensors(name):
    from hi_b200.config.registry import lookup
    from hi_b200.parts.model import Model

    cfg = CONFIGS[name]
    arch = lookup(cfg)
    assert arch.name == "fofisun"
    model = Model(arch.build_spec(arch.parse_config(cfg, None)), torch.float32, "cpu")
    want = {arch.normalize_tensor_name(k): tuple(v.shape) for k, v in make_weights(cfg, 1).items()}
    have = {s.name: tuple(s.shape) for s in model.tensor_specs() if not s.optional}
    assert set(want) - {"head"} == set(have)
    assert all(want[k] == have[k] for k in have)


def test_every_run_of_a_layer_has_a_cache_of_its_own():
    from hi_b200.config.registry import lookup
    from hi_b200.parts.model import Model

    arch = lookup(FO_A)
    spec = arch.build_spec(arch.parse_config(FO_A, None))
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 1, 2, 3] and [e.cache for e in spec.schedule] == list(range(6))
    model = Model(spec, torch.float32, "cpu")
    cs = model.cache_specs
    assert cs[0].window == ("sliding", 40, 5) and cs[1].window == cs[3].window == ("sliding", 23, 19) and cs[5].window is None
    assert cs[0].keep_first == 5 and cs[5].keep_first == 0
    # the last taps - 1 projected values: q (heads x 2 x dim), k (kv_heads x 2 x dim), v (kv_heads x vdim)
    assert cs[0].state_shape == (2 * (4 * 32 + 2 * 32 + 2 * 24),) and cs[1].state_shape == (3 * (2 * 32 + 32 + 32),)
    assert (cs[0].kv_heads, cs[0].head_dim) == (2, 32)
    bf = Model(spec, torch.bfloat16, "cpu").cache_specs
    assert bf[0].head_dim == 64                                    # rows that the tensor-core kernels take
    c = Model(lookup(FO_C).build_spec(lookup(FO_C).parse_config(FO_C, None)), torch.float32, "cpu").cache_specs
    assert c[0].state_shape == () and c[1].state_shape == () and c[2].state_shape == (3 * (48 + 48 + 8),)


def test_attention_refuses_what_is_not_built():
    from hi_b200.parts.registry import BuildEnv, build
    from hi_b200.parts.spec import PartSpec

    env = BuildEnv(dtype=torch.float32, device=torch.device("cpu"), hidden_size=32)
    base = {"hidden_size": 32, "num_heads": 2, "num_kv_heads": 1, "head_dim": 16, "differential": 0.3}
    for bad in ({"sink": True}, {"softcap": 5.0}, {"weights": "sigmoid"}, {"temperature": (4.0, 0.5)}, {"qk_norm": True}):
        with pytest.raises(ValueError):
            build("mixer", PartSpec("attention", {**base, **bad}), env, "x")


def test_inspect_runs_without_a_gpu(tmp_path, capsys):
    from fofisun_configs import write_model
    from hi_b200.cli import main

    write_model(str(tmp_path / "m"), FO_D, 3)
    assert main(["inspect", str(tmp_path / "m")]) == 0
    text = capsys.readouterr().out
    assert "sandwich" in text and "attention" in text and "routed_experts" in text


# --------------------------------------------------------------------------- the cache manager keeps the first tokens
@pytest.mark.parametrize("page,window,keep", [(4, 6, 3), (4, 6, 4), (4, 6, 9), (8, 1, 1), (4, 16, 0), (16, 5, 40)])
def test_pages_of_kept_tokens_stay_and_the_rest_of_the_past_goes(page, window, keep):
    from hi_b200.cache.pages import FREED, CacheManager
    from hi_b200.parts.spec import CacheSpec

    spec = CacheSpec(kv_heads=1, head_dim=16, window=("sliding", window, keep))
    m = CacheManager([spec, CacheSpec(kv_heads=1, head_dim=16)], [64, 64], page, 2)
    m.open("a")
    done = 0
    for n in (1, 2, 7, 30, 1, 1, 1, 13, 1, 5):
        before = m.pages_needed("a", n)
        free = m.pools[0].free
        m.reserve("a", n)
        assert m.pools[0].free == free - before[0]
        table = m.table(0, "a")
        for pos in range(done + n):                       # everything a query of this step may read is there
            reads = pos < keep or any(0 <= q - pos < window for q in range(done, done + n))
            if reads:
                assert table[pos // page] != FREED, (pos, done, n)
        m.commit("a", n)
        done += n
        m.check_invariants()
        live = {b for b, p in enumerate(m.table(0, "a")) if p != FREED}
        want = {pos // page for pos in range(done) if pos < keep or pos >= max(0, done - window + 1)}
        want |= {b for b in range(-(-keep // page)) if b < len(m.table(0, "a"))}
        tail = {b for b in live if b * page >= done - page + 1}        # the block being written may be kept for the next token
        assert want - {done // page} <= live and live <= want | tail
    m.close("a")
    assert m.pools[0].free == 64 and m.pools[1].free == 64
    m.check_invariants()
    with pytest.raises(ValueError):
        CacheManager([CacheSpec(kv_heads=1, head_dim=16, window=("chunk", 8, 2))], [4], 4, 1)


def test_a_request_fits_by_its_window_and_its_kept_tokens():
    """A long request fits a pool that holds its window, its kept tokens and the page being written; one page less is
    refused when the request is added."""
    from hi_b200.cache.pages import CacheManager
    from hi_b200.engine.scheduler import Request, Scheduler, SchedulerConfig
    from hi_b200.parts.spec import CacheSpec
    from hi_b200.sampling import SamplingParams

    spec = CacheSpec(kv_heads=1, head_dim=16, window=("sliding", 16, 10))
    need = 3 + 4 + 1                                      # kept blocks, window, the page being written (pages of 4)
    for pages, ok in ((need, True), (need - 1, False)):
        sched = Scheduler(CacheManager([spec], [pages], 4, 2), SchedulerConfig(max_batch_size=2, max_batched_tokens=8))
        if ok:
            sched.add(Request("a", list(range(50)), SamplingParams(max_tokens=20)))
        else:
            with pytest.raises(Exception, match="insufficient_gpu_memory"):
                sched.add(Request("a", list(range(50)), SamplingParams(max_tokens=20)))
