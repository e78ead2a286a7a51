"""Darotar in the engine against the plain implementation: every mixer (its own latents and another layer's) and the
experts alone, whole prompts, decoding through the cache, portions down to two tokens, mixed batches with pages and slots
used again, planted keys far away, at page borders and on both sides of a window's edge, a sink that matters, a peaked
softmax, long decoding through captured steps, configurations of other sizes, generation through the entry point, the
trace replay and the command line."""
import numpy as np
import pytest
import torch

import harness as h
import plain_darotar as plain
from darotar_configs import CONFIGS, attention, config, latent, make_weights, peaked, plain_logits, write_model

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
# A position's error is the largest difference of its logits over the largest logit. The float32 runs are the sharp
# ones: rounding gives a few 1e-6 there, while a lost, doubled or shifted key, a sink left out or a norm in the wrong
# place moves the logits by a thousand times that. In bfloat16 these small models magnify rounding, so there the MEDIAN
# error of a comparison's positions is held to the tolerance and no position may be wildly off.
TOL = {"float32": 5e-5, "bfloat16": 6e-2}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    base = tmp_path_factory.mktemp("darotar")
    out = {}
    for name, cfg in CONFIGS.items():
        d = str(base / name)
        out[name] = (cfg, d, write_model(d, cfg, seed=60 + ord(name)))
    return out


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def engine(mdir, dtype, **kw):
    from hi_b200.engine.core import Engine

    kw.setdefault("kv_page_size", 16)
    kw.setdefault("kv_cache_tokens", 2048)
    kw.setdefault("max_active_requests", 4)
    return Engine.from_dir(mdir, dtype=dtype, **kw)


def compare(cfg, weights, requests, got, tol, what, forced=None):
    """Every wanted row against the plain model; names the first wrong token. ``forced``: the engine's own expert
    choices in a bfloat16 run (reduced precision may pick the other of two nearly equal logits; the logits are then
    compared given that choice)."""
    errs, over = [], []
    sharp = tol < 1e-3
    for rid, toks in requests.items():
        ref = plain_logits(cfg, weights, toks, forced=(forced or {}).get(rid))
        scale = float(ref.abs().max())
        rows = got.get(rid, {})
        assert rows, f"{what}: no logits came back for request {rid!r}"
        for p in sorted(rows):
            err = float(np.abs(rows[p].astype(np.float64) - ref[p].numpy()).max()) / scale
            assert np.isfinite(err), f"{what}: request {rid!r}, position {p}: not finite"
            assert err <= 8 * tol, f"{what}: request {rid!r} first differs at position {p} of {len(toks)}: rel err {err:.3e}"
            errs.append(err)
            if err > tol:
                over.append((rid, p, err))
    if sharp:
        # a norm over a handful of numbers that nearly cancel magnifies 32-bit rounding at single positions
        assert len(over) <= max(1, 0.02 * len(errs)), f"{what}: {len(over)} of {len(errs)} positions over {tol:.1e}; the first: {over[:3]}"
    else:
        assert float(np.median(errs)) <= tol, f"{what}: median error {float(np.median(errs)):.3e} of {len(errs)} positions"


def replay(eng, steps, dtype):
    got, forced = h.replay_in_process(eng, steps, record_routing=(dtype == "bfloat16"))
    return got, ({r: {k: v.long() for k, v in layers.items()} for r, layers in forced.items()} if dtype == "bfloat16" else None)


# --------------------------------------------------------------------------- every mixer and the experts alone
LAYERS = [pytest.param(name, i, id=f"{name}{i}") for name, cfg in CONFIGS.items() for i in range(len(cfg["layers"]))]


def _mixer_part(cfg, index, w, dt):
    from hi_b200.config.darotar import DarotarConfig
    from hi_b200.parts.darotar import build_darotar_spec
    from hi_b200.parts.registry import build
    from test_vinurax_engine import _env

    spec = build_darotar_spec(DarotarConfig.from_json(cfg)).layers[index].mixer
    part = build("mixer", spec, _env(dt, cfg["width"]), f"l{index}.mix")
    part.load(lambda name: w[name].to(DEV).to(dt) if name in w else None)
    return part


@pytest.mark.parametrize("dt,tol", [(torch.float32, 2e-5), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("name,index", LAYERS)
def test_mixer_alone(dt, tol, name, index):
    """Two requests in four steps (a portion each, a portion beside a single token, single tokens, a single token
    beside a portion) on scattered pages, against the plain mixer on the whole inputs. A layer that reads another's
    latents runs behind that layer, which has other inputs."""
    from hi_b200.parts.context import CacheView
    from test_vinurax_engine import _ctx

    cfg = CONFIGS[name]
    width, page, eps = cfg["width"], 8, cfg["norm"]["eps"]
    layer = cfg["layers"][index]
    w = make_weights(cfg, 5 + index)
    source = layer["mixer"].get("kv_from")
    part = _mixer_part(cfg, index, w, dt)
    writer = None if source is None else _mixer_part(cfg, source, w, dt)
    cs = part.cache_spec()
    pages = torch.full((12, cs.kv_heads, page, cs.head_dim), 50.0, dtype=dt, device=DEV)       # what others left there
    view = CacheView(group=0, writes=source is None, k_pages=pages, v_pages=pages.clone() if cs.values else None)
    table = torch.tensor([[7, 2, 9, 4, 6], [1, 11, 0, 5, 3]], dtype=torch.int32)
    g = torch.Generator().manual_seed(3)
    xs = [torch.randn(n, width, generator=g).to(dt).float() for n in (33, 29)]
    other = [torch.randn(n, width, generator=g).to(dt).float() for n in (33, 29)]
    cuts = [([13, 17], [0, 0]), ([18, 1], [13, 17]), ([1, 1], [31, 18]), ([1, 10], [32, 19])]
    got = [[], []]
    for lens, starts in cuts:
        rows = lambda t: torch.cat([t[i][s: s + n] for i, (n, s) in enumerate(zip(lens, starts))]).to(DEV).to(dt)
        if writer is not None:
            writer.forward(rows(other), _ctx(lens, starts, page, table, [1, 0]),
                           CacheView(group=0, writes=True, k_pages=pages))
        out = part.forward(rows(xs), _ctx(lens, starts, page, table, [1, 0]), view)
        a = 0
        for i, n in enumerate(lens):
            got[i].append(out[a: a + n].float().cpu())
            a += n
    wd = {k: v.double() for k, v in w.items()}
    for i in range(2):
        if layer["type"] == "attention":
            want = plain.attention(xs[i].double(), layer["mixer"], wd, f"l{index}.mix", eps)
        else:
            at = index if source is None else source
            c = plain.latents((xs if source is None else other)[i].double(), cfg["layers"][at]["mixer"], wd, f"l{at}.mix", eps)
            want = plain.latent_attention(xs[i].double(), layer["mixer"], wd, f"l{index}.mix", eps, c)
        have = torch.cat(got[i]).double()
        assert have.shape == want.shape
        errs = (have - want).abs().amax(dim=1) / want.abs().max()
        if dt == torch.float32:
            assert float(errs.max()) <= tol, f"request {i}: token {int(errs.argmax())}: rel err {float(errs.max()):.3e}"
        else:
            assert float(errs.median()) <= tol and float((errs > 8 * tol).float().mean()) <= 0.1, \
                f"request {i}: median rel err {float(errs.median()):.3e}, worst {float(errs.max()):.3e}"


@pytest.mark.parametrize("dt,tol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("name,index", [("A", 0), ("A", 1), ("A", 4), ("B", 0), ("B", 1), ("C", 1), ("C", 2), ("D", 0), ("D", 2), ("E", 0), ("E", 3)])
def test_experts_alone(dt, tol, name, index):
    """The routed feed-forward with the engine's own choice of experts handed to the plain mixture: 3 and 150 tokens
    (the few-rows and the many-rows kernels). The router reads float32 rows, the experts their rounding."""
    from hi_b200.config.darotar import DarotarConfig
    from hi_b200.parts.context import Pending
    from hi_b200.parts.darotar import build_darotar_spec
    from hi_b200.parts.registry import build
    from test_vinurax_engine import _ctx, _env

    cfg = CONFIGS[name]
    width, mlp = cfg["width"], cfg["layers"][index]["mlp"]
    w = make_weights(cfg, 11)
    spec = build_darotar_spec(DarotarConfig.from_json(cfg)).layers[index].feed_forward
    part = build("feed_forward", spec, _env(dt, width), f"l{index}.mlp")
    part.load(lambda n: w[n].to(DEV).to(dt) if n in w else None)
    wd = {k: v.double() for k, v in w.items()}
    for n in (3, 150):
        x = torch.randn(n, width, generator=torch.Generator().manual_seed(n))
        taps = {}
        ctx = _ctx([n], [0], 8, torch.zeros((1, 32), dtype=torch.int32), [0])
        ctx.tap = lambda k, t: taps.__setitem__(k, t.clone())
        out = part.forward(x.to(DEV).to(dt), ctx, normed_f32=x.to(DEV))
        assert isinstance(out, Pending)
        have = out.materialize(n).double().cpu()
        ids = taps[f"l{index}.mlp.router_ids"].long().cpu()
        own, _s = plain.router_choice(x.double(), mlp, wd, f"l{index}.mlp")
        assert (own.sort(-1).values == ids.sort(-1).values).all()
        want = plain.mixture(x.double(), mlp, wd, f"l{index}.mlp", forced_ids=ids)
        err = float((have - want).abs().max() / want.abs().max())
        assert err <= tol, f"{n} tokens: rel err {err:.3e}"


@pytest.mark.parametrize("name", ["A", "D"])
def test_the_stream_after_every_layer(name, models):
    """Layer by layer in 32-bit: what every layer reads is the plain model's stream."""
    from hi_b200.engine.core import StepEntry

    cfg, mdir, weights = models[name]
    toks = tokens(cfg, 60, 9)
    seen = []
    eng = engine(mdir, "float32")
    eng.step([StepEntry("a", toks, [59])], tap=lambda n, t: seen.append((n, t.double().cpu())) if n.endswith("stream_in") else None)
    wd, streams = {k: v.double() for k, v in weights.items()}, []
    plain.forward(cfg, wd, toks, streams=streams)
    assert [n for n, _t in seen] == [f"l{i}.stream_in" for i in range(len(cfg["layers"]))]
    for (n, t), want in zip(seen, [wd["embed"][toks]] + streams):
        assert float((t - want).abs().max() / want.abs().max()) < 5e-6, n


# --------------------------------------------------------------------------- the model in the engine
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_four_ways_of_cutting(name, dtype, models):
    cfg, mdir, weights = models[name]
    requests = {"p": tokens(cfg, 150, 1), "q": tokens(cfg, 37, 2), "r": tokens(cfg, 1, 3), "s": tokens(cfg, 2, 4),
                "t": tokens(cfg, 64, 5), "u": tokens(cfg, 97, 6)}
    eng = engine(mdir, dtype, kv_cache_tokens=352, debug_poison=True)
    prompt = {r: min(len(t), max(2, len(t) - 24)) for r, t in requests.items()}      # the rest is decoded token by token
    for what, steps in (("whole", h.trace_whole(requests)), ("decode", h.trace_tail_decode(requests, tail=20)),
                        ("portions", h.trace_portions(requests)),
                        ("mixed", h.trace_mixed(requests, max_tokens=352, page=16, seed=7, max_live=4, prefill_len=prompt))):
        got, forced = replay(eng, steps, dtype)
        compare(cfg, weights, requests, got, TOL[dtype], f"{name} {dtype} {what}", forced)
    assert len(eng.manager.requests) == 0


@pytest.mark.parametrize("name", ["A", "D"])
def test_mixed_batches_use_pages_and_slots_again(name, models):
    """More requests than slots and than the pool holds at once, in two orders: every request's logits equal the
    plain model's whatever ran beside it and whichever pages and slot it got."""
    cfg, mdir, weights = models[name]
    requests = {i: tokens(cfg, n, 30 + i) for i, n in enumerate((70, 33, 48, 5, 90, 17, 64, 31, 2, 55))}
    for seed, live in ((1, 4), (2, 2)):
        eng = engine(mdir, "float32", kv_cache_tokens=272, max_active_requests=live, debug_poison=True)
        steps = h.trace_mixed(requests, max_tokens=272, page=16, seed=seed, max_live=live)
        got, _ = h.replay_in_process(eng, steps)
        compare(cfg, weights, requests, got, TOL["float32"], f"{name} mixed seed {seed}")
        assert eng.manager.snapshot()["groups"][0]["allocations"] > 272 // 16      # pages were handed out again


@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_far_keys_and_window_edges_under_a_peaked_softmax(name, models, tmp_path):
    """Softmax scales times 6: nearly all weight on one key, so a key that is lost, doubled or shifted shows (the
    oldest key of a window, the one just outside it, a key hundreds of tokens back). The peaked scores magnify
    float32 rounding too, so the bound is 1e-3; a wrong key moves these logits by tenths."""
    cfg = peaked(CONFIGS[name], 6.0)
    mdir = str(tmp_path / "peaked")
    weights = write_model(mdir, cfg, seed=77)
    requests = {"long": tokens(cfg, 300, 8), "short": tokens(cfg, 90, 9)}
    eng = engine(mdir, "float32", kv_cache_tokens=1024)
    for what, steps in (("whole", h.trace_whole(requests)), ("decode", h.trace_tail_decode(requests, tail=60)),
                        ("portions", h.trace_portions(requests, sizes=(100, 3, 61, 2, 29, 17, 2, 50, 5))),
                        ("mixed", h.trace_mixed(requests, max_tokens=1024, page=16, seed=3, max_live=2))):
        got, _ = h.replay_in_process(eng, steps)
        compare(cfg, weights, requests, got, 9.9e-4, f"{name} peaked {what}")


WINDOW = 48


def _planted_embedding(w):
    """Token 1 asks, token 2 answers; both stand out in single dims that the mixer's maps read. A large eps keeps what is
    small small in every norm."""
    emb = 0.05 * torch.randn(16, 32, generator=torch.Generator().manual_seed(1))
    emb[:, :4] = 0.0
    emb[1, 0], emb[2, 1] = 24.0, 24.0
    w["embed"] = emb
    w["l0.norm1"] = torch.full((32,), 3.0)


def _planted_attention(window):
    """One attention layer made so that the last token's query matches one earlier token's key, which is the only value
    that is not zero; the match lies in a dim that does not turn."""
    cfg = config(16, 32, 1.0, [attention(1, 1, 16, 0.5, 100.0, dims=4, factor=2.0, window=window)], mult=0.9)
    w = make_weights(cfg, 9)
    _planted_embedding(w)
    w["l0.mix.q"], w["l0.mix.k"] = torch.zeros(16, 32), torch.zeros(16, 32)
    w["l0.mix.q"][12, 0] = 1.0
    w["l0.mix.k"][12, 1] = 1.0
    return cfg, {k: v.to(torch.bfloat16).float() for k, v in w.items()}


def _planted_latent(sink=1.0):
    """The same with one latent-attention layer: the answering token's latent is the only one that is not zero."""
    cfg = config(16, 32, 1.0, [latent(1, 8, 4, 8, 8, 8, 1.2, 100.0)], mult=0.9)
    w = make_weights(cfg, 9)
    _planted_embedding(w)
    for nme in ("dq", "uq", "dkv", "uk"):
        w[f"l0.mix.{nme}"] = torch.zeros_like(w[f"l0.mix.{nme}"])
    w["l0.mix.dq"][0, 0] = w["l0.mix.uq"][0, 0] = w["l0.mix.dkv"][0, 1] = w["l0.mix.uk"][0, 0] = 1.0
    w["l0.mix.dq.norm"] = w["l0.mix.dkv.norm"] = torch.ones(8)
    w["l0.mix.g"] = torch.zeros(8, 32)
    w["l0.mix.sink"] = torch.tensor([sink])
    return cfg, {k: v.to(torch.bfloat16).float() for k, v in w.items()}


def _check_planted(tmp_path, cfg, w, toks, without, seen, what, tail):
    ref, ref_without = plain_logits(cfg, w, toks)[-1], plain_logits(cfg, w, without)[-1]
    moved = float((ref - ref_without).abs().max()) / float(ref.abs().max())
    assert moved > 0.05 if seen else moved < 1e-9, (what, moved)
    mdir = str(tmp_path / "planted")
    write_model(mdir, cfg, 0, weights=w)
    n = len(toks)
    for how, steps in (("whole", h.trace_whole({"a": toks})), ("decode", h.trace_tail_decode({"a": toks}, tail=tail)),
                       ("portions", h.trace_portions({"a": toks}, sizes=(15, 2, 1, 7, n - 60, 2, 4, 9, 3)))):
        for dtype in ("float32", "bfloat16"):
            got, _ = replay(engine(mdir, dtype, kv_cache_tokens=512), steps, "float32")
            compare(cfg, w, {"a": toks}, got, TOL[dtype], f"{what} {how} {dtype}")
            have = torch.from_numpy(got["a"][n - 1]).double()
            if seen:        # the answer is there, also under bfloat16's rounding
                assert float((have - ref).abs().max()) < 0.3 * float((have - ref_without).abs().max()), f"{what} {how} {dtype}"


@pytest.mark.parametrize("kind", ["attention", "latent"])
@pytest.mark.parametrize("where", [0, 1, 15, 16, 17, 255, 256, 300])
def test_a_planted_key_far_away_and_at_page_borders(where, kind, tmp_path):
    """No window; the answering token at the sequence's first places, on both sides of a page's border and hundreds of
    tokens back."""
    cfg, w = _planted_attention(None) if kind == "attention" else _planted_latent()
    toks = [3 + (i % 11) for i in range(400)]
    toks[where], toks[-1] = 2, 1
    without = list(toks)
    without[where] = 3
    _check_planted(tmp_path, cfg, w, toks, without, True, f"planted key at {where}", tail=3)


@pytest.mark.parametrize("back", [1, WINDOW - 2, WINDOW - 1, WINDOW, WINDOW + 1, 3 * WINDOW])
def test_a_planted_key_on_both_sides_of_the_window_edge(back, tmp_path):
    """Read while back < window, and not at all from there on; also after decoded tokens have moved the window over it."""
    cfg, w = _planted_attention(WINDOW)
    n = 200
    toks = [3 + (i % 11) for i in range(n)]
    toks[-1], toks[n - 1 - back] = 1, 2
    without = list(toks)
    without[n - 1 - back] = 3
    _check_planted(tmp_path, cfg, w, toks, without, back < WINDOW, f"planted key {back} back", tail=60)


def test_the_sink_takes_its_share(tmp_path):
    """The planted latent again with a sink that outweighs the planted key: the read-out shrinks in the plain model, and
    the engine follows it."""
    toks = [3 + (i % 11) for i in range(60)]
    toks[20], toks[-1] = 2, 1
    small = plain_logits(*_planted_latent(), toks)[-1]
    cfg, w = _planted_latent(sink=30.0)
    large = plain_logits(cfg, w, toks)[-1]
    assert float((small - large).abs().max()) > 0.05 * float(small.abs().max())
    mdir = str(tmp_path / "sink")
    write_model(mdir, cfg, 0, weights=w)
    for steps in (h.trace_whole({"a": toks}), h.trace_tail_decode({"a": toks}, tail=3)):
        got, _ = h.replay_in_process(engine(mdir, "float32", kv_cache_tokens=128), steps)
        compare(cfg, w, {"a": toks}, got, 5e-5, "a sink that outweighs the keys")


def test_long_decoding_and_first_tokens(models):
    """300 tokens decoded one by one after a two-token prompt (captured steps), beside a request that starts
    later; positions 0 and 1 are compared too."""
    cfg, mdir, weights = models["A"]
    requests = {"a": tokens(cfg, 300, 11), "b": tokens(cfg, 120, 12)}
    for dtype in ("float32", "bfloat16"):
        eng = engine(mdir, dtype)
        steps = [([("a", requests["a"][:2], [0, 1])], [])]
        for i in range(2, 300):
            entries = [("a", [requests["a"][i]], [0])]
            j = i - 100
            if 0 <= j < 120:
                entries.append(("b", [requests["b"][j]], [0]))
            steps.append((entries, [r for r, n in (("a", 299), ("b", 219)) if i == n]))
        got, forced = replay(eng, steps, dtype)
        compare(cfg, weights, requests, got, TOL[dtype], f"long decoding {dtype}", forced)
        assert len(eng._graphs) >= 1 and any(g.captured for g in eng._graphs.values())


def test_other_page_sizes_and_kernel_choices(models):
    """Page sizes 8 and 64; in bfloat16 rows of 64 and 128 go through the tensor-core attention kernels with pages of 64
    (single tokens, short portions, portions of a tile and more)."""
    from hi_b200.kernels import ops

    for name in ("A", "B"):
        cfg, mdir, weights = models[name]
        requests = {"x": tokens(cfg, 333, 14), "y": tokens(cfg, 40, 15)}
        for page in (8, 64):
            before = dict(ops.CALLS)
            eng = engine(mdir, "bfloat16", kv_page_size=page, kv_cache_tokens=1024)
            for steps in (h.trace_whole(requests), h.trace_tail_decode(requests, tail=8),
                          h.trace_portions(requests, sizes=(140, 5, 2, 150, 30))):
                got, forced = replay(eng, steps, "bfloat16")
                compare(cfg, weights, requests, got, TOL["bfloat16"], f"{name} page {page}", forced)
            used = {k for k, v in ops.CALLS.items() if v > before.get(k, 0)}
            every = {"sandwich_step", "qkv_post", "latent_append", "rmsnorm_rows", "rope_copy", "gate_rows", "attention_decode",
                     "attention_prefill", "router_plan", "moe_gate_up_tc"} | ({"attention_prefill_tc"} if page == 64 else set())
            assert all(any(k.startswith(w) for k in used) for w in every), (sorted(every), sorted(used))


def test_long_portions_beside_single_tokens(models):
    """Portions of a tile of new tokens and more (the tcgen05 kernel) in one step with single decoded tokens of other
    requests (the decode kernel), pages of 64."""
    cfg, mdir, weights = models["B"]
    requests = {"a": tokens(cfg, 420, 31), "b": tokens(cfg, 200, 32), "c": tokens(cfg, 170, 33)}
    a, b, c = requests["a"], requests["b"], requests["c"]
    steps = [([("b", b[:60], list(range(60)))], []),
             ([("a", a[:150], list(range(150))), ("b", b[60:61], [0])], []),
             ([("a", a[150:300], list(range(150))), ("b", b[61:62], [0]), ("c", c[:129], list(range(129)))], []),
             ([("b", b[62:200], list(range(138))), ("a", a[300:301], [0]), ("c", c[129:130], [0])], ["b"]),
             ([("a", a[301:420], list(range(119))), ("c", c[130:170], list(range(40)))], ["a", "c"])]
    for dtype in ("float32", "bfloat16"):
        eng = engine(mdir, dtype, kv_page_size=64, kv_cache_tokens=1024)
        got, forced = replay(eng, steps, dtype)
        compare(cfg, weights, requests, got, TOL[dtype], f"long portions beside single tokens {dtype}", forced)


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_greedy_generation_through_the_entry_point(name, models):
    """hi_b200.generate (scheduler, sampler, launch-ahead) against greedy decoding of the plain model."""
    import hi_b200

    cfg, mdir, weights = models[name]
    prompts = [tokens(cfg, n, 40 + n) for n in (9, 1, 30, 17, 5)]
    outs = hi_b200.generate(mdir, prompts, hi_b200.SamplingParams(max_tokens=10, ignore_eos=True), dtype="float32",
                            kv_page_size=16, max_batch_size=3, kv_cache_tokens=512, max_batched_tokens=24)
    for prompt, out in zip(prompts, outs):
        assert len(out.token_ids) == 10
        ref = plain_logits(cfg, weights, list(prompt) + list(out.token_ids))
        for k, tok in enumerate(out.token_ids):
            logits = ref[len(prompt) - 1 + k]
            top2 = torch.topk(logits, 2).values
            if float(top2[0] - top2[1]) > 1e-3 * float(logits.abs().max()):
                assert tok == int(logits.argmax()), f"prompt of {len(prompt)}: token {k} is {tok}, plain model says {int(logits.argmax())}"


def test_trace_replay_as_a_user_runs_it(models, tmp_path):
    for name, dtype, seed in (("D", "float32", 5), ("A", "float32", 6)):
        cfg, mdir, weights = models[name]
        requests = {"a": tokens(cfg, 80, 21), "b": tokens(cfg, 33, 22), "c": tokens(cfg, 3, 23), "d": tokens(cfg, 50, 24),
                    "e": tokens(cfg, 20, 25)}
        steps = h.trace_mixed(requests, max_tokens=192, page=64, seed=seed, max_live=4)
        got = h.replay_subprocess(mdir, dtype, steps, max_tokens=192, out_dir=str(tmp_path / name), vocab=cfg["vocab"],
                                  extra=["--max-live", "4"])
        compare(cfg, weights, requests, got, TOL[dtype], f"trace_run {name} {dtype}")


def test_command_line_run(models, capsys):
    """``python -m hi_b200 run``: the next token, the top logits and greedy generation of a Darotar folder."""
    import json

    from hi_b200.cli import main

    cfg, mdir, weights = models["D"]
    prompt = tokens(cfg, 12, 50)
    assert main(["run", mdir, "--tokens", ",".join(map(str, prompt)), "--max-tokens", "5", "--top-k", "3",
                 "--dtype", "float32", "--kv-page-size", "16", "--include-logits"]) == 0
    report = json.loads(capsys.readouterr().out)
    ref = plain_logits(cfg, weights, prompt)[-1]
    assert report["next_token"] == int(ref.argmax()) and report["logit_count"] == cfg["vocab"]
    assert float((torch.tensor(report["logits"], dtype=torch.float64) - ref).abs().max()) <= 3e-5 * float(ref.abs().max())
    assert [t["token_id"] for t in report["top_logits"]] == torch.topk(ref, 3).indices.tolist()
    assert len(report["generated_tokens"]) == 5 and report["generated_tokens"][0] == report["next_token"]
