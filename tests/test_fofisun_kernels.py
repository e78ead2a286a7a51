"""The kernels that Fofisun brought or extended, each against the same arithmetic in plain PyTorch (float64 on the CPU):
convolution of the projected q, k, v with norms and append, attention with kept first tokens in every kernel, the two maps'
difference with norm and gate (merged from split partials, and inside the tcgen05 prefill kernel), the sandwich boundary,
sinusoidal positions, gelu, the clamped unit (dense, and in the experts' products), the router's bias."""
import math

import pytest
import torch

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


def rnd(*shape, seed=0, std=1.0):
    return std * torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def close(got, want, tol):
    got, want = got.detach().double().cpu(), want.double()
    assert got.shape == want.shape, (got.shape, want.shape)
    assert bool(torch.isfinite(got).all())
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))
    assert err <= tol, f"rel err {err:.3e} > {tol:.1e}"


def ops():
    from hi_b200.kernels import ops as o

    return o


# --------------------------------------------------------------------------- small kernels
@pytest.mark.parametrize("width", [192, 51, 2, 1030])
def test_embedding_with_positions(width):
    table = rnd(40, width, seed=1)
    toks = torch.tensor([0, 39, 7, 7, 12], dtype=torch.int32)
    pos = torch.tensor([0, 1, 17, 4099, 1_000_003], dtype=torch.int32)
    f = torch.tensor([10000.0 ** (-2.0 * (c // 2) / width) for c in range(width)], dtype=F64)
    angle = pos.double()[:, None] * f
    want = 0.5 * table[toks.long()].double() + torch.where(torch.arange(width) % 2 == 0, torch.sin(angle), torch.cos(angle))
    turns = (f[0::2] / (2 * math.pi)).contiguous().to(DEV)
    got = ops().embed_position(table.to(DEV), toks.to(DEV), pos.to(DEV), turns, scale=0.5)
    assert float((got.double().cpu() - want).abs().max()) < 2e-6       # also a million positions on


@pytest.mark.parametrize("dt,tol", [(torch.float32, 1e-6), (torch.bfloat16, 8e-3)])
def test_gelu_and_clamped_unit(dt, tol):
    o = ops()
    for n in (7, 4096):
        x = rnd(n, seed=2, std=2.0).to(dt)
        xd = x.double()
        close(o.gelu(x.to(DEV)), 0.5 * xd * (1 + torch.erf(xd / math.sqrt(2))), tol)
    for rows, inter, pad, col in ((5, 24, 8, True), (33, 256, 8, True), (4, 9, 1, True), (700, 64, 0, False), (3, 10, 0, False)):
        x = rnd(rows, 2 * inter + pad, seed=rows, std=1.5).to(dt)
        xd = x.double()
        g, u = xd[:, :inter].clamp(max=0.9), xd[:, inter: 2 * inter].clamp(-0.9, 0.9)
        want = g * torch.sigmoid(1.702 * g) * (u + 1)
        if col:
            want = want * torch.sigmoid(xd[:, 2 * inter: 2 * inter + 1])
        close(o.glu_limit(x.to(DEV), inter, 0.9, 2 * inter if col else -1), want, tol)


@pytest.mark.parametrize("width", [64, 51, 2048, 4096, 8192, 8196])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_sandwich_step(width, dt):
    o = ops()
    n, k = 9, 3
    tol = 3e-6 if dt == torch.float32 else 8e-3
    for routed, delta2, rows in ((False, False, False), (True, False, False), (True, True, True), (False, True, True)):
        x, d = rnd(n, width, seed=1, std=3.0), rnd(n, width, seed=2).to(dt)
        d2 = rnd(n, width, seed=5).to(dt) if delta2 else None
        wy, w = 1 + 0.3 * rnd(width, seed=3), 1 + 0.3 * rnd(width, seed=4)
        y = d.double() + (d2.double() if delta2 else 0)
        kw = {}
        if routed:
            r, slot = rnd(n * k, width, seed=6), torch.randperm(n * k, generator=torch.Generator().manual_seed(1))
            f = rnd(n * k, seed=7).abs()
            y = y + (r[slot].double() * f.double()[:, None]).view(n, k, width).sum(1)
            kw = dict(routed=r.to(DEV), slot_of_entry=slot.to(torch.int32).to(DEV), top_k=k, routed_weight=f.to(DEV))
        rm = lambda t, e: t / torch.sqrt((t * t).mean(-1, keepdim=True) + e)
        xs = x.double() + rm(y, 1e-5) * wy.double()
        h = rm(xs, 1e-6) * w.double()
        row_map = torch.tensor([4, 0, 8], dtype=torch.int32) if rows else None
        xd = x.to(DEV)
        got = o.sandwich_step(xd, wy.to(DEV), 1e-5, delta=d.to(DEV), delta2=None if d2 is None else d2.to(DEV), weight=w.to(DEV), eps=1e-6,
                              out_dtype=dt, row_map=None if row_map is None else row_map.to(DEV), also_f32=True, **kw)
        sel = row_map.long() if rows else slice(None)
        close(got[0], h[sel], tol)
        close(got[1], h[sel], 3e-6)
        close(xd, x.double() if rows else xs, 3e-6)
        if not rows:
            xd = x.to(DEV)
            assert o.sandwich_step(xd, wy.to(DEV), 1e-5, delta=d.to(DEV), delta2=None if d2 is None else d2.to(DEV), **kw) is None
            close(xd, xs, 3e-6)


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,experts,top,hidden,inter", [(3, 4, 2, 64, 32), (150, 5, 3, 72, 40), (200, 17, 2, 256, 128), (30, 8, 1, 51, 9)])
def test_experts_with_limits_and_router_bias(dt, n, experts, top, hidden, inter):
    """Router with a bias, softmax over the chosen logits, and the clamped unit in the few-rows, general and tcgen05 products."""
    o = ops()
    x, wr, b = rnd(n, hidden, seed=1), rnd(experts, hidden, seed=2, std=hidden ** -0.5), rnd(experts, seed=3)
    mode = o.ROUTER_SOFTMAX | o.ROUTER_RENORMALIZE
    ids, scores, plan = o.router_plan(x.to(DEV), wr.to(DEV), top, mode, bias=b.to(DEV))
    z = x.double() @ wr.double().T + b.double()
    want = torch.topk(z, top, dim=-1)
    order = ids.long().cpu()
    assert (order.sort(-1).values == want.indices.sort(-1).values).all()
    close(scores, torch.softmax(torch.gather(z, 1, order), -1), 2e-6)
    limit = 0.7
    xb = x.to(dt)
    wg, wu = (rnd(experts, inter, hidden, seed=s, std=1.5 * hidden ** -0.5).to(dt) for s in (4, 5))
    ones = torch.ones(n, top)
    xd, e = xb.double()[:, None, :].expand(n, top, hidden), order
    g = torch.einsum("ntk,ntik->nti", xd, wg.double()[e]).clamp(max=limit)
    u = torch.einsum("ntk,ntik->nti", xd, wu.double()[e]).clamp(-limit, limit)
    act = (g * torch.sigmoid(1.702 * g) * (u + 1)).reshape(n * top, inter)
    slot = plan.slot_of_entry.long().cpu()
    want_rows = torch.empty_like(act)
    want_rows[slot] = act
    tol = 5e-6 if dt == torch.float32 else 1e-2
    for few in (True, False):
        close(o.moe_gate_up(xb.to(DEV), plan, top, wg.to(DEV), wu.to(DEV), ones.to(DEV), few, "clamped", limit), want_rows, tol)
    if o.moe_tc_supported(xb.to(DEV), wu.to(DEV)):
        close(o.moe_gate_up_tc(xb.to(DEV), plan, top, wg.to(DEV), wu.to(DEV), ones.to(DEV), limit), want_rows, tol)
        o.check_tc_status()


# --------------------------------------------------------------------------- convolution, norms, append
def _pages(n_pages, nkv, page, hd, dt):
    return torch.full((n_pages, nkv, page, hd), 7.0, dtype=dt, device=DEV)


@pytest.mark.parametrize("dt,tol", [(torch.float32, 2e-6), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("heads,kvh,maps,dim,vdim,hd,taps,rot", [
    (4, 2, 2, 16, 24, 64, 3, None), (2, 1, 2, 64, 128, 128, 4, None), (3, 3, 2, 10, 6, 32, 5, None), (16, 2, 2, 64, 128, 128, 4, None),
    (4, 2, 1, 32, 32, 32, 2, None), (4, 1, 1, 32, 24, 32, 4, (16, False)), (2, 2, 2, 12, 24, 32, 3, (6, True)), (2, 1, 2, 16, 32, 32, None, None),
    (2, 1, 2, 16, 32, 64, 1, None), (5, 5, 2, 128, 256, 256, 4, None)])
def test_conv_qkv(dt, tol, heads, kvh, maps, dim, vdim, hd, taps, rot):
    """Three requests in steps of portions and of single tokens; pages, state rows and queries against the whole sequences."""
    o = ops()
    page = 8
    channels = (heads + kvh) * maps * dim + kvh * vdim
    width = -(-channels // 8) * 8 + 16
    lens = (45, 9, 30)
    projs = [rnd(n, width, seed=20 + i).to(dt) for i, n in enumerate(lens)]
    w = 0.6 * rnd(channels, taps, seed=3) if taps else None
    qn, kn = 1 + 0.3 * rnd(dim, seed=4), 1 + 0.3 * rnd(dim, seed=5)
    inv = torch.tensor([100.0 ** (-2.0 * j / (2 * rot[0])) for j in range(rot[0])]) if rot else None
    state = torch.zeros(4, (taps - 1) * channels, device=DEV) if taps and taps > 1 else None
    k_pages, v_pages = _pages(20, kvh, page, hd, dt), _pages(20, kvh, page, hd, dt)
    table = torch.randperm(20, generator=torch.Generator().manual_seed(9))[:18].view(3, 6).to(torch.int32)
    slots = [3, 0, 2]
    got_q = [[], [], []]
    done = [0, 0, 0]
    # many rows at once (several rows a thread), odd portions, single tokens alone and beside portions
    for step in ([(0, 33), (2, 20)], [(0, 2), (1, 3), (2, 1)], [(0, 1), (1, 1), (2, 1)], [(0, 1), (1, 1), (2, 1)], [(0, 8), (1, 4), (2, 7)]):
        seqs = [s for s, _n in step]
        x = torch.cat([projs[s][done[s]: done[s] + n] for s, n in step]).to(DEV)
        pos = torch.cat([torch.arange(done[s], done[s] + n) for s, n in step]).to(torch.int32).to(DEV)
        sot = torch.cat([torch.full((n,), i) for i, (_s, n) in enumerate(step)]).to(torch.int32).to(DEV)
        cu = torch.tensor([0] + torch.tensor([n for _s, n in step]).cumsum(0).tolist(), dtype=torch.int32, device=DEV)
        sl = torch.tensor([slots[s] for s in seqs], dtype=torch.int32, device=DEV)
        q = o.conv_qkv(x, None if w is None else w.t().contiguous().to(DEV), state, True, 1e-5, qn.to(DEV), kn.to(DEV),
                       None if inv is None else inv.to(DEV), bool(rot and rot[1]), 1.2 if rot else 1.0, pos, sot, cu, sl,
                       table[seqs].contiguous().to(DEV), k_pages, v_pages, True, all(n == 1 for _s, n in step), heads, kvh, maps,
                       dim, vdim)
        at = 0
        for s, n in step:
            got_q[s].append(q[at: at + n].cpu())
            at += n
            done[s] += n
    assert tuple(done) == lens
    for s, n in enumerate(lens):
        u = projs[s].double()[:, :channels]
        if w is not None:
            padded = torch.cat([torch.zeros(taps - 1, channels, dtype=F64), u])
            u = sum(padded[j: j + n] * w.double()[:, j] for j in range(taps))
        nq, nk = heads * maps * dim, kvh * maps * dim

        def encode(t, weight):
            t = t / torch.sqrt((t * t).mean(-1, keepdim=True) + 1e-5) * weight.double()
            if inv is None:
                return t
            a = torch.arange(n, dtype=F64)[:, None] * inv.double()
            c, sn = (1.2 * torch.cos(a))[:, None, None], (1.2 * torch.sin(a))[:, None, None]
            out, p = t.clone(), rot[0]
            lo, hi = (t[..., 0: 2 * p: 2], t[..., 1: 2 * p: 2]) if rot[1] else (t[..., :p], t[..., p: 2 * p])
            ra, rb = lo * c - hi * sn, hi * c + lo * sn
            if rot[1]:
                out[..., 0: 2 * p: 2], out[..., 1: 2 * p: 2] = ra, rb
            else:
                out[..., :p], out[..., p: 2 * p] = ra, rb
            return out

        qs, ks = encode(u[:, :nq].view(n, heads, maps, dim), qn), encode(u[:, nq: nq + nk].view(n, kvh, maps, dim), kn)
        vs = u[:, nq + nk:].view(n, kvh, vdim)
        want_q = torch.zeros(n, heads, maps, hd, dtype=F64)
        want_k, want_v = torch.zeros(n, kvh, hd, dtype=F64), torch.zeros(n, kvh, hd, dtype=F64)
        for m in range(maps):
            want_q[:, :, m, m * dim: (m + 1) * dim] = qs[:, :, m]
            want_k[:, :, m * dim: (m + 1) * dim] = ks[:, :, m]
        want_v[..., :vdim] = vs
        close(torch.cat(got_q[s]), want_q.view(n, heads * maps, hd), tol)
        rows = [(int(table[s, p // page]), p % page) for p in range(n)]
        close(torch.stack([k_pages[a, :, b] for a, b in rows]), want_k, tol)
        close(torch.stack([v_pages[a, :, b] for a, b in rows]), want_v, tol)
        if state is not None:
            close(state[slots[s]], projs[s].double()[n - taps + 1:, :channels].reshape(-1), 1e-7)


# --------------------------------------------------------------------------- attention with kept first tokens, two maps
def _attention_case(dt, nh, nkv, hd, page, lens, starts, seed):
    """Random keys and values of several requests on scattered pages; pages that a window of 1 with `keep` would have given
    back are not distinguished here (every page is live)."""
    total = [s + n for s, n in zip(starts, lens)]
    width = max(-(-t // page) for t in total)
    n_pages = sum(-(-t // page) for t in total) + 3
    perm = torch.randperm(n_pages, generator=torch.Generator().manual_seed(seed)).tolist()
    table = torch.full((len(lens), width), -1, dtype=torch.int32)
    k_pages = rnd(n_pages, nkv, page, hd, seed=seed + 1).to(dt)
    v_pages = rnd(n_pages, nkv, page, hd, seed=seed + 2).to(dt)
    for s, t in enumerate(total):
        for b in range(-(-t // page)):
            table[s, b] = perm.pop()
    q = rnd(sum(lens), nh, hd, seed=seed + 3).to(dt)
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lens)]).to(torch.int32)
    sot = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).to(torch.int32)
    cu = torch.tensor([0] + torch.tensor(lens).cumsum(0).tolist(), dtype=torch.int32)
    return q, k_pages, v_pages, table, pos, sot, cu


def _plain_attention(q, k_pages, v_pages, table, pos, sot, scale, window, keep):
    n, nh, hd = q.shape
    _, nkv, page, _ = k_pages.shape
    out = torch.zeros(n, nh, hd, dtype=F64)
    for t in range(n):
        i = int(pos[t])
        keys = [j for j in range(i + 1) if window == 0 or i - j < window or j < keep]
        at = [(int(table[int(sot[t]), j // page]), j % page) for j in keys]
        k = torch.stack([k_pages[a, :, b] for a, b in at]).double()
        v = torch.stack([v_pages[a, :, b] for a, b in at]).double()
        for h in range(nh):
            g = h // (nh // nkv)
            out[t, h] = torch.softmax(k[:, g] @ q[t, h].double() * scale, 0) @ v[:, g]
    return out


WINDOWS = [(0, 0), (40, 0), (40, 5), (23, 19), (64, 64), (65, 1), (1, 3), (100, 130), (16, 500)]


@pytest.mark.parametrize("window,keep", WINDOWS)
@pytest.mark.parametrize("dt,tol,hd", [(torch.float32, 3e-6, 32), (torch.bfloat16, 1e-2, 64), (torch.bfloat16, 1e-2, 128)])
def test_attention_with_kept_first_tokens(dt, tol, hd, window, keep):
    """Every kernel that takes the shape: general, decode, mma.sync prefill, tcgen05 prefill; pages of 16 and 64."""
    o = ops()
    nh, nkv, scale = 4, 2, 0.3 * hd ** -0.5
    for page in (16, 64):
        lens, starts = (3, 1, 70, 1), (200, 31, 90, 330)
        q, kp, vp, table, pos, sot, cu = _attention_case(dt, nh, nkv, hd, page, lens, starts, seed=page + window)
        want = _plain_attention(q, kp, vp, table, pos, sot, scale, window, keep)
        dev = [t.to(DEV) for t in (q, kp, vp, table)]
        got = o.paged_attention(*dev, sot.to(DEV), pos.to(DEV), 0, window, scale, 331, keep=keep)
        close(got, want, tol)
        if dt == torch.float32:
            continue
        got = o.prefill_attention(*dev, cu.to(DEV), pos.to(DEV), len(lens), 70, 0, window, scale, keep=keep)
        close(got, want, tol)
        got = o.prefill_attention_tc(*dev, cu.to(DEV), pos.to(DEV), len(lens), 70, 0, window, scale, keep=keep)
        o.check_tc_status()
        close(got, want, tol)
        got = o.decode_attention(*dev, sot.to(DEV), pos.to(DEV), 0, window, scale, 331, keep=keep)
        close(got, want, tol)


@pytest.mark.parametrize("window,keep", [(0, 0), (40, 5), (65, 1), (100, 130)])
@pytest.mark.parametrize("dt,hd,vdim,heads,nkv", [(torch.float32, 48, 40, 3, 1), (torch.bfloat16, 64, 64, 2, 1), (torch.bfloat16, 128, 100, 4, 2),
                                                  (torch.bfloat16, 64, 50, 20, 1), (torch.bfloat16, 192, 192, 2, 2), (torch.bfloat16, 224, 80, 2, 1)])
def test_two_maps_with_norm_and_gate(dt, hd, vdim, heads, nkv, window, keep):
    """The difference of the maps by every route: split partials of the general, decode and mma.sync kernels through the merge
    kernel, and the tcgen05 kernel that finishes the row itself."""
    o = ops()
    lam, eps, mul, scale, page = 0.45, 1e-5, 0.7, 0.4 * hd ** -0.5, 64
    lens, starts = (5, 1, 66, 1), (150, 31, 60, 330)
    q, kp, vp, table, pos, sot, cu = _attention_case(dt, 2 * heads, nkv, hd, page, lens, starts, seed=heads + hd)
    vp[..., vdim:] = 0
    n = q.shape[0]
    proj = rnd(n, heads * vdim + 24, seed=8, std=1.5).to(dt).to(DEV)
    gate = proj[:, 8: 8 + heads * vdim]
    a = _plain_attention(q, kp, vp, table, pos, sot, scale, window, keep).view(n, heads, 2, hd)[..., :vdim]
    d = a[:, :, 0] - lam * a[:, :, 1]
    d = d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * mul
    tol = 5e-5 if dt == torch.float32 else 3e-2
    dev = [t.to(DEV) for t in (q, kp, vp, table)]
    for g in (gate, None):
        want = (d.reshape(n, -1) * torch.sigmoid(gate.double().cpu()) if g is not None else d.reshape(n, -1))
        fin = (lam, eps, mul, vdim, g)
        new = lambda: torch.empty(n, heads * vdim, dtype=dt, device=DEV)
        close(o.diff_merge(*o.paged_attention(*dev, sot.to(DEV), pos.to(DEV), 0, window, scale, 331, keep=keep, parts=True), *fin, new()), want, tol)
        if not o.decode_attention_supported(dt, 2 * heads, nkv, hd):
            continue
        close(o.diff_merge(*o.decode_attention(*dev, sot.to(DEV), pos.to(DEV), 0, window, scale, 331, keep=keep, parts=True), *fin, new()), want, tol)
        close(o.diff_merge(*o.prefill_attention(*dev, cu.to(DEV), pos.to(DEV), 4, 66, 0, window, scale, keep=keep, parts=True), *fin, new()), want, tol)
        got = o.diff_prefill_attention_tc(*dev, cu.to(DEV), pos.to(DEV), 4, 66, 0, window, keep, scale, *fin)
        o.check_tc_status()
        close(got, want, tol)
        # single tokens left to the decode kernel, merged into their own rows of the same result
        rows = torch.tensor([5, 72], device=DEV)
        got = o.diff_prefill_attention_tc(*dev, cu.to(DEV), pos.to(DEV), 4, 66, 0, window, keep, scale, *fin, skip_single=True)
        got[rows] = 99.0
        part = o.decode_attention(dev[0].index_select(0, rows), *dev[1:], sot.to(DEV).index_select(0, rows), pos.to(DEV).index_select(0, rows),
                                  0, window, scale, 331, keep=keep, parts=True)
        close(o.diff_merge(*part, *fin, got, rows=rows), want, tol)


def test_pages_that_were_given_back_do_not_reach_a_result():
    """Pages of 16 inside tiles of 64: those behind the window and past the kept tokens are gone from the table, and the pool's
    other pages hold NaN: the tcgen05 and mma.sync kernels, the decode kernel and the general kernel give finite, right rows."""
    o = ops()
    hd, page, window, keep, heads = 64, 16, 70, 5, 2
    lens, starts = (90,), (260,)
    q, kp, vp, table, pos, sot, cu = _attention_case(torch.bfloat16, 2 * heads, 1, hd, page, lens, starts, seed=4)
    want = _plain_attention(q, kp, vp, table, pos, sot, 0.1, window, keep)
    live = {int(table[0, b]) for b in range(table.shape[1]) if b == 0 or b * page + page > 260 - window + 1}
    for b in range(table.shape[1]):
        if int(table[0, b]) not in live:
            table[0, b] = -1
    for p in range(kp.shape[0]):
        if p not in live:
            kp[p], vp[p] = float("nan"), float("nan")
    vp_tail = 350 % page
    vp[int(table[0, -1]), :, vp_tail:] = float("nan")             # rows past the portion's end
    dev = [t.to(DEV) for t in (q, kp, vp, table)]
    close(o.prefill_attention_tc(*dev, cu.to(DEV), pos.to(DEV), 1, 90, 0, window, 0.1, keep=keep), want, 1e-2)
    o.check_tc_status()
    close(o.prefill_attention(*dev, cu.to(DEV), pos.to(DEV), 1, 90, 0, window, 0.1, keep=keep), want, 1e-2)
    close(o.decode_attention(*dev, sot.to(DEV), pos.to(DEV), 0, window, 0.1, 350, keep=keep), want, 1e-2)
    close(o.paged_attention(*dev, sot.to(DEV), pos.to(DEV), 0, window, 0.1, 350, keep=keep), want, 1e-2)


@pytest.mark.parametrize("dt,tol", [(torch.float32, 1e-6), (torch.bfloat16, 8e-3)])
def test_gate_rows(dt, tol):
    x, g = rnd(11, 3, 16, seed=1).to(dt), rnd(11, 40, seed=2).to(dt)
    gate = g.to(DEV)[:, 4: 4 + 30]
    want = (x[..., :10].double().reshape(11, 30)) * torch.sigmoid(g[:, 4:34].double())
    close(ops().gate_rows(x.to(DEV), gate, 10), want, tol)


@pytest.mark.parametrize("dt,tol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("extra", ["conv", "gate", "keep", "conv+gate+rotation", "keep+sink"])
def test_the_mechanisms_one_by_one_in_the_attention_mixer(dt, tol, extra):
    """What a design may combine otherwise: a convolution, an output gate or kept first tokens on attention with one map,
    with a rotation, with a sink; two requests in four steps against the formulas."""
    import plain_fofisun as plain
    from hi_b200.parts.context import CacheView
    from hi_b200.parts.registry import build
    from hi_b200.parts.spec import PartSpec
    from test_vinurax_engine import _ctx, _env

    width, heads, kvh, dim, vdim, page, eps = 48, 4, 2, 32, 24, 8, 1e-5
    p = {"hidden_size": width, "num_heads": heads, "num_kv_heads": kvh, "head_dim": dim, "value_dim": vdim, "scale": 0.3, "names": "short",
         "qk_norm_weighted": True, "qk_norm_eps": eps}
    if "conv" in extra:
        p["conv"] = 3
    if "gate" in extra:
        p["output_gate"] = True
    if "rotation" in extra:
        p["position"] = PartSpec("rope_yarn", {"head_dim": dim, "dims": 12, "base": 100.0})
    if "sink" in extra:
        p["sink"] = "learned"
    window = 9 if "keep" in extra else None
    if window:
        p["window"] = ("sliding", window, 3)
    part = build("mixer", PartSpec("attention", p), _env(dt, width), "m")
    w = {}
    for i, s in enumerate(part.tensor_specs()):
        if not s.optional:
            t = rnd(*s.shape, seed=60 + i)
            w[s.name] = (1 + 0.3 * t if s.name.endswith("norm") else t * (s.shape[-1] ** -0.5 * 1.5 if len(s.shape) == 2 else 1.0)).to(torch.bfloat16).float()
    part.load(lambda name: w[name].to(DEV).to(dt) if name in w else None)
    cs = part.cache_spec()
    view = CacheView(group=0, k_pages=torch.zeros((12, kvh, page, cs.head_dim), dtype=dt, device=DEV))
    view.v_pages = torch.zeros_like(view.k_pages)
    if cs.state_shape:
        view.state = torch.zeros((3, *cs.state_shape), dtype=torch.float32, device=DEV)
    table = torch.tensor([[7, 2, 9, 4, 6], [1, 11, 0, 5, 3]], dtype=torch.int32)
    xs = [rnd(n, width, seed=n).to(dt).float() for n in (33, 29)]
    got = [[], []]
    for lens, starts in (([13, 17], [0, 0]), ([18, 1], [13, 17]), ([1, 1], [31, 18]), ([1, 10], [32, 19])):
        x = torch.cat([xs[i][s: s + n] for i, (n, s) in enumerate(zip(lens, starts))])
        out = part.forward(x.to(DEV).to(dt), _ctx(lens, starts, page, table, [2, 0]), view)
        a = 0
        for i, n in enumerate(lens):
            got[i].append(out[a: a + n].double().cpu())
            a += n
    wd = {k: v.double() for k, v in w.items()}
    for i, x in enumerate(xs):
        h, t = x.double(), x.shape[0]
        u = {n: h @ wd[f"m.{n}"].T for n in "qkv"}
        if "conv" in extra:
            u = {n: plain.short_convolution(v, wd[f"m.{n}.conv"]) for n, v in u.items()}
        q = plain.rms_norm(u["q"].view(t, heads, dim), wd["m.q.norm"], eps)
        k = plain.rms_norm(u["k"].view(t, kvh, dim), wd["m.k.norm"], eps)
        if "rotation" in extra:
            ang = torch.arange(t, dtype=F64)[:, None] * torch.tensor([100.0 ** (-2.0 * j / 12) for j in range(6)], dtype=F64)
            for z in (q, k):
                lo, hi = z[..., :6].clone(), z[..., 6:12].clone()
                z[..., :6] = lo * torch.cos(ang)[:, None] - hi * torch.sin(ang)[:, None]
                z[..., 6:12] = hi * torch.cos(ang)[:, None] + lo * torch.sin(ang)[:, None]
        see = plain.visible(t, {"size": window, "keep_first": 3} if window else None)
        rows = []
        for a in range(heads):
            s = torch.where(see, (q[:, a] @ k[:, a // 2].T) * 0.3, torch.full((t, t), -math.inf, dtype=F64))
            e = torch.exp(s)
            den = e.sum(-1, keepdim=True) + (math.exp(float(wd["m.sink"][a])) if "sink" in extra else 0.0)
            rows.append((e / den) @ u["v"].view(t, kvh, vdim)[:, a // 2])
        o = torch.cat(rows, -1)
        if "gate" in extra:
            o = o * torch.sigmoid(h @ wd["m.g"].T)
        close(torch.cat(got[i]), o @ wd["m.o"].T, tol)
