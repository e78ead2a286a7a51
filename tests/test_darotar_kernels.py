"""The kernels that Darotar extended, each against the same arithmetic in plain PyTorch (float64 on the CPU): encoding and
append of q and k where the keys are the values too (both forms of the kernel, and inside the one-launch decode
attention), the boundary that hands on the stream itself, and attention over shared rows with a learned sink in every
attention kernel."""
import pytest
import torch

from plain_darotar import rms_norm, rotate, softmax_weights, visible

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


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


def table(dims, base, factor=1.0):
    return torch.tensor([base ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=torch.float64).float()


# heads, kv heads, dim, row length, rotating dims, neighbouring pairs
ENCODINGS = [(4, 2, 64, 64, 64, True), (3, 1, 128, 128, 64, True), (8, 8, 16, 16, 16, False), (5, 5, 32, 32, 16, True),
             (6, 2, 10, 16, 6, True), (2, 1, 40, 48, 40, False), (2, 2, 64, 64, 4, True), (2, 1, 272, 272, 100, True)]


@pytest.mark.parametrize("dt,tol", [(torch.float32, 2e-6), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("nh,nkv,dim,hd,rot,near", ENCODINGS)
def test_keys_that_are_values(dt, tol, nh, nkv, dim, hd, rot, near):
    """q and k rotated and then normed; the value row of a token is the projected key bit for bit; rows of other tokens
    in the pages stay; a token without a page writes nothing."""
    o, eps, page, n = ops(), 1e-2, 8, 21
    qk = torch.zeros(n, nh + nkv, hd)
    qk[:, :, :dim] = rnd(n, nh + nkv, dim, seed=nh + dim, std=0.7)
    qk = qk.to(dt)
    pos = torch.arange(n, dtype=torch.int32)
    sot = torch.zeros(n, dtype=torch.int32)
    bt = torch.tensor([[3, 0, -1]], dtype=torch.int32)            # the tokens from 16 on have no page
    kp, vp = rnd(5, nkv, page, hd, seed=1).to(dt).to(DEV), rnd(5, nkv, page, hd, seed=2).to(dt).to(DEV)
    k0, v0 = kp.clone(), vp.clone()
    q = o.qkv_post(qk.view(n, -1).to(DEV), nh, nkv, hd, pos.to(DEV), table(rot, 50.0, 2.0).to(DEV), near, True, eps, None,
                   sot.to(DEV), bt.to(DEV), kp, vp, page, True, norm_dim=0 if hd == dim else dim, values_are_keys=True)
    spec = {"base": 50.0, "dims": rot, "scaling": {"factor": 2.0}}
    want = rms_norm(rotate(qk[:, :, :dim].double(), spec, near), None, eps)
    close(q[:, :, :dim], want[:, :nh], tol)
    assert hd == dim or float(q[:, :, dim:].abs().max()) == 0.0
    for t in range(16):
        at = (3 if t < 8 else 0, slice(None), t % 8)
        close(kp[at][:, :dim], want[t, nh:], 4 * tol)
        assert torch.equal(vp[at].cpu(), qk[t, nh:])
    untouched = [1, 2, 4]
    assert torch.equal(kp[untouched], k0[untouched]) and torch.equal(vp[untouched], v0[untouched])


@pytest.mark.parametrize("nh,nkv,hd,rot,chunk", [(8, 2, 64, 64, 0), (4, 4, 128, 32, 0), (16, 1, 128, 128, 64)])
def test_one_launch_decode_where_keys_are_values(nh, nkv, hd, rot, chunk):
    """The one-launch decode attention against encoding, decode attention and merge on their own: the appended keys and
    values are the same bits, the outputs agree to bfloat16 rounding."""
    o, dt, page = ops(), torch.bfloat16, 64
    starts = [0, 1, 63, 64, 255, 1030, 3000]
    blocks = [s // page + 1 for s in starts]
    perm = torch.randperm(sum(blocks), generator=torch.Generator().manual_seed(3)).tolist()
    bt = torch.full((len(starts), max(blocks)), -1, dtype=torch.int32)
    for i, b in enumerate(blocks):
        bt[i, :b] = torch.tensor([perm.pop() for _ in range(b)], dtype=torch.int32)
    kp, vp = rnd(sum(blocks), nkv, page, hd, seed=1).to(dt), rnd(sum(blocks), nkv, page, hd, seed=2).to(dt)
    qk = rnd(len(starts), (nh + nkv) * hd, seed=5, std=1.5).to(dt).to(DEV)
    pos, sot = torch.tensor(starts, dtype=torch.int32).to(DEV), torch.arange(len(starts), dtype=torch.int32).to(DEV)
    inv, bt, longest = table(rot, 1000.0, 4.0).to(DEV), bt.to(DEV), max(starts) + 1
    for _round in range(2):
        k1, v1, k2, v2 = kp.to(DEV), vp.to(DEV), kp.to(DEV), vp.to(DEV)
        q = o.qkv_post(qk, nh, nkv, hd, pos, inv, True, True, 1e-5, None, sot, bt, k1, v1, page, True, values_are_keys=True)
        want = o.decode_attention(q, k1, v1, bt, sot, pos, chunk, 0, 0.1, longest)
        got = o.decode_attention_fused(qk, nh, nkv, hd, pos, inv, True, True, 1e-5, None, sot, bt, k2, v2, chunk, 0, 0.1,
                                       longest, values_are_keys=True)
        assert got is not None
        assert torch.equal(k1, k2) and torch.equal(v1, v2), "the appended keys or values differ"
        close(got, want.double().cpu(), 1e-2)
    o.check_tc_status()


@pytest.mark.parametrize("width", [64, 51, 2048, 8192, 8196])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("routed", [False, True])
def test_boundary_that_hands_on_the_stream(width, dt, routed):
    """x + rmsnorm(result) * w in place, and its rounding beside it (float32: the stream is its own copy)."""
    from hi_b200.parts.context import NormedPending, Pending

    n, k, eps = 9, 2, 1e-3
    x, wy = rnd(n, width, seed=1, std=3.0), 0.4 * (1 + 0.3 * rnd(width, seed=3))
    if routed:
        r, slot = rnd(n * k, width, seed=6), torch.randperm(n * k, generator=torch.Generator().manual_seed(1))
        y = r[slot].double().view(n, k, width).sum(1)
        delta = Pending(routed=r.to(DEV), slot_of_entry=slot.to(torch.int32).to(DEV), top_k=k)
    else:
        d = rnd(n, width, seed=2).to(dt)
        y, delta = d.double(), d.to(DEV)
    stream = x.to(DEV)
    h = NormedPending(delta=delta, weight=wy.to(DEV), eps=eps).read(stream, dt)
    want = x.double() + rms_norm(y, wy.double(), eps)
    close(stream, want, 2e-6)
    assert h.dtype == dt and torch.equal(h, stream.to(dt)) and (dt == torch.bfloat16 or h is stream)


@pytest.mark.parametrize("dt,tol", [(torch.float32, 1e-6), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("rows,heads,hd,vdim,before", [(5, 3, 16, 16, 8), (70, 16, 128, 128, 64), (9, 4, 64, 24, 16), (7, 3, 5, 5, 2),
                                                       (3, 2, 16, 12, 8), (1, 40, 64, 64, 1)])
def test_gate_of_every_element(dt, tol, rows, heads, hd, vdim, before):
    """The gate is a column slice behind ``before`` other columns: aligned and not."""
    o, proj = rnd(rows, heads, hd, seed=1).to(dt), rnd(rows, before + heads * vdim + 8, seed=2, std=2.0).to(dt)
    gate = proj.to(DEV)[:, before: before + heads * vdim]
    want = o[:, :, :vdim].double().reshape(rows, -1) * torch.sigmoid(proj[:, before: before + heads * vdim].double())
    close(ops().gate_rows(o.to(DEV), gate, vdim), want, tol)


@pytest.mark.parametrize("nh,nkv,window", [(40, 2, 0), (40, 2, 100), (34, 2, 0)])
def test_decode_attention_with_more_than_a_row_tile_of_heads(nh, nkv, window):
    """More than 16 query heads on a key head, values apart from keys, one split and many: against the plain softmax."""
    o, dt, page, hd, total = ops(), torch.bfloat16, 64, 128, 1500
    k, v = rnd(2, total, nkv, hd, seed=1).to(dt), rnd(2, total, nkv, hd, seed=2).to(dt)
    q, starts = rnd(2, nh, hd, seed=3, std=2.0).to(dt), [total - 1, 70]
    blocks = -(-total // page)
    bt = torch.randperm(2 * blocks, generator=torch.Generator().manual_seed(4)).to(torch.int32).view(2, blocks)
    kp, vp = torch.zeros(2 * blocks, nkv, page, hd, dtype=dt), torch.zeros(2 * blocks, nkv, page, hd, dtype=dt)
    want = []
    for i, at in enumerate(starts):
        for b in range(blocks):
            part = slice(b * page, min(total, (b + 1) * page))
            kp[int(bt[i, b]), :, : part.stop - part.start] = k[i, part].transpose(0, 1)
            vp[int(bt[i, b]), :, : part.stop - part.start] = v[i, part].transpose(0, 1)
        lo, seen = max(0, at + 1 - window) if window else 0, []
        for a in range(nh):
            kd, vd = (t[i, lo: at + 1, a // (nh // nkv)].double() for t in (k, v))
            seen.append(torch.softmax(kd @ q[i, a].double() * 0.1, -1) @ vd)
        want.append(torch.stack(seen))
    got = o.decode_attention(q.to(DEV), kp.to(DEV), vp.to(DEV), bt.to(DEV), torch.arange(2, dtype=torch.int32, device=DEV),
                             torch.tensor(starts, dtype=torch.int32, device=DEV), 0, window, 0.1, total)
    close(got, torch.stack(want), 1.5e-2)


@pytest.mark.parametrize("dt,tol", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("hd", [64, 128, 192, 208])
@pytest.mark.parametrize("heads", [4, 20])
def test_attention_over_shared_rows_with_a_learned_sink(dt, tol, hd, heads):
    """Rows that are keys and values of all heads, a sink per head (below, among and above the scores): a long portion
    (tcgen05), a short one (mma.sync), single tokens, and both in one step."""
    from hi_b200.parts.attention import attend_over_pages
    from test_vinurax_engine import _ctx

    page, total, scale = 64, 300, 0.3 * hd ** -0.5
    rows = rnd(2, total, hd, seed=hd).to(dt)
    q = rnd(2, total, heads, hd, seed=heads + 1, std=2.0).to(dt)
    sinks = torch.linspace(-3.0, 8.0, heads)
    want = []
    for i in range(2):
        r = rows[i].double()
        want.append(torch.stack([softmax_weights((q[i, :, a].double() @ r.T) * scale, visible(total, None), sinks[a].double()) @ r
                                 for a in range(heads)], dim=1))
    bt = torch.tensor([[7, 2, 9, 4, 6], [1, 8, 0, 5, 3]], dtype=torch.int32)
    pages = torch.full((10, 1, page, hd), 30.0, dtype=dt, device=DEV)
    for i in range(2):
        for b in range(5):
            part = rows[i, b * page: (b + 1) * page]
            pages[int(bt[i, b]), 0, : part.shape[0]] = part.to(DEV)
    for lens, starts in (([300, 170], [0, 0]), ([140, 1], [160, 299]), ([9, 2], [290, 64]), ([1, 1], [299, 63]), ([3, 1], [0, 0])):
        ctx = _ctx(lens, starts, page, bt, [0, 1])
        qs = torch.cat([q[i, s: s + n] for i, (n, s) in enumerate(zip(lens, starts))]).to(DEV)
        out = attend_over_pages(qs, pages, pages, ctx.block_tables[0], ctx, heads, 1, hd, 0, 0, scale, sink_values=sinks.to(DEV))
        close(out, torch.cat([want[i][s: s + n] for i, (n, s) in enumerate(zip(lens, starts))]), tol)
