"""The kernels Pivinex brought, each alone, against its plain twin (tests/plain_ops.py, float64 on
the CPU): windowed latent attention without a sink in all its forms, the query latent's norm, the
corrected softmax choice, identity experts, the stream around a parallel block."""

import math

import pytest
import torch

import plain_ops
import plain_pivinex

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32, BF16, I32 = torch.float32, torch.bfloat16, torch.int32
PAGE = 16


@pytest.fixture(scope="module")
def ops():
    from hetero_serve_b200.kernels import CudaOps
    return CudaOps(DEV)


@pytest.fixture(scope="module")
def plain():
    return plain_ops.PlainOps()


def rnd(*shape, seed=0, std=1.0, dtype=F32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * std).to(dtype)


def dev(*ts):
    out = tuple(t.to(DEV).contiguous() for t in ts)
    return out if len(out) > 1 else out[0]


def ints(*v):
    return torch.tensor(v, dtype=I32)


def close(got, want, tol):
    err = (got.detach().cpu().double() - want.double()).abs().max().item()
    assert err <= tol, err


class Batch:
    """Requests ``(start, new)`` over a pool of random rows; pages wholly behind the window of a
    request's first new token are taken out of its table (-1), as the cache manager leaves it."""

    def __init__(self, requests, width, window, dtype, seed):
        self.requests, self.window = requests, window
        g = torch.Generator().manual_seed(seed)
        need = [-(-(s + n) // PAGE) for s, n in requests]
        order = torch.randperm(sum(need) + 3, generator=g)
        self.table = torch.full((len(requests), max(need) + 1), -1, dtype=I32)
        at = 0
        for r, ((s, _n), k) in enumerate(zip(requests, need)):
            self.table[r, :k] = order[at:at + k].to(I32)
            at += k
            self.table[r, :max(0, s + 1 - window) // PAGE] = -1
        self.pool = rnd(sum(need) + 3, 1, 1, PAGE, width, seed=seed + 1, std=0.7).to(dtype)
        self.pos = torch.cat([torch.arange(s, s + n) for s, n in requests]).to(I32)
        self.req = torch.cat([torch.full((n,), r) for r, (_s, n) in enumerate(requests)]).to(I32)
        self.start = torch.tensor([0] + [n for _s, n in requests]).cumsum(0)[:-1].to(I32)
        self.len = torch.tensor([n for _s, n in requests], dtype=I32)
        self.host = [(f"r{r}", r, s, n) for r, (s, n) in enumerate(requests)]
        self.n = int(self.len.sum())
        self.status = torch.zeros(1, dtype=I32, device=DEV)


def attend(ops, plain, b, heads, rank, rot, scale=0.3, seed=5, plan=None, std=0.3, sink=None, **kw):
    stride = rot + 5
    qa = rnd(b.n, heads * rank, seed=seed, std=std)
    qr = rnd(b.n, 2 + heads * stride, seed=seed + 1, std=std)
    args = dict(n_heads=heads, rank=rank, rot_dim=rot, qr_head_stride=stride, qr_offset=2,
                scale=scale, page_size=PAGE, window=b.window)
    want = torch.zeros(b.n, heads * rank, dtype=torch.float64)
    plain.latent_attention(want, qa, qr, b.pool, b.table, b.pos, b.req, sink, status=None, **args)
    got = torch.full((b.n, heads * rank), 7.0, dtype=F32, device=DEV)
    ops.latent_attention(got, dev(qa), dev(qr), dev(b.pool), dev(b.table), dev(b.pos), dev(b.req),
                         None if sink is None else dev(sink), status=b.status, plan=plan, **args, **kw)
    assert int(b.status.item()) == 0              # a page behind the window is not looked up
    return got, want


# -- latent attention with a window, without a sink -------------------------------------------
@pytest.mark.parametrize("splits", [None, 1, 4])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window", [1, 2, 31, 32, 33, 100, 500])
def test_windowed_latent_attention_on_the_cuda_cores(ops, plain, window, dtype, splits):
    b = Batch([(0, 3), (31, 2), (64, 1), (200, 4), (97, 1)], 22 + 6, window, dtype, seed=window)
    ops.latent_splits = splits
    try:
        got, want = attend(ops, plain, b, 3, 22, 6)
    finally:
        ops.latent_splits = None
    close(got, want, 2e-5)


@pytest.mark.parametrize("rank, rot, heads", [(32, 8, 3), (64, 16, 8), (272, 24, 5), (16, 4, 20),
                                              (512, 64, 16), (24, 8, 1), (40, 2, 17),
                                              (128, 64, 2), (120, 80, 3)])
@pytest.mark.parametrize("window", [1, 17, 64, 300])
def test_windowed_latent_attention_of_single_tokens_by_list(ops, plain, rank, rot, heads, window):
    """A step of single tokens with a plan and a bfloat16 cache: queries and weights keep float32's
    mantissa on the tensor cores too."""
    b = Batch([(0, 1), (5, 1), (63, 2), (64, 1), (299, 1), (300, 1), (350, 4), (16, 3)], rank + rot, window,
              BF16, seed=40 + window)
    plan = ops.make_plan(b.host, b.n, PAGE)
    assert plan.tile_cap == 0 and plan.decode_cap == b.n
    got, want = attend(ops, plain, b, heads, rank, rot, scale=0.2, plan=plan)
    close(got, want, 2e-5)
    got, want = attend(ops, plain, b, heads, rank, rot, scale=0.2, plan=plan, sink=rnd(heads, seed=3))
    close(got, want, 2e-5)


@pytest.mark.parametrize("rank, rot, heads", [(32, 8, 3), (272, 24, 5), (16, 4, 70)])
@pytest.mark.parametrize("window", [1, 20, 129, 400])
def test_windowed_latent_attention_of_portions_in_absorbed_form(ops, plain, rank, rot, heads, window):
    b = Batch([(50, 150), (31, 2), (0, 37), (310, 70)], rank + rot, window, BF16, seed=60 + window)
    plan = ops.make_plan(b.host, b.n, PAGE)
    assert plan.tile_cap == 4 and plan.decode_cap == 2
    got, want = attend(ops, plain, b, heads, rank, rot, scale=0.2, plan=plan)
    close(got, want, 2e-2)
    before = got.clone()
    more, _ = attend(ops, plain, b, heads, rank, rot, scale=0.2, plan=plan, singles_only=True)
    single = torch.zeros(b.n, dtype=torch.bool)
    single[150:152] = True
    assert torch.equal(more[single.to(DEV)], before[single.to(DEV)])
    assert bool((more[~single.to(DEV)] == 7.0).all())           # the portions were left alone


def expanded(ops, b, q, w_uk, w_uv, heads, D, P, V, R, scale, freq):
    """The expanded form through its three operations; rows of single tokens keep their 7s."""
    plan = ops.make_plan(b.host, b.n, PAGE)
    rows = ops.latent_prompt_rows(plan, len(b.requests), n_heads=heads, dim=D, rot_dim=P, vdim=V,
                                  rank=R, window=b.window, scale=scale)
    assert rows == b.n + min(len(b.requests), plan.tile_cap) * (b.window - 1)
    z = lambda *shape: torch.zeros(*shape, dtype=BF16, device=DEV)
    lat, rope = z(rows, R), z(rows, 64)
    pad = -(-D // 64) * 64
    qp, base = z(b.n, heads * (pad + 64)), torch.zeros(len(b.requests), dtype=I32, device=DEV)
    ops.latent_gather(lat, rope, qp, base, dev(q), dev(b.pool), dev(b.table), dev(b.start), dev(b.len),
                      dev(b.pos), dev(b.req), n_heads=heads, dim=D, rank=R, rot_dim=P, window=b.window,
                      page_size=PAGE, status=b.status, freq=dev(freq), rot_dims=P)
    kv = z(rows, heads * (D + V))
    ops.linear(kv, lat, dev(torch.cat([w_uk, w_uv]).to(BF16)))
    out = torch.full((b.n, heads * V), 7.0, dtype=BF16, device=DEV)
    ops.latent_prompt_attention(out, qp, kv, rope, base, plan, n_heads=heads, dim=D, rot_dim=P,
                                vdim=V, rank=R, window=b.window, scale=scale, status=b.status)
    assert int(b.status.item()) == 0
    return out


def per_head(b, q, w_uk, w_uv, heads, D, P, V, R, scale, base, tokens):
    """The same from the equations, token by token, in float64."""
    rows = b.pool.view(-1, PAGE, R + P).double()
    want = torch.zeros(b.n, heads * V, dtype=torch.float64)
    for t in tokens:
        r, p = int(b.req[t]), int(b.pos[t])
        js = torch.arange(max(0, p + 1 - b.window), p + 1)
        key = rows[b.table[r, js // PAGE].long(), js % PAGE]
        for h in range(heads):
            qh = q[t, h * (D + P):(h + 1) * (D + P)].double()
            k = key[:, :R] @ w_uk[h * D:(h + 1) * D].double().T
            v = key[:, :R] @ w_uv[h * V:(h + 1) * V].double().T
            s = (k @ qh[:D] + key[:, R:] @ plain_pivinex.rotate_pairs(qh[D:], p, base)) * scale
            want[t, h * V:(h + 1) * V] = torch.softmax(s, 0) @ v
    return want


@pytest.mark.parametrize("D, P, V, R, heads", [(64, 32, 64, 64, 4), (24, 8, 40, 56, 3), (128, 64, 128, 96, 2),
                                               (72, 6, 104, 40, 2), (8, 2, 8, 8, 5), (120, 64, 48, 256, 1)])
@pytest.mark.parametrize("window", [1, 30, 128, 129, 257])
def test_portions_in_expanded_form(ops, D, P, V, R, heads, window):
    """Portions from the start, behind it, of several tiles, one token over a tile, beside single
    tokens; head sizes that fill one or two chunks, or a part of one."""
    b = Batch([(0, 140), (31, 2), (270, 129), (3, 5), (90, 1), (128, 128)], R + P, window, BF16, seed=window + D)
    base = 700.0
    freq = (base ** (-2.0 * torch.arange(P // 2, dtype=torch.float64) / P)).float()
    q = rnd(b.n, heads * (D + P), seed=9)
    w_uk, w_uv = rnd(heads * D, R, seed=10, std=R ** -0.5), rnd(heads * V, R, seed=11, std=R ** -0.5)
    w_uk, w_uv = w_uk.to(BF16).float(), w_uv.to(BF16).float()
    got = expanded(ops, b, q, w_uk, w_uv, heads, D, P, V, R, 0.25, freq).cpu().double()
    single = (b.len[b.req.long()] <= 4)
    assert bool((got[single] == 7.0).all())
    tokens = [t for t in range(b.n) if not single[t] and (t % 7 == 0 or t in (0, 1, 127, 128, 139, 269, 270, 275))]
    want = per_head(b, q, w_uk, w_uv, heads, D, P, V, R, 0.25, base, tokens)
    err = (got[tokens] - want[tokens]).abs().max().item()
    assert err < 2.5e-2, err


@pytest.mark.parametrize("window", [5, 128, 150])
def test_expanded_form_finds_one_key_at_the_edges_of_the_window(ops, window):
    """Each query of a portion meets one key that stands out; just inside the window it takes all
    of the weight, just outside it takes none."""
    D, P, V, R, heads, n, start = 16, 8, 16, 24, 2, 200, 160
    scale = 1.0
    freq = torch.ones(P // 2)
    w_uk, w_uv = torch.zeros(heads * D, R), rnd(heads * V, R, seed=21)
    for h in range(heads):
        w_uk[h * D, 0] = 1.0
    w_uv[:, 0] = 0.0
    w_uv = w_uv.to(BF16).float()
    for place in (0, 1, 15, 16, 127, 128, 129, 170, 299, 359):
        b = Batch([(start, n)], R + P, window, BF16, seed=31)
        rows = b.pool.view(-1, PAGE, R + P)
        rows[:, :, R:] = 0
        rows[:, :, 0] = 0
        page = int(b.table[0, place // PAGE])
        if page >= 0:
            rows[page, place % PAGE, 0] = 5.0
        q = torch.zeros(b.n, heads * (D + P))
        q[:, 0] = q[:, D + P] = 6.0
        got = expanded(ops, b, q, w_uk, w_uv, heads, D, P, V, R, scale, freq).cpu().double()
        tokens = [t for t in range(n) if abs(start + t - place - window) <= 2 or abs(start + t - place) <= 1
                  or t in (0, n - 1)]
        want = per_head(b, q, w_uk, w_uv, heads, D, P, V, R, scale, 1.0, tokens)
        assert (got[tokens] - want[tokens]).abs().max().item() < 3e-2, place


# -- the query latent beside the append, per-head products by list ------------------------------
@pytest.mark.parametrize("dtype, tol", [(F32, 3e-6), (BF16, 3e-2)])
@pytest.mark.parametrize("rank, rot, q_rank", [(24, 8, 40), (130, 6, 9), (8, 2, 300)])
def test_append_with_a_query_latent(ops, plain, dtype, tol, rank, rot, q_rank):
    b = Batch([(0, 20), (13, 7)], rank + rot, 1 << 20, dtype, seed=3)
    proj = rnd(b.n, q_rank + rank + rot, seed=4, std=2.0)
    wn, qn = rnd(rank, seed=5).abs() + 0.5, rnd(q_rank, seed=6).abs() + 0.5
    freq = (50.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot)).float()
    req = b.req.clone()
    req[5] = -1                                             # a padding row
    want_pool, want_q = torch.zeros(b.pool.shape, dtype=torch.float64), torch.zeros(b.n, q_rank, dtype=torch.float64)
    args = dict(c_offset=q_rank, rank=rank, rot_dim=rot, eps=1e-3, page_size=PAGE, rot_dims=rot, q_offset=0)
    plain.latent_append(want_pool, proj, wn, b.table, b.pos, req, status=None, freq=freq, q_out=want_q,
                        q_norm=qn, **args)
    pool = torch.zeros(b.pool.shape, dtype=dtype, device=DEV)
    cq = torch.full((b.n, q_rank), 7.0, dtype=dtype, device=DEV)
    ops.latent_append(pool, dev(proj), dev(wn), dev(b.table), dev(b.pos), dev(req), status=b.status,
                      freq=dev(freq), q_out=cq, q_norm=dev(qn), **args)
    close(pool, want_pool, tol)
    close(cq, want_q, tol)


@pytest.mark.parametrize("n_single", [3, 70])
def test_grouped_linear_on_listed_tokens(ops, plain, n_single):
    """Only the plan's single-query tokens are touched, on either kernel."""
    host = [("p", 0, 10, 30)] + [(f"s{i}", i + 1, i, 1) for i in range(n_single)] + [("q", 99, 0, 9)]
    n = 30 + n_single + 9
    plan = ops.make_plan(host, n, PAGE)
    assert plan.decode_cap == n_single
    a, w = rnd(n, 4 * 40, seed=1), rnd(3, 32, 50, seed=2).to(BF16)
    want = torch.zeros(n, 150, dtype=torch.float64)
    plain.grouped_linear(want, a, w, a_offset=8, a_group_stride=40)
    got = torch.full((n, 150), 7.0, dtype=F32, device=DEV)
    ops.grouped_linear(got, dev(a), dev(w), a_offset=8, a_group_stride=40,
                       w_nk=dev(w.transpose(1, 2)), singles=plan)
    close(got[30:30 + n_single], want[30:30 + n_single], 1e-1 if n_single >= 64 else 1e-4)
    assert bool((got[:30] == 7.0).all()) and bool((got[30 + n_single:] == 7.0).all())


# -- the choice and the experts -------------------------------------------------------------------
@pytest.mark.parametrize("E, top", [(12, 4), (1, 1), (7, 7), (72, 8), (300, 3)])
@pytest.mark.parametrize("hdt", [F32, BF16])
def test_route_by_corrected_softmax(ops, plain, E, top, hdt):
    T, width = 37, 50
    h, wr = rnd(T, width, seed=90).to(hdt), rnd(E, width, seed=91, std=0.3)
    corr = rnd(E, seed=92, std=0.5 / E)
    req = torch.zeros(T, dtype=I32)
    req[5] = -1
    live = [t for t in range(T) if t != 5]
    z = (h.double() @ wr.double().T).float()
    for correction in (corr, None):
        wi, ww = torch.zeros(T, top, dtype=I32), torch.zeros(T, top, dtype=torch.float64)
        plain.moe_route_softmax(wi, ww, h, wr, correction, req, top=top, scale=1.7)
        for handed in (None, z):
            gi = torch.full((T, top), -7, dtype=I32, device=DEV)
            gw = torch.zeros(T, top, dtype=F32, device=DEV)
            ops.moe_route_softmax(gi, gw, dev(h), dev(wr), None if correction is None else dev(correction),
                                  dev(req), top=top, scale=1.7, z=None if handed is None else dev(handed))
            assert torch.equal(gi.cpu()[live], wi[live]) and bool((gi[5] == -7).all())
            close(gw[live], ww[live], 1e-6)


def test_route_weighs_without_the_correction_and_breaks_ties_low(ops):
    h = torch.zeros(1, 4)
    gi, gw = torch.zeros(1, 3, dtype=I32, device=DEV), torch.zeros(1, 3, dtype=F32, device=DEV)
    ops.moe_route_softmax(gi, gw, dev(h), dev(torch.zeros(5, 4)), dev(torch.tensor([0.0, -1.0, 0.0, 2.0, 0.0])),
                          dev(ints(0)), top=3, scale=2.0)
    assert gi.cpu().tolist() == [[3, 0, 2]] and (gw.cpu() - 0.4).abs().max() < 1e-6


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("fresh", [False, True])
@pytest.mark.parametrize("T, width, ff, E, identity, top", [(19, 40, 28, 5, 3, 3), (300, 64, 96, 6, 2, 3),
                                                            (9, 36, 20, 1, 12, 9), (140, 96, 64, 3, 1, 4),
                                                            (700, 128, 64, 5, 2, 2), (333, 192, 128, 9, 1, 3)])
def test_identity_experts(ops, plain, T, width, ff, E, identity, top, fresh, dt):
    """Row kernels and sorted tiles; tokens all of whose choices pass the input through, and a
    choice outside every range, which adds nothing."""
    h = rnd(T, width, seed=1).to(dt)
    wg, wu = rnd(E, ff, width, seed=2, std=0.3).to(dt), rnd(E, ff, width, seed=3, std=0.3).to(dt)
    wd = rnd(E, width, ff, seed=4, std=0.3).to(dt)
    g = torch.Generator().manual_seed(5)
    idx = torch.stack([torch.randperm(E + identity, generator=g)[:top] for _ in range(T)]).to(I32)
    idx[2] = E
    wts = torch.rand(T, top, generator=g)
    wts[4, 0] = 0.0
    gpu_idx = idx.clone()
    gpu_idx[4, 0] = E + identity                           # outside: nothing
    req = torch.zeros(T, dtype=I32)
    req[3] = -1
    x = rnd(T, width, seed=6)
    want = x.double().clone()
    plain.moe_experts(want, None, h, wg, wu, wd, idx, wts, req, limit=0.0, act="silu", identity=identity,
                      fresh=fresh)
    got = dev(x.clone())
    y = torch.full((T * top, ff), float("nan"), dtype=F32, device=DEV)
    ops.moe_experts(got, y, dev(h), dev(wg), dev(wu), dev(wd), dev(gpu_idx), dev(wts), dev(req), limit=0.0,
                    act="silu", identity=identity, fresh=fresh)
    scale = want.abs().max().item()
    close(got, want, (1e-2 if dt == BF16 and T * top >= 256 else 1e-5) * scale)
    assert torch.equal(got[3].cpu(), x[3])


# -- the stream around a parallel block --------------------------------------------------------------
@pytest.mark.parametrize("width", [44, 130, 256, 1024, 4096, 4100, 37])
@pytest.mark.parametrize("dt", [F32, BF16])
def test_embed_norm(ops, plain, width, dt):
    T, V = 9, 31
    table = rnd(V, width, seed=1, std=2.0).to(dt)
    g, b, g2 = rnd(width, seed=2) + 1.0, rnd(width, seed=3), rnd(width, seed=4) + 1.0
    ids, req = ints(3, 30, 0, 5, -2, 7, 7, 1, 2), ints(0, 0, 1, -1, 2, 2, 0, 0, 0)
    feedback = ints(9, 11, 13)
    for bias, norm in ((None, None), (b, (g2, None, 1e-3)), (None, (g2, b, 1e-6))):
        want, wkeep, wout = (torch.zeros(T, width, dtype=torch.float64) for _ in range(3))
        plain.embed_norm(want, ids, req, table, g, bias, 1e-5, None, feedback=feedback, keep=wkeep,
                         out=wout if norm else None, norm=norm)
        got, keep = (torch.full((T, width), 7.0, dtype=F32, device=DEV) for _ in range(2))
        out = torch.full((T, width), 7.0, dtype=dt, device=DEV)
        status = torch.zeros(1, dtype=I32, device=DEV)
        on = lambda n: None if n is None else tuple(dev(v) if torch.is_tensor(v) else v for v in n)
        ops.embed_norm(got, dev(ids), dev(req), dev(table), dev(g), None if bias is None else dev(bias), 1e-5,
                       status, feedback=dev(feedback), keep=keep, out=out if norm else None, norm=on(norm))
        close(got, want, 2e-5)
        assert torch.equal(got, keep) and int(status.item()) == 0
        if norm:
            close(out, wout, (3e-6 if dt == F32 else 4e-3) * max(8.0, wout.abs().max().item()))
        assert bool((got[3] == 0).all())
    ops.embed_norm(got, dev(ints(V, 0, 0, 0, 0, 0, 0, 0, 0)), dev(req), dev(table), dev(g), None, 1e-5, status)
    assert int(status.item()) == 1 and bool((got[0] == 0).all())


@pytest.mark.parametrize("width", [44, 130, 256, 2048, 4100, 37])
@pytest.mark.parametrize("odt", [F32, BF16])
def test_residual_mix(ops, plain, width, odt):
    T = 7
    x, y1, y2, again = (rnd(T, width, seed=s) for s in (1, 2, 3, 4))
    s1, s2, g, b = (rnd(width, seed=s) for s in (5, 6, 7, 8))
    for kw, norm in ((dict(y1=y1, s1=s1, y2=y2, s2=s2, again=again), (g, None, 1e-5)),
                     (dict(y1=y1, s1=s1), None), (dict(again=again), (g, b, 1e-3)),
                     (dict(y1=y1, s1=s1, y2=y2, s2=s2), (g, b, 1e-6))):
        want, wout = x.double().clone(), torch.zeros(T, width, dtype=torch.float64)
        plain.residual_mix(want, **kw, out=wout if norm else None, norm=norm)
        got, out = dev(x.clone()), torch.zeros(T, width, dtype=odt, device=DEV)
        on = None if norm is None else tuple(dev(v) if torch.is_tensor(v) else v for v in norm)
        ops.residual_mix(got, **{k: dev(v) for k, v in kw.items()}, out=out if norm else None, norm=on)
        close(got, want, 1e-6 * 8)
        if norm:
            close(out, wout, (3e-6 if odt == F32 else 4e-3) * max(8.0, wout.abs().max().item()))
