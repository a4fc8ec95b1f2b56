"""The kernels of the Nukodra parts, each mechanism alone, against the plain implementation's
function of the same mechanism (tests/plain_nukodra.py, float64 on the CPU) or the operation's
plain twin: copies of the stream, attention with row norms, rotation, capped scores and a sink,
gates in the per-head products and the expanded latent attention, the state-space recurrence over
portions and single tokens, and norms in parts behind a gate."""

import math

import pytest
import torch

import plain_nukodra as P
from plain_ops import PlainOps

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32, BF16, I32, F64 = torch.float32, torch.bfloat16, torch.int32, torch.float64


@pytest.fixture(scope="module")
def ops():
    from hetero_serve_b200.kernels import CudaOps
    return CudaOps(DEV)


def rnd(*shape, seed=0, std=1.0, mean=0.0, dtype=F32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * std + mean).to(dtype)


def dev(*ts):
    out = tuple(t.to(DEV).contiguous() for t in ts)
    return out if len(out) > 1 else out[0]


def ints(v):
    return torch.tensor(list(v), dtype=I32, device=DEV)


def close(got, want, tol):
    want = want.double()
    err = ((got.detach().cpu().double() - want).abs() / (1.0 + want.abs())).max().item()
    assert err <= tol, err


# -- copies of the stream -------------------------------------------------------------------------
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("width", [37, 96, 1024, 1280, 4100])
def test_hyper_mix(ops, streams, width):
    """The copies mixed from the old ones, in place and from one row that stands for all; what the
    next sublayer reads, with and without its norm; the plain sum."""
    if width > 2000 and streams not in (2, 5):
        pytest.skip("two counts are enough for the wide row")
    T, eps = 9, 1e-5
    X, y = rnd(T, streams * width, seed=1), rnd(T, width, seed=2)
    mix, wr, rd = rnd(streams, streams, seed=3), rnd(streams, seed=4), rnd(streams, seed=5)
    g = rnd(width, seed=6, std=0.2, mean=1.0)
    w = {"c.in": torch.ones(streams, dtype=F64), "c.mix": mix.double(), "c.out": wr.double()}

    def plain(X):
        return P.connect(X.view(T, streams, width).transpose(0, 1).double(), w, "c.", lambda u: y.double())

    new = plain(X)
    u_want = torch.einsum("s,stw->tw", rd.double(), new)
    for dt, tol in ((F32, 1e-5), (BF16, 1e-2)):
        Xd, u, out = dev(X.clone()), torch.zeros(T, width, device=DEV), torch.zeros(T, width, dtype=dt, device=DEV)
        ops.hyper_mix(Xd, Xd, dev(y), streams=streams, mix=dev(mix), write=dev(wr), read=dev(rd), u=u,
                      out=out, norm=(dev(g), eps))
        close(Xd.view(T, streams, width).transpose(0, 1), new, 1e-5)
        close(u, u_want, 1e-5)
        close(out, P.unit_rms(u_want, eps) * g.double(), tol)
    one = rnd(T, width, seed=7)                       # one row for all copies
    new = plain(one.repeat(1, streams))
    Xd, u = torch.zeros(T, streams * width, device=DEV), torch.zeros(T, width, device=DEV)
    ops.hyper_mix(Xd, dev(one), dev(y), streams=streams, mix=dev(mix), write=dev(wr), u=u)
    close(Xd.view(T, streams, width).transpose(0, 1), new, 1e-5)
    close(u, new.sum(0), 1e-5)
    out = torch.zeros(T, width, device=DEV)           # no sublayer yet
    ops.hyper_mix(None, dev(one), streams=streams, read=dev(rd), out=out, norm=(dev(g), eps))
    close(out, P.unit_rms(one.double() * rd.double().sum(), eps) * g.double(), 1e-4)


# -- attention with row norms, rotation, a cap and a sink ------------------------------------------
def _plain_attention(rows, H, G, D, V, offs, wq, wk, rot, scale, window, cap, sink, eps):
    T = rows.shape[0]
    r = rows.double()
    q_off, k_off, v_off, g_off = offs
    q = P.unit_rms(r[:, q_off:q_off + H * D], eps) * wq.double()
    k = P.unit_rms(r[:, k_off:k_off + G * D], eps) * wk.double()
    q, k = P.rotate_rows(q.view(T, H, D), rot), P.rotate_rows(k.view(T, G, D), rot)
    v = r[:, v_off:v_off + G * V].view(T, G, V)
    of = torch.tensor([h // (H // G) for h in range(H)])
    o = P.softmax_over_visible(q, k[:, of], v[:, of], scale, window, cap, sink)
    return o.reshape(T, H * V) * torch.sigmoid(r[:, g_off:g_off + H * V])


@pytest.mark.parametrize("dtype, tol", [(F32, 2e-5), (BF16, 5e-2)])
@pytest.mark.parametrize("H, G, D, V, window, rot, cap, sinks", [
    (4, 2, 26, 18, 21, 14, 15.0, True), (1, 1, 32, 32, 9, 32, 1.0, True),
    (2, 2, 8, 6, 1, 2, 0.0, True), (8, 2, 64, 64, 48, 64, 30.0, True),
    (4, 4, 128, 128, 40, 64, 20.0, False), (3, 1, 20, 258, 0, 20, 5.0, True),
    (6, 2, 48, 48, 70, 48, 0.0, True), (10, 2, 96, 96, 90, 64, 25.0, True),
    (20, 1, 64, 128, 33, 0, 10.0, True), (2, 1, 112, 80, 130, 112, 30.0, True),
    (16, 4, 72, 104, 64, 24, 12.0, True), (4, 2, 256, 64, 40, 128, 30.0, True)])
@pytest.mark.parametrize("planned", ["no", "yes", "clusters", "dense"])
def test_span_attention(ops, monkeypatch, dtype, tol, H, G, D, V, window, rot, cap, sinks, planned):
    """Two requests whose pages are scattered over the pool, in portions that end inside pages and
    windows; then single tokens.  Every position is compared.  The pages behind the window are
    taken out of the table: nothing may look them up.  Unused rows of the pool are NaN.  With the
    step's work lists portions run as tiles, "dense": over rows gathered from their pages; "clusters": single tokens on the kernel for many keys,
    whose products keep float32's mantissa, whatever the window."""
    if planned == "clusters":
        monkeypatch.setattr(ops, "span_decode_keys", 0)
    eps, page, scale = 1e-5, 16, 2.0 / math.sqrt(D)
    q_off = 8
    k_off = q_off + H * D
    v_off = k_off + G * D
    g_off = v_off + G * V
    width = g_off + H * V + 4
    rows = {"a": rnd(150, width, seed=41), "b": rnd(77, width, seed=42)}
    wq, wk = rnd(H * D, seed=44, std=0.2, mean=1.3), rnd(G * D, seed=45, std=0.2, mean=1.3)
    sink = rnd(H, seed=46, mean=2.0) if sinks else None
    r = {"base": 500.0, "dims": rot}
    want = {k: _plain_attention(x, H, G, D, V, (q_off, k_off, v_off, g_off), wq, wk, r, scale, window,
                                cap, None if sink is None else sink.double(), eps)
            for k, x in rows.items()}
    freq = dev((500.0 ** (-2.0 * torch.arange(rot // 2, dtype=F64) / max(rot, 1))).float()) if rot else None
    n_pages, max_pages = 24, 10
    perm = torch.randperm(n_pages, generator=torch.Generator().manual_seed(43)).tolist()
    table = torch.full((2, max_pages), -1, dtype=I32)
    table[0], table[1] = torch.tensor(perm[:10]), torch.tensor(perm[10:20])
    table = dev(table)
    pool = torch.full((n_pages, G, page, D + V), float("nan"), dtype=dtype, device=DEV)
    status = torch.zeros(1, dtype=I32, device=DEV)
    wqd, wkd, sk = dev(wq), dev(wk), dev(sink) if sinks else None
    plan = [[("a", 37)], [("a", 2), ("b", 30)], [("b", 1), ("a", 58)], [("a", 1), ("b", 1)],
            [("b", 45), ("a", 1)], [("a", 1)]] + [[("a", 1)]] * 17 + [[("a", 33)]]
    fed = {"a": 0, "b": 0}
    idx = {"a": 0, "b": 1}
    for step in plan:
        proj = dev(torch.cat([rows[r][fed[r]:fed[r] + k] for r, k in step]))
        T = proj.shape[0]
        tok_pos = ints(p for r, k in step for p in range(fed[r], fed[r] + k))
        tok_req = ints(row for row, (r, k) in enumerate(step) for _ in range(k))
        starts, at = [], 0
        for _r, k in step:
            starts.append(at)
            at += k
        tab = table[[idx[r] for r, k in step]].contiguous()
        q = torch.zeros(T, H * D, device=DEV)
        sizes = dict(n_heads=H, n_kv_heads=G, head_dim=D, value_dim=V, page_size=page, status=status)
        ops.span_prepare(q, pool, proj, tab, tok_pos, tok_req, q_off=q_off, k_off=k_off, v_off=v_off,
                         qk_norm=False, eps=eps, writes=True, wq=wqd, wk=wkd, freq=freq, rot_dims=rot,
                         **sizes)
        if window:
            for row, (r, k) in enumerate(step):
                tab[row, :max(0, fed[r] - window + 1) // page] = -1
        out = torch.full((T, H * V), float("nan"), dtype=dtype, device=DEV)
        work = ops.make_plan([(row, row, fed[r], k) for row, (r, k) in enumerate(step)], T, page) \
            if planned != "no" else None
        more = dict(req_start=ints(starts), req_len=ints(k for _r, k in step)) if planned == "dense" else {}
        ops.span_attention(out, q, pool, tab, tok_pos, tok_req, scale=scale, slopes=None,
                           window=window, keep_first=0, gate=proj, gate_offset=g_off, out_scale=1.0,
                           plan=work, softcap=cap, sinks=sk, **more, **sizes)
        at = 0
        for r, k in step:
            close(out[at:at + k], want[r][fed[r]:fed[r] + k], tol)
            fed[r] += k
            at += k
    assert int(status.item()) == 0


def test_span_prepare_turns_far_positions(ops):
    """Positions in the hundred thousands: the angle's error does not grow with the position."""
    H, D, rot, page = 2, 16, 16, 16
    pos = [0, 1, 17, 99_999, 250_001]
    proj = rnd(len(pos), 2 * H * D + D, seed=3)
    freq = (1e4 ** (-2.0 * torch.arange(rot // 2, dtype=F64) / rot)).float()
    q = torch.zeros(len(pos), H * D, device=DEV)
    pool = torch.zeros(1, 1, page, 2 * D, device=DEV)
    one = torch.ones(H * D)
    ops.span_prepare(q, pool, dev(proj), ints([0] * 4).view(1, 4), ints(pos), ints([0] * len(pos)),
                     n_heads=H, n_kv_heads=1, head_dim=D, value_dim=D, q_off=0, k_off=None, v_off=None,
                     qk_norm=False, eps=1e-6, writes=False, page_size=page,
                     status=torch.zeros(1, dtype=I32, device=DEV), wq=dev(one), freq=dev(freq), rot_dims=rot)
    v = P.unit_rms(proj[:, :H * D].double(), 1e-6).view(-1, H, D)
    ang = torch.tensor(pos, dtype=F64)[:, None] * freq.double()
    c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
    lo, hi = v[..., :8], v[..., 8:]
    close(q, torch.cat([lo * c - hi * s, hi * c + lo * s], -1).reshape(len(pos), -1), 2e-6)


# -- gates ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("T, groups, k, n", [(3, 3, 20, 14), (9, 2, 64, 72), (130, 4, 64, 96), (70, 1, 32, 8)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_grouped_linear_with_a_gate(ops, T, groups, k, n, dtype):
    a, w = rnd(T, groups * k, seed=1), rnd(groups, k, n, seed=2, std=1 / math.sqrt(k), dtype=dtype)
    gate = rnd(T, groups * n + 5, seed=3)
    out = torch.zeros(T, groups * n, dtype=dtype, device=DEV)
    ops.grouped_linear(out, dev(a), dev(w), w_nk=dev(w.transpose(1, 2).contiguous()) if dtype == BF16 else None,
                       gate=dev(gate), gate_offset=5)
    want = torch.zeros(T, groups * n, dtype=F64)
    PlainOps().grouped_linear(want, a, w, gate=gate, gate_offset=5)
    close(out, want, 1e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("parts, dim", [(1, 56), (4, 13), (2, 1024), (3, 100), (1, 4096)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_norm_in_parts_behind_the_gate(ops, parts, dim, dtype):
    T, eps = 5, 1e-5
    o, gate, w = rnd(T, parts * dim, seed=1, std=0.01), rnd(T, parts * dim + 3, seed=2, std=2.0), rnd(parts * dim, seed=3)
    out = torch.zeros(T, parts * dim, dtype=dtype, device=DEV)
    ops.head_norm_gate(out, dev(o), dev(w), dev(gate), gate_offset=3, heads=parts, dim=dim, eps=eps,
                       gate_act="silu", gate_first=True)
    v = (o.double() * P.silu(gate[:, 3:].double())).view(T, parts, dim)
    close(out, P.unit_rms(v, eps).reshape(T, -1) * w.double(), 1e-5 if dtype == F32 else 1e-2)


@pytest.mark.parametrize("H, D, rot, V, R, window", [
    (3, 64, 32, 64, 64, 0), (2, 72, 16, 104, 96, 0), (4, 128, 64, 128, 128, 0), (5, 16, 8, 24, 32, 0),
    (3, 64, 32, 64, 64, 150), (2, 128, 16, 64, 40, 1)])
def test_expanded_latent_attention(ops, H, D, rot, V, R, window):
    """Prompt portions in expanded form with and without a window, beside single tokens; queries as
    columns of a wider row, and a gate.  One key in the first pages stands out."""
    page, n_pages, scale = 16, 40, 1.5 / math.sqrt(D + rot)
    wk, wv = rnd(H * D, R, seed=1, std=1 / math.sqrt(R), dtype=BF16), rnd(H * V, R, seed=2, std=1 / math.sqrt(R), dtype=BF16)
    length = {"a": 330, "b": 170}
    rows = {r: rnd(n, R + rot, seed=3 + i, dtype=BF16) for i, (r, n) in enumerate(length.items())}
    rows["a"][5] *= 3.0
    perm = torch.randperm(n_pages, generator=torch.Generator().manual_seed(5))
    table = torch.full((2, 24), -1, dtype=I32)
    table[0, :21], table[1, :11] = perm[:21].int(), perm[21:32].int()
    pool = torch.full((n_pages, page, R + rot), float("nan"), dtype=BF16)
    for i, r in enumerate(("a", "b")):
        for p in range(length[r]):
            pool[table[i, p // page], p % page] = rows[r][p]
    freq = (900.0 ** (-2.0 * torch.arange(rot // 2, dtype=F64) / rot)).float()
    gate_off = H * (D + rot) + 8
    width = gate_off + H * V
    status = torch.zeros(1, dtype=I32, device=DEV)
    for step in ([("a", 0, 130), ("b", 0, 60)], [("b", 60, 1), ("a", 130, 150)],
                 [("a", 280, 50), ("b", 61, 109)]):
        T = sum(n for _r, _s, n in step)
        proj = rnd(T, width, seed=9)
        starts, at = [], 0
        for _r, _s, n in step:
            starts.append(at)
            at += n
        tok_pos = ints(p for _r, s, n in step for p in range(s, s + n))
        tok_req = ints(i for i, (_r, _s, n) in enumerate(step) for _ in range(n))
        tab = dev(table[[0 if r == "a" else 1 for r, _s, _n in step]])
        plan = ops.make_plan([(i, i, s, n) for i, (_r, s, n) in enumerate(step)], T, page)
        sizes = dict(n_heads=H, dim=D, rot_dim=rot, vdim=V, rank=R, window=window, scale=scale)
        n_rows = ops.latent_prompt_rows(plan, len(step), **sizes)
        assert n_rows > 0
        lat, rope = (torch.zeros(n_rows, c, dtype=BF16, device=DEV) for c in (R, 64))
        qp = torch.zeros(T, H * (-(-D // 64) * 64 + 64), dtype=BF16, device=DEV)
        base = torch.zeros(len(step), dtype=I32, device=DEV)
        projd = dev(proj)
        ops.latent_gather(lat, rope, qp, base, projd, dev(pool), tab, ints(starts),
                          ints(n for _r, _s, n in step), tok_pos, tok_req, n_heads=H, dim=D, rank=R,
                          rot_dim=rot, window=window, page_size=page, status=status, freq=dev(freq),
                          rot_dims=rot)
        kv = torch.zeros(n_rows, H * (D + V), dtype=BF16, device=DEV)
        ops.linear(kv, lat, dev(torch.cat([wk, wv])))
        out = torch.full((T, H * V), float("nan"), dtype=BF16, device=DEV)
        ops.latent_prompt_attention(out, qp, kv, rope, base, plan, status=status, gate=projd,
                                    gate_offset=gate_off, **sizes)
        for (r, s, n), t0 in zip(step, starts):
            if n <= 4:
                continue                        # another operation's tokens
            c, kr = rows[r][:, :R].double(), rows[r][:, R:].double()
            k = torch.cat([(c @ wk.double().T).view(-1, H, D), kr[:, None].expand(-1, H, rot)], 2)
            v = (c @ wv.double().T).view(-1, H, V)
            for i in list(range(0, n, 7)) + [n - 1]:
                p = s + i
                q = proj[t0 + i, :H * (D + rot)].double().view(H, D + rot)
                ang = p * freq.double()
                x, y = q[:, D::2].clone(), q[:, D + 1::2].clone()
                q = q.clone()
                q[:, D::2] = x * torch.cos(ang) - y * torch.sin(ang)
                q[:, D + 1::2] = y * torch.cos(ang) + x * torch.sin(ang)
                lo = max(0, p + 1 - window) if window else 0
                wts = torch.softmax(torch.einsum("jhn,hn->hj", k[lo:p + 1], q) * scale, 1)
                o = torch.einsum("hj,jhv->hv", wts, v[lo:p + 1]).reshape(-1)
                o = o * torch.sigmoid(proj[t0 + i, gate_off:].double())
                close(out[t0 + i], o, 4e-2)
    assert int(status.item()) == 0


# -- the state-space recurrence ---------------------------------------------------------------------
def _ssm_weights(H, G, N, V, taps, seed=1):
    C = H * V + 2 * G * N
    return dict(conv_w=rnd(taps, C, seed=seed, std=0.5), conv_b=rnd(C, seed=seed + 1, std=0.3),
                dt_bias=rnd(H, seed=seed + 2, std=0.8, mean=-1.5), a_log=rnd(H, seed=seed + 3, std=0.8, mean=-0.5)), \
        rnd(H, seed=seed + 4)


def _activated(rows, w, H, G, N, V):
    """rows [T, x | B | C | dt] before the convolution -> (activated x | B | C, dt)."""
    C = H * V + 2 * G * N
    r = rows.double()
    dt = torch.nn.functional.softplus(r[:, C:C + H] + w["dt_bias"].double(), threshold=1e9)
    return P.silu(P.short_conv(r[:, :C], w["conv_w"].double().T, w["conv_b"].double())), dt


def _walk(xbc, dt, w, skip, H, G, N, V, state=None):
    T, inner = xbc.shape[0], H * V
    of = torch.tensor([h // (H // G) for h in range(H)])
    y, S = P.state_space(xbc[:, :inner].view(T, H, V), xbc[:, inner:inner + G * N].view(T, G, N),
                         xbc[:, inner + G * N:].view(T, G, N), dt, w["a_log"].double(), skip.double(), of,
                         state)
    return y.reshape(T, inner), S


SSM_SIZES = [(6, 2, 14, 10, 3), (4, 4, 8, 8, 1), (1, 1, 1, 8, 2), (5, 1, 9, 7, 5), (8, 2, 64, 32, 4),
             (3, 1, 128, 64, 4), (4, 2, 80, 32, 3), (2, 1, 200, 96, 4), (4, 1, 16, 128, 4), (2, 2, 256, 16, 2),
             (2, 1, 500, 12, 4)]


@pytest.mark.parametrize("H, G, N, V, taps", SSM_SIZES)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_state_space(ops, H, G, N, V, taps, dtype):
    """Two requests in two slots, in portions of one to 150 tokens (longer and shorter than the
    convolution, the staged portions and the chunks), single tokens through the launch of their
    own; the slots start cleared, the others stay untouched.  The
    activated rows are compared by themselves (they may be kept in bfloat16); the plain walk takes
    them as they are, so that what is left of the recurrence's error is float32's."""
    w, skip = _ssm_weights(H, G, N, V, taps)
    wd, sk = {k: dev(v) for k, v in w.items()}, dev(skip)
    C = H * V + 2 * G * N
    sizes = dict(heads=H, groups=G, state_dim=N, vdim=V, taps=taps)
    rows = {"a": rnd(420, C + H, seed=11), "b": rnd(160, C + H, seed=12)}
    acts = {r: _activated(x, w, H, G, N, V) for r, x in rows.items()}
    states = {r: torch.zeros(H, N, V, dtype=F64) for r in rows}
    x_off, width = 8, 8 + C + H + (-(C + H)) % 8
    state = torch.full((4, H * N * V + taps * C), 7.0, device=DEV)
    slot = {"a": 2, "b": 0}
    for s in slot.values():
        state[s] = 0.0
    fed = {"a": 0, "b": 0}
    steps = [[("a", 1)], [("a", 2), ("b", 5)], [("b", 1), ("a", 1)], [("a", 150), ("b", 1)], [("a", 1)],
             [("b", 64), ("a", 3)], [("a", 1), ("b", 1)]] + [[("b", 1)]] * 5 + \
            [[("a", 65), ("b", 70)], [("b", 2)], [("a", 130)], [("a", 1)]]
    tol, chunked = 3e-5, 0
    for step in steps:
        T = sum(k for _r, k in step)
        act, rt = None, F32
        proj = torch.full((T, width), float("nan"))
        proj[:, x_off:x_off + C + H] = torch.cat([rows[r][fed[r]:fed[r] + k] for r, k in step])
        proj = dev(proj)
        starts, at = [], 0
        for _r, k in step:
            starts.append(at)
            at += k
        tok_pos = ints(p for r, k in step for p in range(fed[r], fed[r] + k))
        tok_req = ints(i for i, (_r, k) in enumerate(step) for _ in range(k))
        start, length = ints(starts), ints(k for _r, k in step)
        slots = ints(slot[r] for r, _k in step)
        y = torch.full((T, H * V), float("nan"), device=DEV)
        if all(k == 1 for _r, k in step):
            ops.ssm_step(y, state, proj, sk, tok_req, tok_pos, slots, x_off=x_off, **wd, **sizes)
        else:
            rt = ops.ssm_rows_dtype(dtype, T, sizes)
            chunked += rt == BF16
            act = torch.full((T, C), float("nan"), dtype=rt, device=DEV)
            dts = torch.full((T, 2 * H), float("nan"), device=DEV)
            ops.ssm_prepare(act, dts, proj, state, tok_req, tok_pos, start, slots, x_off=x_off, **wd, **sizes)
            ops.ssm_recurrence(y, state, act, dts, proj, sk, tok_pos, start, length, slots, x_off=x_off, **sizes)
        at = 0
        for r, k in step:
            xbc, dt = (v[fed[r]:fed[r] + k] for v in acts[r])
            if act is not None:
                close(act[at:at + k], xbc, 1e-5 if rt == F32 else 4e-3)
                xbc = act[at:at + k].cpu().double()
            want, states[r] = _walk(xbc, dt, w, skip, H, G, N, V, states[r])
            close(y[at:at + k], want, tol)
            at += k
            fed[r] += k
    for r in rows:
        close(state[slot[r], :H * N * V].view(H, N, V), states[r], tol)
    assert (chunked > 3) == (dtype == BF16 and N % 16 == 0 and V % 16 == 0 and N * V < 16384)
    assert bool((state[1] == 7.0).all()) and bool((state[3] == 7.0).all())


def test_state_space_long_single_steps(ops):
    """Hundreds of single-token steps on a state that hardly decays."""
    H, G, N, V, taps = 4, 2, 24, 16, 4
    w, skip = _ssm_weights(H, G, N, V, taps)
    w["a_log"] = torch.full((H,), -7.0)
    wd, sk = {k: dev(v) for k, v in w.items()}, dev(skip)
    C = H * V + 2 * G * N
    rows = rnd(360, C + H, seed=21)
    want, _ = _walk(*_activated(rows, w, H, G, N, V), w, skip, H, G, N, V)
    state = torch.zeros(1, H * N * V + taps * C, device=DEV)
    for t in range(360):
        y = torch.zeros(1, H * V, device=DEV)
        ops.ssm_step(y, state, dev(rows[t:t + 1]), sk, ints([0]), ints([t]), ints([0]), x_off=0, **wd,
                     heads=H, groups=G, state_dim=N, vdim=V, taps=taps)
        if t % 13 == 0 or t > 350:
            close(y[0], want[t], 3e-5)
