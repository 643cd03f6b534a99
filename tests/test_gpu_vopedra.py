"""Vopedra's mechanisms (matrix memory, HGRN2, selective scan per channel, attention with softmax weights mixed across heads,
the residual step, the gated unit), each kernel alone against the plain oracle of tests/vopedra_oracle.py; whole models are in
tests/test_gpu_vopedra_models.py."""
import math

import pytest
import torch

import vopedra_oracle as O

pytestmark = pytest.mark.gpu

PAGE = 32
F64 = torch.float64


def _batch(portions):
    """portions: [(slot, first position, rows)] in batch order; row numbers are dealt out backwards, so that a row's number says
    nothing about its place.  Returns (descriptor, tensors to keep alive, row numbers per portion)."""
    from dllama_b200.ops import layers as L
    M = sum(n for _, _, n in portions)
    pos, row_seq, rows, start = [0] * M, [0] * M, [], [0]
    owner = []
    nxt = M - 1
    for k, (slot, p0, n) in enumerate(portions):
        mine = []
        for i in range(n):
            pos[nxt], row_seq[nxt] = p0 + i, k
            mine.append(nxt)
            nxt -= 1
        rows += mine
        owner.append(mine)
        start.append(len(rows))
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    keep = [i32(pos), i32(row_seq), i32(start), i32(rows), i32([s for s, _, _ in portions]), i32([p for _, p, _ in portions])]
    return L.mamba_batch(*keep), keep, owner


def _image_rows(xh, ncap, M, K):
    """The bf16 activation image read back as [M][round_up(K, 128)] f32."""
    KP = (K + 127) // 128 * 128
    t = xh[:KP // 128 * (ncap // 8) * 2048].view(torch.bfloat16).view(KP // 128, ncap // 8, 16, 8, 8)      # [K tile][row group][8-column group][row][column]
    return t.permute(1, 3, 0, 2, 4).reshape(ncap, KP)[:M].float()


# ---------------------------------------------------------------------------------------------------------------------
# matrix memory: gates and scan
# ---------------------------------------------------------------------------------------------------------------------
def _gate_inputs(T, H, seed, bias_i=0.0, bias_f=2.0, spread=3.0):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(T, H, generator=g) * spread, torch.randn(T, H, generator=g) * spread, \
        torch.randn(H, generator=g) + bias_i, torch.randn(H, generator=g) + bias_f


def _run_gates(zi, zf, bi, bf, cap, slot, portions, n_slots=3, u0=None):
    """Feeds [T, H] gate inputs of ONE sequence in portions; returns (log_keep, put, floor) [T, H] and u_state."""
    from dllama_b200.ops import layers as L
    T, H = zi.shape
    u = torch.full((n_slots, H), 77.0, device="cuda") if u0 is None else u0
    outs = [torch.zeros(T, H) for _ in range(3)]
    at = 0
    for n in portions:
        b, keep, owner = _batch([(slot, at, n)])
        z = torch.zeros(n, 2 * H + 3, device="cuda")
        rows = torch.tensor(owner[0])
        z[rows.cuda(), :H], z[rows.cuda(), H:2 * H] = zi[at:at + n].cuda(), zf[at:at + n].cuda()
        lk, put, fl = (torch.zeros(n * H, device="cuda") for _ in range(3))
        L.mlstm_gates(b, 1, z, z[:, H:], bi.cuda(), bf.cuda(), cap, u, lk, put, fl, H, n)
        for o, v in zip(outs, (lk, put, fl)):
            o[at:at + n] = v.view(n, H).cpu()[rows]
        at += n
    assert at == T
    return outs, u


@pytest.mark.parametrize("cap", [3.0, 11.0, 30.0])
@pytest.mark.parametrize("portions", [[1], [1] * 40, [40, 1, 87, 2, 130], [300], [1500, 3]])
def test_matrix_memory_gates(cap, portions):
    T, H = sum(portions), 3
    zi, zf, bi, bf = _gate_inputs(T, H, 5)
    zi[T // 3] += 40.0                                        # an input gate that takes the running maximum over
    if T > 4:
        zf[T // 2] -= 60.0                                    # a forget gate that closes
    (lk, put, fl), u = _run_gates(zi, zf, bi, bf, cap, 1, portions)
    a, b = O.mlstm_gates(zi.double() + bi.double(), zf.double() + bf.double(), cap)
    m = torch.zeros(H, dtype=F64)
    for t in range(T):
        m1 = torch.maximum(b[t] + m, a[t])
        assert torch.allclose(lk[t].double(), b[t] + m - m1, atol=2e-5, rtol=2e-5), t
        assert torch.allclose(put[t].double(), torch.exp(a[t] - m1), atol=1e-6, rtol=3e-5), t
        assert torch.allclose(fl[t].double(), torch.exp(-m1), rtol=3e-5, atol=1e-9), t
        m = m1
    assert torch.allclose(u[1].cpu().double(), m, atol=2e-5) and bool((u[0] == 77.0).all()) and bool((u[2] == 77.0).all())


def _memory_case(T, H, d, dv, seed):
    """A memory with a far write that stands out: at one early token the input gate opens wide, its key is the direction of a
    late query, and the forget gates in between stay open -- what is read late is that token's value."""
    g = torch.Generator().manual_seed(seed)
    q, k, v = (torch.randn(T, H, n, generator=g) for n in (d, d, dv))
    a, b = O.mlstm_gates((torch.randn(T, H, generator=g) - 1).double(), (torch.randn(T, H, generator=g) + 4).double(), 9.0)
    if T > 8:
        a[2] += 6.0
        k[2] *= 3.0
        q[T - 1] = k[2] * 2.0
    return q, k, v, a, b


def _split(T, sizes):
    out, at = [], 0
    while at < T:
        for s in sizes:
            n = min(s, T - at)
            if n:
                out.append(n)
            at += n
    return out


SIZES = [(2, 8, 8), (3, 20, 36), (1, 32, 64), (2, 64, 130), (1, 100, 40), (2, 128, 256), (1, 200, 48)]


@pytest.mark.parametrize("H,d,dv", SIZES + [(1, 300, 24)])
@pytest.mark.parametrize("sizes", [[300], [1, 1, 2, 7, 130, 64, 65], [63, 128, 1]])
def test_matrix_memory_scan(H, d, dv, sizes):
    """Head form, chunked (portions of 128 rows and more, where the kernel takes the size) and token by token in one sequence,
    the state carried across portions in a slot that held something else."""
    from dllama_b200.ops import layers as L
    T = 300
    q, k, v, a, b = _memory_case(T, H, d, dv, 11)
    want_o, (S, n, u) = O.mlstm_rows(q.double() * d ** -0.5, k.double(), v.double(), a, b)
    state, n_state = torch.randn(2, H, d, dv, device="cuda"), torch.randn(2, H, d, device="cuda")
    other = state[0].clone()
    m, at = torch.zeros(H, dtype=F64), 0
    can = L.gated_chunked_supported(d, dv, False)
    assert can or d > 256
    for cnt in _split(T, sizes):
        lk, put, fl = [], [], []
        for t in range(at, at + cnt):
            m1 = torch.maximum(b[t] + m, a[t])
            lk.append(b[t] + m - m1)
            put.append(torch.exp(a[t] - m1))
            fl.append(torch.exp(-m1))
            m = m1
        bd, keep, owner = _batch([(1, at, cnt)])
        rows = torch.tensor(owner[0])
        put_rows = lambda x: torch.zeros(cnt, x.shape[1]).index_copy_(0, rows, x.float()).cuda()
        x = put_rows(torch.cat([q[at:at + cnt].reshape(cnt, -1), k[at:at + cnt].reshape(cnt, -1), v[at:at + cnt].reshape(cnt, -1)], 1))
        lkr, putr = put_rows(torch.stack(lk)), put_rows(torch.stack(put))
        y, den = torch.zeros(cnt, H * dv, device="cuda"), torch.zeros(cnt * H, device="cuda")
        kw = {}
        if can and cnt >= 128:
            slots = cnt // L.GATED_CHUNK + 1
            kw = dict(max_chunks=-(-cnt // L.GATED_CHUNK), chunk_slots=slots,
                      scratch=torch.full((L.gated_chunk_floats(cnt, 1, H, d, dv),), float("nan"), device="cuda"))
        L.gated_scan(bd, 1, x, x[:, 2 * H * d:], y, state, H, d, dv, q_scale=d ** -0.5, k=x[:, H * d:], log_keep=lkr, put=putr, den=den,
                     n_state=n_state, **kw)
        o = y.cpu()[rows].double().view(cnt, H, dv)
        dn = torch.maximum(den.cpu().view(cnt, H)[rows].double().abs(), torch.stack(fl)) + 1e-6
        got = o / dn[:, :, None]
        err = (got - want_o[at:at + cnt]).abs().amax((1, 2)) / (want_o[at:at + cnt].abs().amax((1, 2)) + 1e-3)
        assert float(err.max()) < 2e-4, (at, cnt, int(err.argmax()), float(err.max()))
        at += cnt
    assert torch.allclose(state[1].cpu().double(), S, atol=1e-4 * float(S.abs().max())) and torch.allclose(n_state[1].cpu().double(), n, atol=1e-4 * float(n.abs().max()))
    assert bool((state[0] == other).all())


@pytest.mark.parametrize("H,d,dv", SIZES + [(1, 276, 16), (1, 300, 24)])
@pytest.mark.parametrize("sizes", [[300], [1, 1, 2, 7, 130, 64, 65], [63, 128, 1]])
def test_hgrn2_scan(H, d, dv, sizes):
    """Channel form.  Some gates sit at their lower bound of zero for a token (everything before is forgotten at once), some at
    one (nothing is written): quotients of decays would overflow or divide by zero."""
    from dllama_b200.ops import layers as L
    T = 300
    g = torch.Generator().manual_seed(13)
    q, z, v = torch.randn(T, H, d, generator=g), torch.randn(T, H, d, generator=g) * 2 + 3, torch.randn(T, H, dv, generator=g)
    bias, lower = torch.randn(H * d, generator=g), torch.rand(H * d, generator=g) * 0.9
    lower[:: 3] = 0.0
    z[40::37, :, ::3] = -200.0                                # f = 0 exactly
    z[20::29, :, 1::4] = 200.0                                # f = 1 exactly
    f = lower.double() + (1 - lower.double()) / (1 + torch.exp(-(z.reshape(T, -1).double() + bias.double())))
    f = f.view(T, H, d)
    want, S = O.gated_rows(O.silu(q.double()), 1 - f, v.double(), f)
    state = torch.randn(2, H, d, dv, device="cuda")
    can = L.gated_chunked_supported(d, dv, True)
    assert can or d > 256
    at = 0
    for cnt in _split(T, sizes):
        bd, keep, owner = _batch([(1, at, cnt)])
        rows = torch.tensor(owner[0])
        x = torch.zeros(cnt, H * (2 * d + dv)).index_copy_(0, rows, torch.cat([q[at:at + cnt].reshape(cnt, -1), z[at:at + cnt].reshape(cnt, -1),
                                                                              v[at:at + cnt].reshape(cnt, -1)], 1)).cuda()
        y = torch.zeros(cnt, H * dv, device="cuda")
        kw = {}
        if can and cnt >= 128:
            kw = dict(max_chunks=-(-cnt // L.GATED_CHUNK), chunk_slots=cnt // L.GATED_CHUNK + 1,
                      scratch=torch.full((L.gated_chunk_floats(cnt, 1, H, d, dv),), float("nan"), device="cuda"))
        L.gated_scan(bd, 1, x, x[:, 2 * H * d:], y, state, H, d, dv, q_silu=True, f=x[:, H * d:], f_bias=bias.cuda(), lower=lower.cuda(), **kw)
        err = (y.cpu()[rows].double().view(cnt, H, dv) - want[at:at + cnt]).abs().amax((1, 2)) / (want[at:at + cnt].abs().amax((1, 2)) + 0.1)
        assert float(err.max()) < 1e-4, (at, cnt, int(err.argmax()), float(err.max()))
        at += cnt
    assert torch.allclose(state[1].cpu().double(), S, atol=1e-4 * float(S.abs().max()))


def test_gated_scans_of_unequal_sequences_in_one_batch():
    """Three sequences of 200, 1 and 65 rows (two fresh, one going on) in one chunked launch, against each alone."""
    from dllama_b200.ops import layers as L
    H, d, dv = 2, 40, 72
    g = torch.Generator().manual_seed(17)
    spec = [(2, 0, 200), (0, 9, 1), (1, 0, 65)]
    M = sum(n for _, _, n in spec)
    x, bias, lower = torch.randn(M, H * (2 * d + dv), generator=g).cuda(), torch.randn(H * d, generator=g).cuda(), torch.rand(H * d, generator=g).cuda() * 0.5
    start = torch.randn(3, H, d, dv, device="cuda")
    bd, keep, owner = _batch(spec)
    y, state = torch.zeros(M, H * dv, device="cuda"), start.clone()
    scratch = torch.full((L.gated_chunk_floats(M, 3, H, d, dv),), float("nan"), device="cuda")
    L.gated_scan(bd, 3, x, x[:, 2 * H * d:], y, state, H, d, dv, q_silu=True, f=x[:, H * d:], f_bias=bias, lower=lower, max_chunks=4,
                 scratch=scratch, chunk_slots=M // L.GATED_CHUNK + 3)
    for (slot, p0, n), rows in zip(spec, owner):
        b1, keep1, own1 = _batch([(slot, p0, n)])
        x1, y1, s1 = torch.zeros(n, x.shape[1], device="cuda"), torch.zeros(n, H * dv, device="cuda"), start.clone()
        x1[own1[0]] = x[rows]
        L.gated_scan(b1, 1, x1, x1[:, 2 * H * d:], y1, s1, H, d, dv, q_silu=True, f=x1[:, H * d:], f_bias=bias, lower=lower)
        assert torch.allclose(y[rows], y1[own1[0]], atol=2e-4, rtol=2e-4) and torch.allclose(state[slot], s1[slot], atol=2e-4, rtol=2e-4)


@pytest.mark.parametrize("H,dv,full", [(1, 5, True), (3, 24, False), (4, 64, True), (9, 128, False), (2, 300, True), (2, 600, False)])
def test_head_norm(H, dv, full):
    from dllama_b200.ops import layers as L
    M, eps = 37, 1e-3
    g = torch.Generator().manual_seed(19)
    y, den, fl = torch.randn(M, H * dv, generator=g), torch.randn(M, H, generator=g), torch.rand(M, H, generator=g)
    y[0], den[1], fl[1] = 1e-3, 0.0, 0.0                      # eps inside the root shows; the 1e-6 keeps the quotient finite
    w, gate = torch.randn(H * dv if full else dv, generator=g), torch.randn(M, H * dv, generator=g) * 2
    for with_den in (True, False):
        o = y.double().view(M, H, dv)
        if with_den:
            o = o / (torch.maximum(den.double().abs(), fl.double()) + 1e-6)[:, :, None]
        want = (O.unit(o, eps) * (w.double().view(H, dv) if full else w.double())).view(M, H * dv)
        want = want / (1 + torch.exp(-gate.double())) if with_den else want
        out = torch.zeros(M, H * dv, device="cuda")
        kw = dict(den=den.cuda().view(-1), floor=fl.cuda().view(-1), gate=gate.cuda()) if with_den else {}
        L.head_norm(y.cuda(), M, H, dv, eps, w.cuda(), out, **kw)
        assert torch.allclose(out.cpu().double(), want, atol=1e-5, rtol=1e-5)
        ncap = 40
        xh = torch.full((L.xh_bytes(H * dv, ncap),), 0x7f, dtype=torch.uint8, device="cuda")
        L.head_norm(y.cuda(), M, H, dv, eps, w.cuda(), None, image=(xh, ncap), **kw)
        img = _image_rows(xh, ncap, M, H * dv).cpu()
        assert torch.equal(img[:, :H * dv], out.cpu().bfloat16().float()) and bool((img[:, H * dv:] == 0).all())


# ---------------------------------------------------------------------------------------------------------------------
# selective scan per channel
# ---------------------------------------------------------------------------------------------------------------------
def _selective_case(T, c, n, seed):
    g = torch.Generator().manual_seed(seed)
    x, dt, z = (torch.randn(T, c, generator=g) for _ in range(3))
    B, C = torch.randn(T, n, generator=g), torch.randn(T, n, generator=g)
    A_log, bias, D = torch.randn(c, n, generator=g) - 1, torch.randn(c, generator=g) - 3, torch.randn(c, generator=g)
    dt[T // 2:T // 2 + 2] += 30.0                             # a step so large that every fast state is gone behind it
    if T > 8:
        x[1], dt[1], B[1] = 8.0, 3.0, 2.0                     # an early token written with a large step ...
        A_log[: c // 2] -= 6.0                                # ... that slow channels still hold at the end
    return x, dt, z, B, C, A_log, bias, D


@pytest.mark.parametrize("c,n", [(5, 3), (33, 8), (64, 16), (130, 24), (256, 32), (31, 33), (40, 64), (20, 100)])
@pytest.mark.parametrize("sizes", [[260], [1] * 7 + [2, 3, 16, 17, 130, 63], [64, 128]])
def test_selective_scan(c, n, sizes):
    from dllama_b200.ops import layers as L
    T, r = 260, 7
    x, dt, z, B, C, A_log, bias, D = _selective_case(T, c, n, 23)
    step = O.softplus(dt.double() + bias.double())
    y, S = O.selective_rows(x.double(), step, -torch.exp(A_log.double()), B.double(), C.double())
    want = (y + D.double() * x.double()) * O.silu(z.double())
    A2 = (-torch.exp(A_log.double()) / math.log(2.0)).float().cuda()
    state = torch.randn(2, c, n, device="cuda")
    other, at = state[0].clone(), 0
    can = L.selective_chunked_supported(n)
    assert can == (n <= 32)
    for k, cnt in enumerate(_split(T, sizes)):
        bd, keep, owner = _batch([(1, at, cnt)])
        rows = torch.tensor(owner[0])
        put = lambda t: torch.zeros(cnt, t.shape[1]).index_copy_(0, rows, t[at:at + cnt]).cuda()
        xs, dts, zs, dbc = put(x), put(dt), put(z), torch.cat([torch.full((cnt, r), 9.0, device="cuda"), put(B), put(C)], 1).contiguous()
        kw = {}
        if can and cnt >= 128:
            slots = cnt // L.SELECTIVE_CHUNK + 1
            kw = dict(max_chunks=-(-cnt // L.SELECTIVE_CHUNK), chunk_slots=slots, scratch=torch.full((slots * c * (n + 1),), float("nan"), device="cuda"))
        ncap = (cnt + 7) // 8 * 8
        image = k % 2 == 1                                    # every other portion leaves through the bf16 image
        out, xh = torch.zeros(cnt, c, device="cuda"), torch.full((L.xh_bytes(c, ncap),), 0x7f, dtype=torch.uint8, device="cuda")
        L.selective_scan(bd, 1, xs, dts, dbc[:, r:], dbc[:, r + n:], bias.cuda(), A2, D.cuda(), state, None if image else out, c, n, cnt, z=zs,
                         image=(xh, ncap) if image else None, **kw)
        w = want[at:at + cnt]
        if image:
            img = _image_rows(xh, ncap, cnt, c).cpu()
            assert bool((img[:, c:] == 0).all())
            got, tol = img[rows, :c].double(), 6e-3
        else:
            got, tol = out.cpu()[rows].double(), 1e-4
        err = (got - w).abs() / (w.abs() + w.abs().amax(1, keepdim=True) * 0.05 + 1e-2)
        assert float(err.max()) < tol, (at, cnt, float(err.max()))
        at += cnt
    assert torch.allclose(state[1].cpu().double(), S, atol=1e-4 * float(S.abs().max()), rtol=1e-3) and bool((state[0] == other).all())


def test_selective_scan_of_unequal_sequences_in_one_batch():
    from dllama_b200.ops import layers as L
    c, n = 70, 12
    spec = [(1, 0, 150), (2, 5, 1), (0, 0, 64), (3, 7, 3)]
    M = sum(k for _, _, k in spec)
    x, dt, z, B, C, A_log, bias, D = (t.cuda() for t in _selective_case(M, c, n, 29))
    A2, start = -torch.exp(A_log) / math.log(2.0), torch.randn(4, c, n, device="cuda")
    bd, keep, owner = _batch(spec)
    y, state, slots = torch.zeros(M, c, device="cuda"), start.clone(), M // L.SELECTIVE_CHUNK + 4
    L.selective_scan(bd, 4, x, dt, B, C, bias, A2, D, state, y, c, n, 150, z=z, max_chunks=3, chunk_slots=slots,
                     scratch=torch.full((slots * c * (n + 1),), float("nan"), device="cuda"))
    for (slot, p0, k), rows in zip(spec, owner):
        b1, keep1, own = _batch([(slot, p0, k)])
        alone = [torch.zeros(k, t.shape[1], device="cuda").index_copy_(0, torch.tensor(own[0]).cuda(), t[rows]) for t in (x, dt, z, B, C)]
        y1, s1 = torch.zeros(k, c, device="cuda"), start.clone()
        L.selective_scan(b1, 1, alone[0], alone[1], alone[3], alone[4], bias, A2, D, s1, y1, c, n, k, z=alone[2])
        assert torch.allclose(y[rows], y1[own[0]], atol=1e-3, rtol=1e-3) and torch.allclose(state[slot], s1[slot], atol=1e-3, rtol=1e-3)


# ---------------------------------------------------------------------------------------------------------------------
# attention with softmax weights mixed across heads
# ---------------------------------------------------------------------------------------------------------------------
def _case(T, H, G, d, dv, seed):
    """For chosen queries one key far back (position 0, a page border, the query's own place, ...) is made the direction of one of
    the query's heads, so that its weight is near one: a kernel that misses the key, the value head or the mix returns another
    value."""
    g = torch.Generator().manual_seed(seed)
    q, k, v = torch.randn(T, H, d, generator=g), torch.randn(T, G, d, generator=g), torch.randn(T, G, dv, generator=g)
    talk = torch.eye(H) * 0.8 + torch.randn(H, H, generator=g) * 0.5
    places = [0, 1, 31, 32, 33, 63, 64]
    for n, i in enumerate(range(3, T, 5)):
        j = (places + [i, i - 1, max(0, i - 100)])[n % 10]
        if j <= i:
            h = n % H
            u = k[j, h // (H // G)]
            q[i, h] = u / u.norm() ** 2 * 40.0
    return q, k, v, talk


def _rows(q, k, v, talk, scale, ctype, tc, portions, n_splits=1, image=False):
    from dllama_b200.ops import layers as L
    T, H, d = q.shape
    G, dv = k.shape[1], v.shape[2]
    n_pages = (T + PAGE - 1) // PAGE
    cache = (torch.randn(n_pages + 2, G, PAGE, d + dv, device="cuda") * 50).to(ctype)
    table = torch.tensor([[0] * n_pages, list(range(n_pages + 1, 1, -1))], dtype=torch.int32, device="cuda")
    freqs, tk, out = torch.zeros(1, dtype=F64, device="cuda"), talk.float().cuda().contiguous(), []
    for p0, n in portions:
        pos, slot = torch.arange(p0, p0 + n, dtype=torch.int32, device="cuda"), torch.ones(n, dtype=torch.int32, device="cuda")
        qq, kk, vv = (t[p0:p0 + n].reshape(n, -1).float().cuda().contiguous() for t in (q, k, v))
        L.window_kv_write(kk, n, G, d, 0, freqs, 1.0, pos, slot, table, cache, q=qq, q_heads=H, v=vv, vdim=dv)
        wide = torch.full((n, H * G * dv), float("nan"), device="cuda")
        if tc:
            rq = L.talk_tc_rows(H, G, d, dv, 0, n, G)
            tiles = [list(range(i, min(i + rq, n))) for i in range(0, n, rq)]
            L.talk_attention_tiles(qq, wide, H, G, d, dv, scale, 0, pos, slot, table, cache, tiles, rq, n_splits=n_splits, value_heads=G)
        else:
            L.window_attention(qq, wide, n, H, G, d, 0, scale, 0.0, 0, pos, slot, table, cache, vdim=dv, value_heads=G)
        o = torch.zeros(n, H * dv, device="cuda")
        if image:
            ncap = (n + 7) // 8 * 8
            xh = torch.full((L.xh_bytes(H * dv, ncap),), 0x7f, dtype=torch.uint8, device="cuda")
            L.talk_mix(wide, tk, n, H, G, dv, None, image=(xh, ncap))
            img = _image_rows(xh, ncap, n, H * dv)
            assert bool((img[:, H * dv:] == 0).all())
            o = img[:, :H * dv].contiguous()
        else:
            L.talk_mix(wide, tk, n, H, G, dv, o)
        out.append(o.cpu())
    return torch.cat(out).double().reshape(T, H, dv)


HEADS = [(2, 1, 16, 24), (4, 2, 32, 64), (6, 3, 24, 40), (4, 4, 40, 8), (8, 4, 64, 128), (10, 5, 16, 72), (16, 4, 128, 128)]


@pytest.mark.parametrize("H,G,d,dv", HEADS + [(6, 2, 9, 5)])
def test_mixed_weights_per_row_kernel(H, G, d, dv):
    T = 140
    q, k, v, talk = _case(T, H, G, d, dv, 31)
    want = O.softmax_then_mix_rows(q.double(), k.double(), v.double(), 1.0, talk.double())
    for portions in ([(0, T)], [(0, 33), (33, 1), (34, 2), (36, 64), (100, 40)]):
        got = _rows(q, k, v, talk, 1.0, torch.float32, False, portions)
        assert torch.allclose(got, want, atol=2e-4, rtol=2e-4), float((got - want).abs().max())


@pytest.mark.parametrize("H,G,d,dv", HEADS + [(32, 8, 64, 64), (16, 2, 32, 96), (9, 3, 24, 64)])
@pytest.mark.parametrize("n_splits", [1, 3, 16])
def test_mixed_weights_tile_kernel(H, G, d, dv, n_splits):
    from dllama_b200.ops import layers as L
    T = 140
    q, k, v, talk = _case(T, H, G, d, dv, 37)
    assert L.talk_tc_supported(H, G, d, dv, 0, torch.bfloat16, G)
    qb, kb, vb = (t.bfloat16().double() for t in (q, k, v))                   # what the kernel multiplies
    want = O.softmax_then_mix_rows(qb, kb, vb, 1.0, talk.double())
    for portions in ([(0, T)], [(0, 37), (37, 1), (38, 2), (40, 60), (100, 40)], [(i, 1) for i in range(T)] if n_splits > 1 and H <= 6 else [(0, 70), (70, 70)]):
        got = _rows(q, k, v, talk, 1.0, torch.bfloat16, True, portions, n_splits, image=len(portions) == 2)
        err = (got - want).abs().amax((1, 2))
        assert float(err.max()) < 0.05, (portions[:3], int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 32, 64), (8, 4, 64, 128), (6, 3, 24, 40)])
def test_mixed_weights_of_many_decoded_rows(H, G, d, dv):
    """One-row tiles by the hundred (batched decoding): one CTA serves all heads of a row."""
    from dllama_b200.ops import layers as L
    T = 300
    q, k, v, talk = _case(T, H, G, d, dv, 41)
    want = O.softmax_then_mix_rows(q.bfloat16().double(), k.bfloat16().double(), v.bfloat16().double(), 0.5, talk.double())
    n_pages = (T + PAGE - 1) // PAGE
    cache = torch.zeros(n_pages, G, PAGE, d + dv, dtype=torch.bfloat16, device="cuda")
    table = torch.arange(n_pages - 1, -1, -1, dtype=torch.int32, device="cuda").view(1, -1)
    pos, slot = torch.arange(T, dtype=torch.int32, device="cuda"), torch.zeros(T, dtype=torch.int32, device="cuda")
    qq, kk, vv = (t.reshape(T, -1).cuda().contiguous() for t in (q, k, v))
    L.window_kv_write(kk, T, G, d, 0, torch.zeros(1, dtype=F64, device="cuda"), 1.0, pos, slot, table, cache, q=qq, q_heads=H, v=vv, vdim=dv)
    rq = L.talk_tc_rows(H, G, d, dv, 0, 1, G)
    for n_splits in (1, 2):
        wide, o = torch.full((T, H * G * dv), float("nan"), device="cuda"), torch.zeros(T, H * dv, device="cuda")
        L.talk_attention_tiles(qq, wide, H, G, d, dv, 0.5, 0, pos, slot, table, cache, [[i] for i in range(T)], rq, n_splits=n_splits, value_heads=G)
        L.talk_mix(wide, talk.cuda().contiguous(), T, H, G, dv, o)
        assert float((o.cpu().double().view(T, H, dv) - want).abs().max()) < 0.05


def test_tile_kernel_without_a_mix_still_serves_plain_and_folded_heads():
    """The same kernel family with one value head per query head: identity mix of the wide form equals the plain form."""
    from dllama_b200.ops import layers as L
    H, G, d, dv, T = 6, 3, 32, 40, 90
    q, k, v, _ = _case(T, H, G, d, dv, 43)
    wide = _rows(q, k, v, torch.eye(H), 1.0, torch.bfloat16, True, [(0, T)])
    cache = torch.zeros(3, G, PAGE, d + dv, dtype=torch.bfloat16, device="cuda")
    table = torch.arange(3, dtype=torch.int32, device="cuda").view(1, -1)
    pos, slot = torch.arange(T, dtype=torch.int32, device="cuda"), torch.zeros(T, dtype=torch.int32, device="cuda")
    qq, kk, vv = (t.reshape(T, -1).cuda().contiguous() for t in (q, k, v))
    L.window_kv_write(kk, T, G, d, 0, torch.zeros(1, dtype=F64, device="cuda"), 1.0, pos, slot, table, cache, q=qq, q_heads=H, v=vv, vdim=dv)
    o = torch.zeros(T, H * dv, device="cuda")
    rq = L.talk_tc_rows(H, G, d, dv, 0, T)
    L.talk_attention_tiles(qq, o, H, G, d, dv, 1.0, 0, pos, slot, table, cache, [list(range(i, min(i + rq, T))) for i in range(0, T, rq)], rq)
    assert torch.allclose(o.cpu().double().view(T, H, dv), wide, atol=1e-3)


@pytest.mark.parametrize("H,G,d,dv,rot", [(4, 2, 32, 16, 32), (6, 3, 24, 40, 8), (3, 3, 10, 7, 0), (8, 1, 64, 64, 16)])
def test_cache_writer_norms_the_whole_projection_before_the_rotary(H, G, d, dv, rot):
    """Queries and keys: one root mean square over all heads' columns, weights per column, then the rotary; positions far out."""
    from dllama_b200.models.layered import rotary_frequencies
    from dllama_b200.ops import layers as L
    T, eps, base, p0 = 11, 1e-2, 700.0, 1000
    g = torch.Generator().manual_seed(47)
    q, k, v = (torch.randn(T, n, generator=g) for n in (H * d, G * d, G * dv))
    q[0] *= 0.01                                              # eps shows
    q[:, :d] *= 5.0                                           # one head dominates: a norm per head would come out otherwise
    wq, wk = torch.randn(H * d, generator=g), torch.randn(G * d, generator=g)
    pos = torch.arange(p0, p0 + T)
    want_q = O.rotate_half_pairs((wq.double() * O.unit(q.double(), eps)).view(T, H, d), pos, base, rot)
    want_k = O.rotate_half_pairs((wk.double() * O.unit(k.double(), eps)).view(T, G, d), pos, base, rot)
    n_pages = (p0 + T) // PAGE + 1
    cache = torch.zeros(2, G, PAGE, d + dv, device="cuda")
    table = torch.zeros(1, n_pages, dtype=torch.int32, device="cuda")
    table[0, (p0 // PAGE) + 1:] = 1
    qq = q.cuda()
    freqs = rotary_frequencies(base, rot).cuda() if rot else torch.zeros(1, dtype=F64, device="cuda")
    L.window_kv_write(k.cuda(), T, G, d, rot, freqs, 1.0, pos.int().cuda(), torch.zeros(T, dtype=torch.int32, device="cuda"), table, cache, q=qq,
                      q_heads=H, v=v.cuda(), vdim=dv, eps=eps, rope_half=True, q_norm=wq.cuda(), k_norm=wk.cuda())
    assert torch.allclose(qq.cpu().double().view(T, H, d), want_q, atol=1e-5, rtol=1e-5)
    for t in range(T):
        line = cache[int(table[0, (p0 + t) // PAGE]), :, (p0 + t) % PAGE].cpu().double()
        assert torch.allclose(line[:, :d], want_k[t], atol=1e-5, rtol=1e-5) and torch.equal(line[:, d:].float(), v[t].view(G, dv))


# ---------------------------------------------------------------------------------------------------------------------
# the residual step and the gated unit
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dim", [30, 88, 192, 1500, 2048, 5000, 9000])
def test_residual_step(dim):
    """Every subset of terms the engine uses; dims the four-column kernel takes and others; eps that shows; a gather of rows."""
    from dllama_b200.ops import layers as L
    M, eps = 21, 1e-2
    g = torch.Generator().manual_seed(53)
    r = lambda *s: torch.randn(*s, generator=g)
    x, a1, a2, a3, na, nb = (r(M, dim) for _ in range(6))
    na[0] *= 1e-2
    wa, wb, vec, w1, w2 = (r(dim) for _ in range(5))
    rows = torch.randint(0, M, (9,), generator=g, dtype=torch.int32)
    D = lambda t: t.double()
    for n_adds, n_norm, use_vec, use_rows, n_out in ((0, 0, False, False, 2), (2, 0, True, False, 2), (3, 0, True, False, 1), (1, 2, False, False, 2),
                                                     (2, 2, True, False, 2), (1, 2, False, True, 1), (0, 1, False, False, 0), (2, 0, False, True, 1)):
        adds, norms = [a1, a2, a3][:n_adds], [(na, wa), (nb, wb)][:n_norm]
        s = D(x) + sum(D(t) for t in adds) + sum(D(w) * O.unit(D(t), eps) for t, w in norms) + (D(vec) if use_vec else 0)
        n = len(rows) if use_rows else M
        if use_rows:
            s = s[rows.long()]
        xo, h1, h2 = (torch.zeros(n, dim, device="cuda") for _ in range(3))
        ncap = (n + 7) // 8 * 8
        xh = torch.full((L.xh_bytes(dim, ncap),), 0x7f, dtype=torch.uint8, device="cuda")
        kw = dict(x_in=x.cuda(), adds=[t.cuda() for t in adds], normed=[(t.cuda(), w.cuda()) for t, w in norms], vec=vec.cuda() if use_vec else None,
                  rows=rows.cuda() if use_rows else None)
        L.residual_step(n, dim, eps, x=xo, outs=[(w1.cuda(), h1), (w2.cuda(), h2)][:n_out], **kw)
        assert torch.allclose(xo.cpu().double(), s, atol=2e-5, rtol=1e-5)
        for w, h in [(w1, h1), (w2, h2)][:n_out]:
            assert torch.allclose(h.cpu().double(), D(w) * O.unit(s, eps), atol=2e-5, rtol=1e-5)
        if n_out:
            L.residual_step(n, dim, eps, outs=[(w1.cuda(), (xh, ncap))], **kw)
            img = _image_rows(xh, ncap, n, dim).cpu()
            assert torch.equal(img[:, :dim], h1.cpu().bfloat16().float()) and bool((img[:, dim:] == 0).all())
    if dim % 4 == 0 and dim <= 8192:                          # the rows of a bf16 table: the embedding
        table = r(40, dim).bfloat16()
        tok = torch.randint(0, 40, (M,), generator=g, dtype=torch.int32)
        out = torch.zeros(M, dim, device="cuda")
        L.residual_step(M, dim, eps, x_in=table.cuda(), rows=tok.cuda(), outs=[(w1.cuda(), out)])
        assert torch.allclose(out.cpu().double(), D(w1) * O.unit(table.double()[tok.long()], eps), atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("ff,W", [(7, 20), (24, 88), (128, 192), (200, 264), (384, 96)])
@pytest.mark.parametrize("M", [1, 3, 8, 9, 31, 40, 150])
def test_gated_unit(ff, W, M):
    """gelu(gate) * up on the weight-streaming and the tiled product (f32 and bf16) and on the tcgen05 product, to f32 rows or straight into
    the next product's image."""
    from dllama_b200.ops import layers as L
    g = torch.Generator().manual_seed(59)
    x, wg, wu = torch.randn(M, W, generator=g), torch.randn(ff, W, generator=g) / 4, torch.randn(ff, W, generator=g) / 4
    both = torch.stack([wg, wu], 1).reshape(2 * ff, W)
    want = O.gelu_tanh(x.double() @ wg.double().T) * (x.double() @ wu.double().T)
    y = torch.zeros(M, ff + 3, device="cuda")
    L.dense(both.cuda(), x.cuda(), y, M, False, epi=L.DENSE_GLU_GELU)
    assert torch.allclose(y[:, :ff].cpu().double(), want, atol=2e-4, rtol=2e-4) and bool((y[:, ff:] == 0).all())
    wb, xb = both.bfloat16(), x.bfloat16()
    gb, ub = wb.view(ff, 2, W)[:, 0].double(), wb.view(ff, 2, W)[:, 1].double()
    want = O.gelu_tanh(xb.double() @ gb.T) * (xb.double() @ ub.T)
    y.zero_()
    L.dense(wb.cuda(), x.cuda(), y, M, True, epi=L.DENSE_GLU_GELU)
    assert torch.allclose(y[:, :ff].cpu().double(), want, atol=2e-4, rtol=2e-4)
    ncap = (M + 7) // 8 * 8
    xh = torch.zeros(L.xh_bytes(W, ncap), dtype=torch.uint8, device="cuda")
    L.xh_from_rows(x.cuda(), M, W, ncap, xh)
    wh = L.make_wh(wb.cuda())
    y.zero_()
    L.dense_tc(wh, 2 * ff, W, xh, ncap, y, M, epi=L.DENSE_GLU_GELU)
    assert torch.allclose(y[:, :ff].cpu().double(), want, atol=2e-4, rtol=2e-4) and bool((y[:, ff:] == 0).all())
    if ff % 128 == 0:
        out = torch.zeros(L.xh_bytes(ff, ncap), dtype=torch.uint8, device="cuda")
        L.dense_tc(wh, 2 * ff, W, xh, ncap, y, M, epi=L.DENSE_GLU_GELU, image=(out, ncap))
        assert torch.equal(_image_rows(out, ncap, M, ff).cpu(), y[:, :ff].cpu().bfloat16().float())
