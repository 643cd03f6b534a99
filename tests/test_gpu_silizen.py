"""Silizen's mechanisms (gated linear attention, the gated delta rule, time mixing and its token shift, attention with a sink of score
zero, soft cap, distance bias and head gates, heads normed ahead of the rotary, unit heads behind the convolution, layer norms in the
residual step, products with bias), each kernel alone against the plain oracle of tests/silizen_oracle.py; whole models are in
tests/test_gpu_silizen_models.py."""
import pytest
import torch

import silizen_oracle as O

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module", autouse=True)
def _one_thread():
    """The oracle is thousands of small products: threads would only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)

PAGE = 32
F64 = torch.float64


def _batch(portions):
    """portions: [(slot, first position, rows)] in batch order; row numbers are dealt out backwards, so that a row's number says
    nothing about its place.  Returns (descriptor, tensors to keep alive, row numbers per portion)."""
    from dllama_b200.ops import layers as L
    M = sum(n for _, _, n in portions)
    pos, row_seq, rows, start, owner, nxt = [0] * M, [0] * M, [], [0], [], M - 1
    for k, (slot, p0, n) in enumerate(portions):
        mine = list(range(nxt, nxt - n, -1))
        nxt -= n
        for i, m in enumerate(mine):
            pos[m], row_seq[m] = p0 + i, k
        rows += mine
        owner.append(mine)
        start.append(len(rows))
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    keep = [i32(pos), i32(row_seq), i32(start), i32(rows), i32([s for s, _, _ in portions]), i32([p for _, p, _ in portions])]
    return L.mamba_batch(*keep), keep, owner


def _image_rows(xh, ncap, M, K):
    """The bf16 activation image read back as [M][round_up(K, 128)] f32."""
    KP = (K + 127) // 128 * 128
    t = xh[:KP // 128 * (ncap // 8) * 2048].view(torch.bfloat16).view(KP // 128, ncap // 8, 16, 8, 8)
    return t.permute(1, 3, 0, 2, 4).reshape(ncap, KP)[:M].float()


def _split(T, sizes):
    out, at = [], 0
    while at < T:
        for s in sizes:
            n = min(s, T - at)
            if n:
                out.append(n)
            at += n
    return out


# ---------------------------------------------------------------------------------------------------------------------
# the three recurrences
# ---------------------------------------------------------------------------------------------------------------------
class Rule:
    """One recurrence with its random inputs: `names` of the per-row inputs with their widths, the oracle and the launch."""

    def __init__(self, kind, T, H, d, dv, G=None, seed=1):
        g = torch.Generator().manual_seed(seed)
        self.kind, self.T, self.H, self.d, self.dv, self.G = kind, T, H, d, dv, G or H
        G = self.G
        rnd = lambda *s: torch.randn(*s, generator=g)
        self.q, self.k, self.v, self.z = rnd(T, G, d), rnd(T, G, d), rnd(T, H, dv), rnd(T, H, d)
        self.bias, self.beta = rnd(H * d), rnd(T, H) * 2
        if kind == "root":
            self.z, self.tau = self.z * 3 + 2, 5.0
            # an early write that a late query asks for; channels that forget at once and channels that keep all
            self.z[40::37, :, ::3], self.z[20::29, :, 1::4] = -2000.0, 200.0
        elif kind == "expexp":
            self.z, self.bonus = self.z - 3, rnd(H, d)
            self.z[40::37, :, ::3], self.z[20::29, :, 1::4] = 30.0, -60.0
        else:
            self.z, self.rate = self.z - 3, torch.rand(H, generator=g) * 2 + 0.1
            self.z[40::37, :, ::3], self.z[20::29, :, 1::4] = 90.0, -90.0
            self.q, self.k = (O.length_one(x.double()).float() for x in (self.q, self.k))
            self.beta[5], self.beta[T // 2] = 30.0, -30.0              # a token that is written whole, one that is not
            if T > 80:
                self.k[70] = self.k[69]                                # the same key again: the second write replaces the first
        if T > 8:
            self.q[T - 1] = self.k[T // 3] * 3
        zb = (self.z.reshape(T, -1).double() + self.bias.double()).view(T, H, d)
        rep = H // G
        q, k = (x.double().repeat_interleave(rep, 1) for x in (self.q, self.k))
        if kind == "root":
            f = O.root_sigmoid(zb, self.tau)
            self.run = lambda a, b, S: O.gated_rows(q[a:b] * 0.5, k[a:b], self.v[a:b].double(), f[a:b], S)
        elif kind == "expexp":
            f = torch.exp(-torch.exp(zb))
            self.run = lambda a, b, S: O.wkv_rows(q[a:b] * 0.5, k[a:b], self.v[a:b].double(), f[a:b], self.bonus.double(), S)
        else:
            f = O.delta_decay(zb, torch.log(self.rate.double()))
            self.run = lambda a, b, S: O.delta_rows(q[a:b] * 0.5, k[a:b], self.v[a:b].double(), f[a:b], O.sigmoid(self.beta[a:b].double()), S)

    def rows(self, a, b):
        n = b - a
        return torch.cat([x[a:b].reshape(n, -1) for x in (self.q, self.k, self.v, self.z, self.beta)], 1)

    def can_chunk(self):
        from dllama_b200.ops import layers as L
        return L.delta_chunked_supported(self.d, self.dv) if self.kind == "delta" else L.gated_chunked_supported(self.d, self.dv, True)

    def launch(self, batch, n_seq, x, y, state, chunks=0, slots=0):
        from dllama_b200.ops import layers as L
        H, G, d, dv, M = self.H, self.G, self.d, self.dv, x.shape[0]
        k0, v0, z0 = G * d, 2 * G * d, 2 * G * d + H * dv
        kw = {"root": lambda: dict(gate=L.GATE_ROOT_SIGMOID, tau=self.tau), "expexp": lambda: dict(gate=L.GATE_EXP_EXP, bonus=self.bonus.reshape(-1).cuda()),
              "delta": lambda: dict(gate=L.GATE_SOFTPLUS, rate=self.rate.cuda(), beta=x[:, z0 + H * d:])}[self.kind]()
        if chunks:
            floats = (L.delta_chunk_floats if self.kind == "delta" else L.gated_chunk_floats)(M, slots - M // L.GATED_CHUNK, H, d, dv)
            kw.update(max_chunks=chunks, chunk_slots=slots, scratch=torch.full((floats,), float("nan"), device="cuda"))
            if self.kind == "delta":
                kw["u"] = torch.full((M, H * dv), float("nan"), device="cuda")
        bias = self.bias.cuda()
        L.gated_scan(batch, n_seq, x, x[:, v0:], y, state, H, d, dv, q_scale=0.5, k=x[:, k0:], f=x[:, z0:], f_bias=bias, k_heads=G if G != H else 0, **kw)
        torch.cuda.synchronize()


SIZES = [(2, 8, 8), (3, 20, 36), (1, 32, 64), (2, 64, 130), (1, 100, 40), (2, 128, 144), (1, 200, 20), (2, 37, 5)]


@pytest.mark.parametrize("kind", ["root", "expexp", "delta"])
@pytest.mark.parametrize("H,d,dv", SIZES + [(1, 300, 24)])
@pytest.mark.parametrize("sizes", [[300], [1, 1, 2, 7, 130, 64, 65], [63, 128, 1]])
def test_recurrence(kind, H, d, dv, sizes):
    """Chunked (portions of 128 rows and more, where the kernels take the size) and token by token in one sequence, the state carried
    across portions in a slot that held something else; decays of exactly 0 and 1 (quotients of decays would break)."""
    from dllama_b200.ops import layers as L
    T = 300
    r = Rule(kind, T, H, d, dv)
    want, S = r.run(0, T, None)
    state = torch.randn(2, H, d, dv, device="cuda")
    other = state[0].clone()
    can = r.can_chunk()
    assert can or d > 256
    at = 0
    for cnt in _split(T, sizes):
        bd, keep, owner = _batch([(1, at, cnt)])
        rows = torch.tensor(owner[0])
        w = r.rows(at, at + cnt)
        x = torch.zeros(cnt, w.shape[1]).index_copy_(0, rows, w).cuda()
        y = torch.full((cnt, H * dv), float("nan"), device="cuda")
        r.launch(bd, 1, x, y, state, *((-(-cnt // L.GATED_CHUNK), cnt // L.GATED_CHUNK + 1) if can and cnt >= 128 else ()))
        err = (y.cpu()[rows].double().view(cnt, H, dv) - want[at:at + cnt]).abs().amax((1, 2)) / (want[at:at + cnt].abs().amax((1, 2)) + 0.1)
        assert float(err.max()) < 1e-4, (at, cnt, int(err.argmax()), float(err.max()))
        at += cnt
    assert torch.allclose(state[1].cpu().double(), S, atol=1e-4 * float(S.abs().max())) and bool((state[0] == other).all())


@pytest.mark.parametrize("kind", ["root", "expexp", "delta"])
def test_recurrence_of_unequal_sequences_in_one_batch(kind):
    """Three sequences of 200, 1 and 65 rows (two fresh, one going on) in one chunked launch, against the oracle of each alone."""
    from dllama_b200.ops import layers as L
    H, d, dv = 2, 40, 72
    spec = [(2, 0, 200), (0, 9, 1), (1, 0, 65)]
    r = Rule(kind, 266, H, d, dv, seed=3)
    start = torch.randn(3, H, d, dv) * 0.3
    state, at = start.clone().cuda(), 0
    bd, keep, owner = _batch(spec)
    x = torch.zeros(266, r.rows(0, 1).shape[1])
    for (slot, p0, n), rows in zip(spec, owner):
        x[rows] = r.rows(at, at + n)
        at += n
    y = torch.full((266, H * dv), float("nan"), device="cuda")
    r.launch(bd, 3, x.cuda(), y, state, 4, 266 // L.GATED_CHUNK + 3)
    at = 0
    for (slot, p0, n), rows in zip(spec, owner):
        want, S = r.run(at, at + n, start[slot].double() if p0 else None)
        assert torch.allclose(y.cpu()[rows].double().view(n, H, dv), want, atol=2e-4, rtol=2e-4), (kind, n)
        assert torch.allclose(state[slot].cpu().double(), S, atol=2e-4, rtol=2e-4)
        at += n


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 24, 16), (6, 1, 32, 40), (3, 3, 16, 8)])
@pytest.mark.parametrize("chunked", [False, True])
def test_delta_rule_heads_share_queries_and_keys(H, G, d, dv, chunked):
    from dllama_b200.ops import layers as L
    T = 150
    r = Rule("delta", T, H, d, dv, G=G, seed=5)
    want, S = r.run(0, T, None)
    bd, keep, owner = _batch([(0, 0, T)])
    rows = torch.tensor(owner[0])
    x = torch.zeros(T, r.rows(0, 1).shape[1]).index_copy_(0, rows, r.rows(0, T)).cuda()
    y, state = torch.zeros(T, H * dv, device="cuda"), torch.zeros(1, H, d, dv, device="cuda")
    r.launch(bd, 1, x, y, state, *((3, 3) if chunked else ()))
    assert torch.allclose(y.cpu()[rows].double().view(T, H, dv), want, atol=1e-4, rtol=1e-4) and torch.allclose(state[0].cpu().double(), S, atol=1e-4)


def test_delta_rule_over_many_chunks():
    """1000 rows with strong writes along few directions: every chunk's triangular system is far from the identity."""
    from dllama_b200.ops import layers as L
    T, H, d, dv = 1000, 1, 32, 24
    r = Rule("delta", T, H, d, dv, seed=7)
    g = torch.Generator().manual_seed(8)
    r.k = O.length_one((torch.randn(T, 1, 4, generator=g) @ torch.randn(4, d, generator=g)).double()).float()      # keys in a space of 4 dimensions
    r.beta[:] = 3.0
    f = O.delta_decay((r.z.reshape(T, -1).double() + r.bias.double()).view(T, H, d), torch.log(r.rate.double()))
    want, S = O.delta_rows(r.q.double() * 0.5, r.k.double(), r.v.double(), f, O.sigmoid(r.beta.double()))
    bd, keep, owner = _batch([(0, 0, T)])
    rows = torch.tensor(owner[0])
    x = torch.zeros(T, r.rows(0, 1).shape[1]).index_copy_(0, rows, r.rows(0, T)).cuda()
    y, state = torch.zeros(T, H * dv, device="cuda"), torch.zeros(1, H, d, dv, device="cuda")
    r.launch(bd, 1, x, y, state, 16, T // L.GATED_CHUNK + 1)
    err = (y.cpu()[rows].double().view(T, H, dv) - want).abs().amax((1, 2)) / (want.abs().amax((1, 2)) + 0.1)
    assert float(err.max()) < 2e-4, (int(err.argmax()), float(err.max()))


# ---------------------------------------------------------------------------------------------------------------------
# convolution with unit heads, token shift, head norm with a SiLU gate
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H,G,d,dv,taps", [(4, 2, 24, 16, 4), (1, 1, 8, 5, 1), (3, 3, 64, 130, 2), (2, 1, 150, 40, 7)])
@pytest.mark.parametrize("wtype", [torch.float32, torch.bfloat16])
def test_convolution_with_unit_heads(H, G, d, dv, taps, wtype):
    from dllama_b200.ops import layers as L
    T, ch, off = 41, 2 * G * d + H * dv, 3
    g = torch.Generator().manual_seed(9)
    x, w = torch.randn(T, ch, generator=g), torch.randn(ch, taps, generator=g).to(wtype)
    x[7] = 0.0                                                # a head of zeros stays zero; 1e-6 shows for the small ones
    x[8:8 + taps] *= 1e-3
    c = O.silu(O.causal_conv_rows(x.double(), w.double()))
    q, k = (O.length_one(t.reshape(T, G, d)).reshape(T, -1) for t in (c[:, :G * d], c[:, G * d:2 * G * d]))
    want = torch.cat([q * d ** -0.5, k, c[:, 2 * G * d:]], 1)
    state = torch.full((2, max(1, taps - 1), ch), 9.0, device="cuda")
    at = 0
    for n in (1, 2, 1, 20, 3, 14):
        bd, keep, owner = _batch([(1, at, n)])
        rows = torch.tensor(owner[0])
        xin = torch.zeros(n, ch + off + 5).index_copy_(0, rows, torch.cat([torch.full((n, off), 7.0), x[at:at + n], torch.zeros(n, 5)], 1)).cuda()
        out = torch.zeros(n, ch, device="cuda")
        L.causal_conv(bd, n, 1, xin, w.cuda(), state, out, act=True, in_off=off, unit=(d, G * d, 2 * G * d, d ** -0.5))
        assert torch.allclose(out.cpu()[rows].double(), want[at:at + n], atol=3e-6, rtol=1e-4), (at, n)
        at += n
    assert bool((state[0] == 9.0).all())


@pytest.mark.parametrize("W", [6, 88, 131, 2048])
def test_token_shift(W):
    """Rows and images, unequal sequences in one batch, the last row carried in a slot that held something else."""
    from dllama_b200.ops import layers as L
    g = torch.Generator().manual_seed(11)
    h, mu = torch.randn(60, W, generator=g), torch.rand(5, W, generator=g)
    want = torch.stack([O.token_shift(h.double(), mu[s].double()) for s in range(5)])
    h2 = torch.randn(9, W, generator=g)
    want2 = torch.stack([O.token_shift(h2.double(), mu[s].double()) for s in range(5)])
    state = torch.full((3, W), 5.0, device="cuda")
    at = 0
    for step, n in enumerate((1, 1, 2, 30, 26)):
        second = step in (1, 3)                               # the other sequence: rows 0 .. 3 in one step, 4 .. 8 two steps later
        a2, n2 = (0, 4) if step == 1 else (4, 5)
        bd, keep, owner = _batch([(2, at, n)] + ([(0, a2, n2)] if second else []))
        M = n + (n2 if second else 0)
        x = torch.zeros(M, W)
        x[owner[0]] = h[at:at + n]
        if second:
            x[owner[1]] = h2[a2:a2 + n2]
        before = state.clone()
        out = torch.full((5, M + 2, W), float("nan"), device="cuda")
        L.token_shift(bd, M, x.cuda(), mu.cuda(), state, out=out)
        assert torch.allclose(out.cpu()[:, owner[0]].double(), want[:, at:at + n], atol=1e-6)
        if second:
            assert torch.allclose(out.cpu()[:, owner[1]].double(), want2[:, a2:a2 + n2], atol=1e-6)
        ncap = (M + 7) // 8 * 8
        nb = L.xh_bytes(W, ncap)
        xh = torch.full((5, nb), 0x7f, dtype=torch.uint8, device="cuda")
        L.token_shift(bd, M, x.cuda(), mu.cuda(), before, images=(xh[0], nb, ncap))
        for s in range(5):
            img = _image_rows(xh[s], ncap, M, W)
            assert torch.equal(img[:, :W], out[s, :M].bfloat16().float()) and bool((img[:, W:] == 0).all())
        assert torch.equal(before, state) and bool((state[1] == 5.0).all())
        at += n
    assert torch.equal(state[2].cpu(), h[59]) and torch.equal(state[0].cpu(), h2[8])


@pytest.mark.parametrize("H,dv,full", [(1, 5, True), (3, 24, False), (9, 128, True), (2, 600, False)])
def test_head_norm_with_a_silu_gate(H, dv, full):
    from dllama_b200.ops import layers as L
    M, eps = 37, 1e-2
    g = torch.Generator().manual_seed(13)
    y, w, gate = torch.randn(M, H * dv, generator=g) * 0.3, torch.randn(H * dv if full else dv, generator=g), torch.randn(M, H * dv + 4, generator=g) * 3
    want = O.unit(y.double().view(M, H, dv), eps)
    want = want.reshape(M, -1) * (w.double() if full else w.double().repeat(H)) * O.silu(gate[:, :H * dv].double())
    out = torch.zeros(M, H * dv, device="cuda")
    L.head_norm(y.cuda(), M, H, dv, eps, w.cuda(), out, gate=gate.cuda(), gate_silu=True)
    assert torch.allclose(out.cpu().double(), want, atol=2e-5, rtol=2e-5)
    ncap = 40
    xh = torch.zeros(L.xh_bytes(H * dv, ncap), dtype=torch.uint8, device="cuda")
    L.head_norm(y.cuda(), M, H, dv, eps, w.cuda(), None, gate=gate.cuda(), gate_silu=True, image=(xh, ncap))
    assert torch.equal(_image_rows(xh, ncap, M, H * dv)[:, :H * dv], out.bfloat16().float())


# ---------------------------------------------------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------------------------------------------------
def _case(T, H, G, d, dv, seed, window=0):
    """For chosen queries one key (position 0, a page border, the query's own place, just inside or just outside the window, ...) is
    made the direction of one of the query's heads, so that its weight is near one where it is visible; the other queries are
    small, so that the sink takes a share that shows."""
    g = torch.Generator().manual_seed(seed)
    q, k, v = torch.randn(T, H, d, generator=g) * 0.1, torch.randn(T, G, d, generator=g), torch.randn(T, G, dv, generator=g)
    for n, i in enumerate(range(3, T, 4)):
        edge = max(window, 2)
        j = [0, 1, 31, 32, 63, 64, i, i - 1, i - edge + 1, i - edge, i - edge - 1, i - edge // 2][n % 12]
        if 0 <= j <= i:
            h = n % H
            u = k[j, h // (H // G)]
            q[i, h] = u / u.norm() ** 2 * 25.0
    return q, k, v


def _attend(q, k, v, scale, ctype, kernel, portions, softcap=0.0, window=0, slopes=None, gate=None, n_splits=1):
    """kernel: "row", "window" (values as wide as keys) or "talk" (any widths)."""
    from dllama_b200.ops import layers as L
    T, H, d = q.shape
    G, dv = k.shape[1], v.shape[2]
    n_pages = (T + PAGE - 1) // PAGE
    cache = (torch.randn(n_pages + 2, G, PAGE, d + dv, device="cuda") * 50).to(ctype)
    table = torch.tensor([[0] * n_pages, list(range(n_pages + 1, 1, -1))], dtype=torch.int32, device="cuda")
    freqs, out = torch.zeros(1, dtype=F64, device="cuda"), []
    opts = dict(sink=torch.zeros(H, device="cuda"), slope=slopes.float().cuda() if slopes is not None else None)
    for p0, n in portions:
        pos, slot = torch.arange(p0, p0 + n, dtype=torch.int32, device="cuda"), torch.ones(n, dtype=torch.int32, device="cuda")
        qq, kk, vv = (t[p0:p0 + n].reshape(n, -1).float().cuda().contiguous() for t in (q, k, v))
        gz = torch.cat([torch.full((n, 2), 99.0), gate[p0:p0 + n]], 1).cuda()[:, 2:] if gate is not None else None
        L.window_kv_write(kk, n, G, d, 0, freqs, 1.0, pos, slot, table, cache, q=qq, q_heads=H, v=vv, vdim=dv)
        o = torch.full((n, H * dv), float("nan"), device="cuda")
        if kernel == "row":
            L.window_attention(qq, o, n, H, G, d, 0, scale, softcap, window, pos, slot, table, cache, vdim=dv, gate=gz, **opts)
        else:
            rq = L.window_tc_rows(H, G) if kernel == "window" else L.talk_tc_rows(H, G, d, dv, 0, n)
            tiles = [list(range(i, min(i + rq, n))) for i in range(0, n, rq)]
            if kernel == "window":
                L.window_attention_tiles(qq, o, H, G, d, 0, scale, softcap, window, pos, slot, table, cache, tiles, n_splits, vdim=dv, gate=gz, **opts)
            else:
                L.talk_attention_tiles(qq, o, H, G, d, dv, scale, window, pos, slot, table, cache, tiles, rq, n_splits, softcap=softcap, gate=gz, **opts)
        out.append(o.cpu())
    return torch.cat(out).double().reshape(T, H, dv)


VARIANTS = [dict(), dict(softcap=15.0), dict(window=40, slope=True), dict(window=33, softcap=9.0, slope=True), dict(slope=True), dict(window=1)]


@pytest.mark.parametrize("kernel,ctype,H,G,d,dv", [("row", torch.float32, 6, 3, 20, 12), ("row", torch.bfloat16, 4, 1, 32, 32), ("window", torch.bfloat16, 6, 3, 32, 32),
                                                  ("window", torch.bfloat16, 5, 5, 64, 64), ("window", torch.bfloat16, 12, 2, 128, 128), ("talk", torch.bfloat16, 4, 2, 24, 40),
                                                  ("talk", torch.bfloat16, 6, 2, 64, 96), ("talk", torch.bfloat16, 8, 8, 40, 128)])
@pytest.mark.parametrize("variant", range(len(VARIANTS)))
def test_attention(kernel, ctype, H, G, d, dv, variant):
    v_ = VARIANTS[variant]
    T, window, softcap = 150, v_.get("window", 0), v_.get("softcap", 0.0)
    q, k, v = _case(T, H, G, d, dv, 17 + variant, window)
    slopes = O.distance_slopes(H) if v_.get("slope") else None
    gate = torch.randn(T, H, generator=torch.Generator().manual_seed(19)) * 2
    qb, kb, vb = (t.to(ctype).double() for t in (q, k, v))
    if kernel == "row":
        qb = q.double()
    want = O.head_gated(O.sink_attention_rows(qb, kb, vb, 0.7, softcap, window, slopes), gate.double()).view(T, H, dv)
    tol = 2e-4 if ctype == torch.float32 else 2e-3 if kernel == "row" else 0.04
    for portions, n_splits in (([(0, T)], 1), ([(0, 37), (37, 1), (38, 2), (40, 60), (100, 50)], 3), ([(0, 120)] + [(i, 1) for i in range(120, T)], 2)):
        got = _attend(q, k, v, 0.7, ctype, kernel, portions, softcap, window, slopes, gate, n_splits)
        err = (got - want).abs().amax((1, 2))
        assert float(err.max()) < tol, (portions[:3], int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("kernel,H,G,d,dv", [("window", 4, 2, 32, 32), ("talk", 4, 2, 24, 40), ("talk", 8, 4, 64, 96)])
def test_attention_of_many_decoded_rows(kernel, H, G, d, dv):
    """One-row tiles by the hundred, the batched form of decoding."""
    from dllama_b200.ops import layers as L
    T, window = 300, 50
    q, k, v = _case(T, H, G, d, dv, 23, window)
    slopes = O.distance_slopes(H)
    gate = torch.randn(T, H, generator=torch.Generator().manual_seed(29))
    want = O.head_gated(O.sink_attention_rows(*(t.bfloat16().double() for t in (q, k, v)), 0.7, 12.0, window, slopes), gate.double()).view(T, H, dv)
    n_pages = (T + PAGE - 1) // PAGE
    cache = torch.zeros(n_pages, G, PAGE, d + dv, dtype=torch.bfloat16, device="cuda")
    table = torch.arange(n_pages - 1, -1, -1, dtype=torch.int32, device="cuda").view(1, -1)
    pos, slot = torch.arange(T, dtype=torch.int32, device="cuda"), torch.zeros(T, dtype=torch.int32, device="cuda")
    qq, kk, vv = (t.reshape(T, -1).cuda().contiguous() for t in (q, k, v))
    L.window_kv_write(kk, T, G, d, 0, torch.zeros(1, dtype=F64, device="cuda"), 1.0, pos, slot, table, cache, q=qq, q_heads=H, v=vv, vdim=dv)
    opts = dict(sink=torch.zeros(H, device="cuda"), slope=slopes.float().cuda(), gate=gate.cuda())
    for n_splits in (1, 2):
        o = torch.zeros(T, H * dv, device="cuda")
        if kernel == "window":
            L.window_attention_tiles(qq, o, H, G, d, 0, 0.7, 12.0, window, pos, slot, table, cache, [[i] for i in range(T)], n_splits, vdim=dv, **opts)
        else:
            rq = L.talk_tc_rows(H, G, d, dv, 0, 1)
            L.talk_attention_tiles(qq, o, H, G, d, dv, 0.7, window, pos, slot, table, cache, [[i] for i in range(T)], rq, n_splits, softcap=12.0, **opts)
        assert float((o.cpu().double().view(T, H, dv) - want).abs().max()) < 0.04


@pytest.mark.parametrize("H,G,d,dv,rot,scaling", [(4, 2, 32, 16, 32, dict(factor=4.0, low=1.0, high=4.0, original=512)), (6, 3, 24, 40, 8, None),
                                                 (3, 3, 10, 7, 0, None), (8, 1, 64, 64, 16, dict(factor=8.0, low=1.0, high=8.0, original=4096))])
def test_cache_writer_norms_every_head_before_the_rotary(H, G, d, dv, rot, scaling):
    from dllama_b200.models.layered import interpolated_rotary
    from dllama_b200.ops import layers as L
    T, eps, base, p0 = 11, 1e-2, 700.0, 1000
    g = torch.Generator().manual_seed(31)
    q, k, v = (torch.randn(T, n, generator=g) for n in (H * d, G * d, G * dv))
    q[0] *= 0.01                                              # eps shows
    q[:, :d] *= 5.0                                           # one head dominates: one norm over all heads would come out otherwise
    wq, wk = torch.randn(d, generator=g), torch.randn(d, generator=g)
    pos = torch.arange(p0, p0 + T)
    fr = O.scaled_frequencies(base, rot, scaling)
    want_q = O.rotate_half_pairs(wq.double() * O.unit(q.double().view(T, H, d), eps), pos, fr)
    want_k = O.rotate_half_pairs(wk.double() * O.unit(k.double().view(T, G, d), eps), pos, fr)
    freqs, mag = interpolated_rotary(base, rot, scaling)
    assert mag == 1.0 and torch.allclose(freqs, fr, rtol=1e-12)
    n_pages = (p0 + T) // PAGE + 1
    cache = torch.zeros(2, G, PAGE, d + dv, device="cuda")
    table = torch.zeros(1, n_pages, dtype=torch.int32, device="cuda")
    table[0, (p0 // PAGE) + 1:] = 1
    qq = q.cuda()
    L.window_kv_write(k.cuda(), T, G, d, rot, freqs.cuda() if rot else torch.zeros(1, dtype=F64, device="cuda"), mag, pos.int().cuda(),
                      torch.zeros(T, dtype=torch.int32, device="cuda"), table, cache, q=qq, q_heads=H, v=v.cuda(), vdim=dv, eps=eps, rope_half=True,
                      q_norm=wq.cuda(), k_norm=wk.cuda(), head_norm=True)
    assert torch.allclose(qq.cpu().double().view(T, H, d), want_q, atol=2e-5, rtol=2e-5)
    for t in range(T):
        line = cache[int(table[0, (p0 + t) // PAGE]), :, (p0 + t) % PAGE].cpu().double()
        assert torch.allclose(line[:, :d], want_k[t], atol=2e-5, rtol=2e-5) and torch.allclose(line[:, d:], v[t].double().view(G, dv))


# ---------------------------------------------------------------------------------------------------------------------
# residual step with layer norms, products with bias
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dim", [30, 88, 192, 1500, 2048, 5000, 9000])
def test_residual_step_with_layer_norms_and_scaled_terms(dim):
    """A row whose mean is far from zero (the variance is that of the deviations), a row that is nearly constant (eps shows)."""
    from dllama_b200.ops import layers as L
    M, eps = 5, 1e-3
    g = torch.Generator().manual_seed(37)
    x, a, b, c = (torch.randn(M, dim, generator=g) for _ in range(4))
    x[1] += 300.0
    x[2], a[2], b[2], c[2] = 2.0 + x[2] * 0.02, 0.0, 0.0, 0.0
    w1, b1, w2, b2 = (torch.randn(dim, generator=g) for _ in range(4))
    want = x.double() + 0.7 * a.double() - 1.3 * b.double() + c.double()
    xo, h1, h2 = (torch.zeros(M, dim, device="cuda") for _ in range(3))
    cu = lambda t: t.cuda()
    L.residual_step(M, dim, eps, x_in=cu(x), adds=[cu(a), cu(b), cu(c)], scales=(0.7, -1.3), x=xo, layer_norm=True,
                    outs=[((cu(w1), cu(b1)), h1), ((cu(w2), cu(b2)), h2)])
    assert torch.allclose(xo.cpu().double(), want, atol=1e-4, rtol=1e-6)
    ref = xo.cpu().double()
    for h, w, bb in ((h1, w1, b1), (h2, w2, b2)):
        assert torch.allclose(h.cpu().double(), O.layer_norm(ref, w.double(), bb.double(), eps), atol=5e-4, rtol=1e-4)
    rows = torch.tensor([4, 1], dtype=torch.int32, device="cuda")
    ncap = 8
    xh = torch.full((L.xh_bytes(dim, ncap),), 0x7f, dtype=torch.uint8, device="cuda")
    L.residual_step(2, dim, eps, x_in=cu(x), adds=[cu(a), cu(b), cu(c)], scales=(0.7, -1.3), rows=rows, layer_norm=True, outs=[((cu(w1), cu(b1)), (xh, ncap))])
    img = _image_rows(xh, ncap, 2, dim)
    assert torch.allclose(img[:, :dim], h1[[4, 1]].bfloat16().float(), atol=1e-2, rtol=1e-2) and bool((img[:, dim:] == 0).all())


@pytest.mark.parametrize("N,K", [(7, 20), (130, 88), (300, 256)])
@pytest.mark.parametrize("M", [1, 3, 9, 40, 150])
def test_products_with_bias_and_scale(N, K, M):
    from dllama_b200.ops import layers as L
    g = torch.Generator().manual_seed(41)
    w, x, bias = torch.randn(N, K, generator=g).bfloat16(), torch.randn(M, K, generator=g).bfloat16().float(), torch.randn(N, generator=g) * 5
    want = x.double() @ w.double().T
    ys = []
    y = torch.zeros(M, N, device="cuda")
    L.dense(w.cuda(), x.cuda(), y, M, True, bias=bias.cuda())
    ys.append(y)
    y = torch.zeros(M, N, device="cuda")
    L.dense(w.cuda(), x.cuda(), y, M, True, bias=bias.cuda(), epi=L.DENSE_SCALE, param=-2.5)
    ys.append(y)
    ncap = (M + 7) // 8 * 8
    xh = torch.zeros(L.xh_bytes(K, ncap), dtype=torch.uint8, device="cuda")
    L.xh_from_rows(x.cuda(), M, K, ncap, xh)
    for kw in (dict(), dict(epi=L.DENSE_SCALE, param=-2.5)):
        y = torch.zeros(M, N, device="cuda")
        L.dense_tc(L.make_wh(w.cuda()), N, K, xh, ncap, y, M, bias=bias.cuda(), **kw)
        ys.append(y)
    for i, y in enumerate(ys):
        ref = (want + bias.double()) * (-2.5 if i & 1 else 1.0)
        assert torch.allclose(y.cpu().double(), ref, atol=1e-3, rtol=1e-4), i
