"""Kernels behind Tirudra models, one mechanism at a time, each against the plain formulas in 64 bits.  Inputs are made so that a fault shows: in the
attention tests one key at an edge carries nearly all of a query's weight, in the recurrence tests slow decays keep the first tokens alive."""
import math

import pytest
import torch

import tirudra_oracle as O

pytestmark = pytest.mark.gpu
F64 = torch.float64


@pytest.fixture(scope="module", autouse=True)
def no_timeouts():
    from ollama_b200.ops import cuda as K
    K.need("stack")
    yield
    assert K.gemm_status() == 0


def rnd(*s, seed=0, scale=1.0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed)) * scale


def close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    err = (got - want).abs().max() / want.abs().max().clamp(min=1e-9)
    assert torch.isfinite(got).all() and err < tol, float(err)


def i32(*v):
    return torch.tensor(v, dtype=torch.int32).cuda()


def up(n, m=8):
    return -(-n // m) * m


# -- attention ----------------------------------------------------------------------------------------------------
class Attn:
    """One sequence in slot 1 of a paged cache with scattered pages; rows of [q | k | v] (or [q | k] where the values are the keys) and gates behind them."""

    def __init__(self, H, G, dim, vdim, size, keep, n, kind, gate="element", keys=False, rot=None, norm=True, seed=0):
        self.H, self.G, self.dim, self.vdim, self.size, self.keep, self.n, self.gate, self.keys, self.norm = H, G, dim, vdim, size, keep, n, gate, keys, norm
        self.f32, self.eps, self.scale = kind == "f32", 1e-3, 0.7 / math.sqrt(dim)
        self.nq, self.nk = H * dim, G * dim
        nv = 0 if keys else G * vdim
        self.n8 = up(self.nq + self.nk + nv)
        self.rows_in = rnd(n, self.n8 + up(H * vdim), seed=seed)
        self.qn, self.kn = 2.0 + 0.5 * rnd(dim, seed=seed + 1), 1.0 + 0.3 * rnd(dim, seed=seed + 2)
        self.freqs, self.mag = (O.rotation(rot) if rot else (torch.zeros(0, dtype=F64), 1.0))
        self.v_off = self.nq if keys else self.nq + self.nk
        self.hd = 64 if max(dim, vdim) <= 64 else 128
        if kind != "tc":
            self.hd = 0
        pages = -(-n // 64)
        self.table = torch.zeros(2, pages + 1, dtype=torch.int32).cuda()
        self.table[1, :pages] = torch.randperm(pages + 3, generator=torch.Generator().manual_seed(seed))[:pages].to(torch.int32).cuda()
        dk, dv = (self.hd, self.hd) if self.hd else (up(dim), up(vdim))
        dt = torch.float32 if self.f32 else torch.float16
        self.kc, self.vc = torch.full((pages + 3, G, 64, dk), 7.0, dtype=dt, device="cuda"), torch.full((pages + 3, G, 64, dv), -9.0, dtype=dt, device="cuda")

    def aim(self, pairs, strength=6.0):
        """The query at position i finds the key at position j and nothing else, for the (i, j) of ``pairs`` (without norm and rotation)."""
        for i, j in pairs:
            k = self.rows_in[j, self.nq:self.nq + self.nk].view(self.G, self.dim)
            k = k / k.norm(dim=-1, keepdim=True)
            self.rows_in[j, self.nq:self.nq + self.nk] = (k * strength).reshape(-1)
            self.rows_in[i, :self.nq] = (k.repeat_interleave(self.H // self.G, 0) * strength * math.sqrt(self.dim)).reshape(-1)

    def values(self):
        return self.rows_in[:, self.v_off:self.v_off + self.G * self.vdim].double().view(self.n, self.G, self.vdim)

    def plain(self):
        """Without the gate, [n, H, vdim]."""
        x = self.rows_in.double()
        q, k = x[:, :self.nq].view(self.n, self.H, self.dim), x[:, self.nq:self.nq + self.nk].view(self.n, self.G, self.dim)
        if self.norm:
            q, k = O.norm_plain(q, self.qn.double(), self.eps), O.norm_plain(k, self.kn.double(), self.eps)
        if len(self.freqs):
            q, k = (O.rotate_half(t, torch.arange(self.n), self.freqs, self.mag) for t in (q, k))
        return O.attend(q, k, self.values(), self.scale, O.window_visible(self.n, self.size or None, self.keep))

    def expected(self):
        g = torch.sigmoid(self.rows_in[:, self.n8:].double())
        g = g[:, :self.H * self.vdim].view(self.n, self.H, self.vdim) if self.gate == "element" else g[:, :self.H, None] if self.gate else 1.0
        return (self.plain() * g).reshape(self.n, -1)

    def _args(self, x):
        from ollama_b200.ops import rows as R
        norm = dict(q_norm=self.qn.cuda(), k_norm=self.kn.cuda()) if self.norm else dict(q_norm=None, k_norm=None)
        self.held = list(norm.values())
        self.f = (self.freqs if len(self.freqs) else torch.zeros(1, dtype=F64)).cuda()
        prep = dict(heads=self.H, dim=self.dim, vdim=self.vdim, eps=self.eps, freqs=self.f, n_rot=2 * len(self.freqs), head_norm=True, v_off=self.v_off, mscale=self.mag, **norm)
        mask = dict(scale=self.scale, window=self.size, keep=self.keep, gate=R.head_gate(x[:, self.n8:], self.gate) if self.gate else R.NO_GATE)
        return R, prep, mask

    def rows(self, lo, hi):
        m, x = hi - lo, self.rows_in[lo:hi].cuda()
        R, prep, mask = self._args(x)
        pos, slots = torch.arange(lo, hi, dtype=torch.int32).cuda(), torch.ones(m, dtype=torch.int32).cuda()
        q = torch.empty(m, self.H, self.hd or self.dim, device="cuda")
        R.paged_append(x, kv_heads=self.G, positions=pos, slots=slots, table=self.table, q_out=q, k_cache=self.kc, v_cache=self.vc, **prep)
        out = torch.full((m, up(self.H * self.vdim + 1)), 5.0, device="cuda", dtype=torch.float32 if self.f32 else torch.bfloat16)
        if self.hd:
            tiles = torch.tensor([(r, min(128, m - r), 1, lo + r) for r in range(0, m, 128)], dtype=torch.int32).cuda()
            R.attn_prefill_paged(q, self.kc, self.vc, tiles, self.table, out, vdim=self.vdim, **mask)
        else:
            R.paged_attn(q, self.kc, self.vc, pos, slots, self.table, out, dim=self.dim, vdim=self.vdim, **mask)
        assert (out[:, self.H * self.vdim:] == 5).all()
        return out[:, :self.H * self.vdim]

    def decode(self, p, splits):
        x = self.rows_in[p:p + 1].cuda()
        R, prep, mask = self._args(x)
        acc, ml = torch.empty(self.H * splits * self.hd, device="cuda"), torch.empty(self.H * splits * 2, device="cuda")
        out = torch.full((1, self.H * self.vdim + 3), 5.0, device="cuda")
        assert R.attn_decode_paged(x, self.kc, self.vc, i32(p), i32(1), self.table, out, 1, softcap=0.0, chunk=0, n_splits=splits, n_ctx=max(self.n, 64), part_acc=acc, part_ml=ml,
                                   **prep, **mask)
        assert (out[:, self.H * self.vdim:] == 5).all()
        return out[:, :self.H * self.vdim]


YARN = {"base": 600.0, "dims": 8, "scaling": {"factor": 3.0, "original": 90, "fast": 9.0, "slow": 0.7}}
SHAPES = [  # H, G, dim, vdim, window, kept, gate, keys as values
    (3, 1, 40, 24, 20, 3, "element", False), (2, 2, 12, 32, 33, 0, "element", False), (4, 2, 64, 64, 128, 70, "element", False), (8, 2, 128, 128, 100, 5, "head", False),
    (6, 3, 96, 96, 0, 0, "head", True), (2, 1, 8, 1, 1, 1, "element", False), (16, 1, 100, 128, 64, 64, "", False), (2, 1, 128, 64, 1000, 9, "element", False),
    (5, 5, 30, 30, 0, 0, "head", True), (4, 1, 16, 16, 65, 200, "element", False),
]


@pytest.mark.parametrize("kind", ["tc", "f16", "f32"])
@pytest.mark.parametrize("shape", SHAPES)
def test_attention_of_prompt_portions(shape, kind):
    H, G, dim, vdim, size, keep, gate, keys = shape
    n = 290
    a = Attn(H, G, dim, vdim, size, keep, n, kind, gate, keys, YARN, seed=dim)
    want, tol = a.expected(), 2e-5 if kind == "f32" else 1e-2
    for cuts in ([n], [2, 62, 1, 65, 3, 128, 7, n]):
        a.kc.fill_(7.0), a.vc.fill_(-9.0)
        at, got = 0, []
        for c in cuts:
            if at < n:
                got.append(a.rows(at, min(at + c, n)))
                at += c
        close(torch.cat(got), want, tol)


@pytest.mark.parametrize("splits", [1, 4])
@pytest.mark.parametrize("shape", SHAPES)
def test_decode_attention(shape, splits):
    H, G, dim, vdim, size, keep, gate, keys = shape
    n = 270
    a = Attn(H, G, dim, vdim, size, keep, n, "tc", gate, keys, YARN, seed=dim + 1)
    want, at = a.expected(), 0
    for p in [0, 1, 19, 20, 21, 63, 64, 65, 99, 100, 127, 128, 129, 191, 192, 255, 256, 269]:
        if p > at:
            a.rows(at, p)
        close(a.decode(p, splits)[0], want[p], 4e-3)
        at = p + 1


@pytest.mark.parametrize("kind", ["tc", "f16", "f32"])
@pytest.mark.parametrize("size,keep", [(0, 0), (64, 0), (96, 4), (128, 64), (130, 65), (1, 130), (200, 128)])
def test_a_single_key_stands_out_at_the_edges(size, keep, kind):
    """Queries aimed at one key: where it is seen it takes nearly all the weight, one place beyond the edge none of it."""
    n = 420
    queries = iter([131, 191, 192, 257, 300, 319, 320, 383, 384, 399, 400, 410, 415, 419])
    pairs, used = [], set()
    for d in (size - 1, size, 1, 0) if size else (130, 63, 64, 1):            # just inside and outside the window
        for _ in range(2):
            i = next(queries)
            if i - d >= 0 and i - d not in used:
                pairs.append((i, i - d))
                used.add(i - d)
    for j in (keep - 1, keep, 0):                                             # the last kept key, the next one, the first
        if j >= 0 and j not in used:
            pairs.append((next(queries), j))
            used.add(j)
    a = Attn(4, 2, 48, 40, size, keep, n, kind, "", norm=False, seed=3)
    a.aim(pairs)
    want, v = a.expected(), a.values()
    for i, j in pairs:
        hit = (want[i].view(4, 40) - v[j].repeat_interleave(2, 0)).abs().max()
        assert (hit < 0.05) == (not size or i - j < size or j < keep), (i, j)
    close(a.rows(0, n), want, 2e-5 if kind == "f32" else 8e-3)
    if kind == "tc":
        for i, _ in pairs:
            for splits in (1, 3):
                close(a.decode(i, splits)[0], want[i], 5e-3)


# -- short convolutions ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("bias", [False, True])
def test_convolution_in_portions_and_steps(taps, bias):
    """Portions of two sequences beside one another, then single tokens in both forms; slots held something else before."""
    from ollama_b200.ops import rows as R
    T, C, act = 70, 24, bias                        # with a bias also the activation
    x, w, b = rnd(2, T, C, seed=taps), rnd(C, taps, seed=1), rnd(C, seed=2) if bias else torch.zeros(C)
    want = torch.stack([O.causal_conv(s.double(), w.double(), b.double()) for s in x])
    want = O.silu(want) if act else want
    wt, bc = w.t().contiguous().cuda(), b.cuda() if bias else None
    state = torch.full((3, max(taps - 1, 1), C), 50.0, device="cuda")

    def portion(parts):
        """parts: (sequence, first, last) -> convolved rows"""
        rows = torch.cat([x[s, lo:hi] for s, lo, hi in parts]).cuda()
        pos = torch.cat([torch.arange(lo, hi) for _, lo, hi in parts]).to(torch.int32).cuda()
        slots = torch.cat([torch.full((hi - lo,), 2 - s) for s, lo, hi in parts]).to(torch.int32).cuda()
        offs = torch.cat([torch.arange(hi - lo) for _, lo, hi in parts]).to(torch.int32).cuda()
        segs, at = [], 0
        for s, lo, hi in parts:
            segs.append((at, hi - lo, 2 - s, lo))
            at += hi - lo
        u = torch.empty_like(rows)
        R.ssm_conv(rows, C, wt, bc, state, slots, pos, offs, u, silu=act)
        R.conv_keep(rows, C, taps, state, torch.tensor(segs, dtype=torch.int32).cuda())
        return u

    got = [[], []]
    for cut in ([(0, 0, 2), (1, 0, 1)], [(1, 1, 30)], [(0, 2, 3), (1, 30, 32)], [(0, 3, 40)]):
        u, at = portion(cut), 0
        for s, lo, hi in cut:
            got[s].append(u[at:at + hi - lo])
            at += hi - lo
    for t in range(10):                             # both sequences decode together
        rows = torch.stack([x[0, 40 + t], x[1, 32 + t]]).cuda()
        slots, pos = i32(2, 1), i32(40 + t, 32 + t)
        u = torch.empty_like(rows)
        if t % 2:
            R.ssm_conv(rows, C, wt, bc, state, slots, pos, torch.zeros_like(pos), u, silu=act, shift=True)
        else:                                       # in the epilogue of a product, here with an identity matrix
            out = torch.zeros_like(rows)
            R.gemv([R.seg(torch.eye(C, device="cuda"), C, out)], C, rows, 2, True, conv=(wt, bc, state), conv_out=u, conv_silu=act, conv_shift=True, slots=slots, positions=pos)
            assert torch.equal(out, rows)
        got[0].append(u[:1]), got[1].append(u[1:])
    fresh = torch.empty(1, C, device="cuda")        # a new sequence in a slot that was used
    R.ssm_conv(x[1, :1].cuda(), C, wt, bc, state, i32(2), i32(0), i32(0), fresh, silu=act, shift=True)
    close(fresh, want[1, :1], 1e-5)
    close(torch.cat(got[0]), want[0, :50], 1e-5)
    close(torch.cat(got[1]), want[1, :42], 1e-5)


# -- recurrence -----------------------------------------------------------------------------------------------------
class Ssd:
    def __init__(self, H, P, N, G, T, dtype, seed=0):
        self.H, self.P, self.N, self.G, self.T, self.dtype = H, P, N, G, T, dtype
        self.vp, self.np = up(P), up(N, 16)
        self.x, self.B, self.C, self.z = (rnd(T, *s, seed=seed + i).to(dtype).float() for i, s in enumerate(((H, P), (G, N), (G, N), (H, P))))
        self.dt, self.bias, self.d = rnd(T, H, seed=seed + 5), -3.0 + 1.5 * rnd(H, seed=seed + 6), rnd(H, seed=seed + 7)
        self.a = -(0.02 + 4.0 * torch.rand(H, generator=torch.Generator().manual_seed(seed)) ** 3)
        self.state = torch.full((3, H, self.vp, self.np), 40.0, device="cuda")
        self.state[..., P:, :] = 0
        self.state[..., N:] = 0

    def rows(self, lo, hi, f32=False):
        """Padded rows x | B | C, z, step sizes, on the device."""
        n = hi - lo
        x, z = (torch.zeros(n, self.H, self.vp) for _ in range(2))
        x[..., :self.P], z[..., :self.P] = self.x[lo:hi], self.z[lo:hi]
        bc = torch.zeros(2, n, self.G, self.np)
        bc[0, ..., :self.N], bc[1, ..., :self.N] = self.B[lo:hi], self.C[lo:hi]
        dt = torch.float32 if f32 else self.dtype
        u = torch.cat([x.view(n, -1), bc[0].view(n, -1), bc[1].view(n, -1)], 1).to(dt).cuda()
        return u, z.view(n, -1).to(dt).cuda(), self.dt[lo:hi].contiguous().cuda()

    def expected(self):
        """Gated results [T, H, P] and the state behind the last row [H, P, N]."""
        dt = O.softplus(self.dt.double() + self.bias.double())
        y = O.ssd_scan(self.x.double(), dt, self.a.double(), self.B.double(), self.C.double(), self.d.double())
        S = torch.zeros(self.H, self.P, self.N, dtype=F64)
        for t in range(self.T):
            b = self.B[t].double().repeat_interleave(self.H // self.G, 0)
            S = torch.exp(self.a.double() * dt[t])[:, None, None] * S + dt[t][:, None, None] * self.x[t].double()[:, :, None] * b[:, None]
        return y * O.silu(self.z.double()), S

    def _call(self, fn, rows, groups_args, *more):
        off = self.H * self.vp
        u, z, dt = rows
        out = torch.zeros(u.shape[0], off, device="cuda", dtype=u.dtype)
        fn(u, off, off + self.G * self.np, z, dt, self.bias.cuda(), self.a.cuda(), self.d.cuda(), self.G, self.state, *more, out)
        return out.view(-1, self.H, self.vp)

    def portion(self, slot, lo, hi):
        """As one portion behind an unrelated sequence of five rows in another slot."""
        from ollama_b200.ops import ssd as D
        rows = [torch.cat([t, s]) for t, s in zip(self.rows(3, 8), self.rows(lo, hi))]
        segs = torch.tensor([(0, 5, 2, 0), (5, hi - lo, slot, lo)], dtype=torch.int32).cuda()
        out = self._call(D.ssd_scan, rows, None, segs)[5:]
        assert (out[..., self.P:] == 0).all()
        return out[..., :self.P]

    def step(self, slots, ts, f32):
        from ollama_b200.ops import ssd as D
        rows = [torch.cat(t) for t in zip(*(self.rows(t, t + 1, f32) for t in ts))]
        return self._call(D.ssd_step, rows, None, i32(*slots), i32(*ts))[..., :self.P]


SSD = [(1, 1, 1, 1), (4, 16, 16, 2), (3, 20, 9, 1), (6, 12, 20, 3), (8, 64, 128, 2), (5, 72, 40, 5), (2, 130, 100, 1), (2, 40, 200, 2), (100, 64, 64, 4), (96, 40, 128, 1), (96, 64, 128, 8), (96, 48, 20, 3)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,P,N,G", SSD)
def test_state_space_portions_and_steps(H, P, N, G, dtype):
    T = 210 if H < 50 else 90
    s = Ssd(H, P, N, G, T, dtype, seed=P)
    want, state = s.expected()
    tol = 1e-5 if dtype == torch.float32 else 6e-3                  # 16-bit results; what they come from is kept to 16 bits and more, as the states show
    for slot, cuts in ((0, [T]), (1, [2, 2, 33, 1, 64, 31, 63, T])):
        at, got = 0, []
        for c in cuts:
            if at < T:
                got.append(s.portion(slot, at, min(at + c, T)))
                at += c
        close(torch.cat(got), want, tol)
        close(s.state[slot, :, :P, :N], state, 1e-5 if dtype == torch.float32 else 3e-5)
        assert (s.state[slot, :, P:] == 0).all() and (s.state[slot, ..., N:] == 0).all()
    for f32 in (True, False) if dtype == torch.bfloat16 else (True,):
        s.portion(0, 0, 60)                                         # a prompt that goes on token by token, beside a sequence that is decoded from its first token
        got = [s.step((0, 1), (60 + t, t), f32) for t in range(25)]
        close(torch.stack([g[0] for g in got]), want[60:85], tol)
        close(torch.stack([g[1] for g in got]), want[:25], tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_slow_state_is_kept_to_full_precision(dtype):
    """Decays of 1 - 1e-5 over a thousand rows, nothing added after the first: an error of the decay would add up."""
    s = Ssd(4, 16, 32, 1, 1000, dtype, seed=4)
    s.a, s.bias, s.dt = torch.full((4,), -1e-3), torch.full((4,), -4.6), torch.zeros(1000, 4)
    s.B[1:] = 0
    want, state = s.expected()
    assert 0.98 < (state.norm() / (O.softplus(torch.tensor(-4.6, dtype=F64)) * (s.x[0, :, :, None] * s.B[0, :, None]).double().norm())) < 0.999
    s.portion(0, 0, 1000)
    close(s.state[0, :, :16], state, 1e-5 if dtype == torch.float32 else 4e-5)
    for t in range(30):
        s.step((1,), (t,), True)
    close(s.state[1, :, :16], Ssd.expected(type("", (), {**s.__dict__, "T": 30}))[1], 2e-6)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 5e-3)])
@pytest.mark.parametrize("H,P,G", [(1, 1, 1), (3, 20, 4), (6, 12, 2), (64, 64, 8), (2, 9, 6), (4, 8, 1)])
def test_norm_in_parts(H, P, G, dtype, tol):
    from ollama_b200.ops import ssd as D
    vp, rows = up(P), 3
    x, w = torch.zeros(rows, H, vp), torch.zeros(H, vp)
    x[..., :P], w[:, :P] = rnd(rows, H, P, seed=1, scale=2), rnd(H, P, seed=2)
    got = x.view(rows, -1).to(dtype).cuda()
    D.group_norm(got, H, P, vp, G, w.view(-1).cuda(), 0.1)
    flat = x[..., :P].reshape(rows, -1).to(dtype).double()
    want = O.rms(flat.view(rows, G, -1), 0.1).reshape(rows, -1) * w[:, :P].reshape(-1).double()
    close(got.view(rows, H, vp)[..., :P].reshape(rows, -1), want, tol)
    assert (got.view(rows, H, vp)[..., P:] == 0).all()


# -- products and experts --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("m,n,nt,k", [(5, 64, 8, 2048), (70, 32, 72, 40), (200, 256, 16, 512), (300, 2048, 8, 264), (16, 4096, 40, 1024), (2048, 2816, 72, 256)])
def test_last_columns_of_a_product_as_rows_of_their_own(m, n, nt, k):
    from ollama_b200.ops import rows as R
    a, w, bias = rnd(m, k, seed=1).bfloat16().cuda(), (rnd(n + nt, k, seed=2) / math.sqrt(k)).bfloat16().cuda(), rnd(n + nt, seed=3).cuda()
    p = (a.double() @ w.double().t() + bias.double()).cpu()
    tail = torch.full((m, nt + 8), 9.0, device="cuda")
    out = torch.zeros(m, n, device="cuda", dtype=torch.bfloat16)
    R.gemm(a, w, out, bias=bias, tail=tail[:, :nt])
    close(out, p[:, :n], 6e-3)
    close(tail[:, :nt], p[:, n:], 1e-5)
    assert (tail[:, nt:] == 9).all()
    h = torch.zeros(m, n // 2, device="cuda", dtype=torch.bfloat16)
    R.gemm(a, w, h, bias=bias, act="glu:silu", tail=tail[:, :nt])
    close(h, O.silu(p[:, 0:n:2]) * p[:, 1:n:2], 8e-3)
    close(tail[:, :nt], p[:, n:], 1e-5)


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("E,same,top,ff,sff,width", [(1, 0, 1, 1, 0, 8), (6, 2, 3, 28, 20, 52), (3, 5, 8, 16, 9, 37), (300, 40, 16, 40, 130, 264), (5, 1, 2, 24, 0, 64)])
@pytest.mark.parametrize("rows", [1, 3, 4, 70])
def test_experts(f32, E, same, top, ff, sff, width, rows):
    """Both forms (few rows, sorted rows): corrected choices, plain weights, identity experts, the gated shared expert, the norm behind."""
    from ollama_b200.engine import blocks as B
    from ollama_b200.engine.stack import _Rows
    from ollama_b200.models.stack import DESIGNS, Expert, ExpertMLP
    dt, n = torch.float32 if f32 else torch.bfloat16, E + same

    def t(*s, seed, scale=1.0):
        return rnd(*s, seed=seed, scale=scale).to(dt)
    w = {"router": t(n, width, seed=1, scale=2 / math.sqrt(width)), "correction": rnd(n, seed=2, scale=0.3)}
    for e in range(E):
        for i, (name, s) in enumerate((("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))):
            w[f"e{e}.{name}"] = t(*s, seed=10 * e + i, scale=1.5 * s[1] ** -0.5)
    names = {"ffn_gate_inp.weight": w["router"], "exp_probs_b.bias": w["correction"]}
    if sff:
        w["shared.sg"] = t(1, width, seed=5, scale=width ** -0.5)
        names["ffn_gate_inp_shexp.weight"] = w["shared.sg"]
        for i, (name, s) in enumerate((("gate", (sff, width)), ("up", (sff, width)), ("down", (width, sff)))):
            w[f"shared.{name}"] = names[f"ffn_{name}_shexp.weight"] = t(*s, seed=9000 + i, scale=1.5 * s[1] ** -0.5)
    for name in ("gate", "up", "down"):
        names[f"ffn_{name}_exps.weight"] = torch.stack([w[f"e{e}.{name}"] for e in range(E)])
    src = B.WeightSource(lambda name: names[name].float().cuda(), "cuda", dt, width)

    def norm(seed):
        v = torch.zeros(src.wp).cuda()
        v[:width] = 1.0 + 0.2 * rnd(width, seed=seed).cuda()
        return B.Norm(v, None)
    pre, post = norm(3), norm(4)

    class Engine:
        class stack:
            eps, residual_mult, design = 1e-5, 1.0, DESIGNS["Tirudra"]
        wp, pdl, _n, gemv_rows, act_dtype = src.wp, True, 0, 4, dt
    Engine.f32, Engine.stack.width = f32, width

    class Meta:
        tokens = torch.zeros(rows, dtype=torch.int32).cuda()
    x = torch.zeros(rows, src.wp).cuda()
    x[:, :width] = rnd(rows, width, seed=6).cuda()
    ffn = B.ExpertFFN(src, "", ExpertMLP(E, top, Expert(ff), Expert(sff) if sff else None, identity=same, **DESIGNS["Tirudra"].experts), pre, f32, post)
    x64 = x[:, :width].double().cpu()
    h = O.norm_plain(x64, pre.g[:width].double().cpu(), 1e-5)
    if not f32 and rows > 4:
        h = h.to(torch.bfloat16).double()                        # what the products read there: no test of a close call
    cfg = {"router": {"experts": E, "identity": same, "top": top}, "shared": {} if sff else None}
    if sff:
        cfg["shared"] = {"ff": sff}
    idx, _ = O.route(h, w["router"].double(), w["correction"].double(), top)
    y = O.moe_ff(h, lambda name: w[name].double(), cfg)
    want = x64 + O.norm_plain(y, post.g[:width].double().cpu(), 1e-5)
    s = B.Step(Engine(), _Rows(rows, "cuda"), Meta(), x, None, rows <= 4)
    ffn.run(s)
    s.flush()
    close(s.x[:, :width], want, 2e-5 if f32 else 1.5e-2)
    assert (s.x[:, width:] == 0).all()
    if same and rows == 70:
        assert (idx >= E).any() and (idx < E).any()


@pytest.mark.parametrize("k", [1, 37, 52, 2048])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 5e-3)])
def test_norm_with_the_normed_result_added_before_it(k, dtype, tol):
    from ollama_b200.ops import rows as R
    kp, rows, eps = up(k), 5, 1e-5
    x, y = torch.zeros(rows, kp).cuda(), torch.zeros(rows, kp).cuda()
    x[:, :k], y[:, :k] = rnd(rows, k, seed=1).cuda(), rnd(rows, k, seed=2, scale=9).cuda()
    w, wy = (torch.cat([rnd(k, seed=s), torch.zeros(kp - k)]).cuda() for s in (3, 4))
    want = (x[:, :k].double() + O.norm_plain(y[:, :k].double(), wy[:k].double(), eps)).cpu()
    h = torch.full((rows, kp), 9.0, device="cuda", dtype=dtype)
    R.norm_rows(x, k, eps, w, h, y=y, wy=wy)
    close(x[:, :k], want, 1e-6)
    close(h[:, :k], O.norm_plain(want, w[:k].double().cpu(), eps), tol)
    assert (h[:, k:] == 0).all() and (x[:, k:] == 0).all()
