"""The kernels behind stack models, one mechanism at a time, against plain statements of the same operation.  Inputs are made so that a
fault shows: in the attention tests one key far away, at a page border or at a chunk's edge carries nearly all of a query's weight."""
import math

import pytest
import torch

import vazatar_oracle as O

pytestmark = pytest.mark.gpu
F64 = torch.float64


def rnd(*s, seed=0, scale=1.0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed)) * scale


def close(got, want, tol):
    got, want = got.double().cpu(), want.double()
    assert torch.isfinite(got).all()
    err = (got - want).abs().max() / want.abs().max().clamp(min=1e-6)
    assert err < tol, float(err)


def close_in(dtype):
    return 1e-5 if dtype == torch.float32 else 8e-3


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("k,ldo", [(7, 8), (52, 56), (136, 136), (4096, 4096)])
def test_norm_pair(dtype, k, ldo):
    from ollama_b200.ops import rows as R
    x, w1, w2 = rnd(5, ldo, seed=1, scale=3), rnd(k, seed=2), rnd(k, seed=3)
    o1, o2 = (torch.full((5, ldo), 9.0, device="cuda", dtype=dtype) for _ in range(2))
    R.norm_rows(x.cuda(), k, 0.5, w1.cuda(), o1, w2.cuda(), o2)
    for o, w in ((o1, w1), (o2, w2)):
        close(o[:, :k], O.norm_plain(x[:, :k].double(), w.double(), 0.5), close_in(dtype))
        assert (o[:, k:] == 0).all()
    R.norm_rows(x.cuda(), k, 0.5, w1.cuda(), o2)
    assert torch.equal(o1, o2)


def test_join_rows():
    from ollama_b200.ops import rows as R
    a, b, o = rnd(3, 16, seed=1), rnd(3, 24, seed=2), torch.full((3, 40), 9.0, device="cuda")
    R.join_rows(a.cuda(), 13, o, b.cuda(), 20, 16)
    assert torch.equal(o.cpu(), torch.cat([a[:, :13], torch.zeros(3, 3), b[:, :20], torch.zeros(3, 4)], 1))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m,n,k", [(1, 8, 8), (33, 56, 72), (130, 200, 24), (300, 264, 520), (16, 96, 4104), (200, 64, 8192)])
def test_gemm_windows_activation_and_accumulation(dtype, m, n, k):
    from ollama_b200.ops import rows as R
    a, w = rnd(m, k + 16, seed=1).to(dtype), rnd(n, k, seed=2).to(dtype)
    want = a[:, :k].double() @ w.double().t()
    out = torch.full((m, n + 16), 2.0, device="cuda")
    R.gemm(a.cuda()[:, :k], w.cuda(), out[:, 8:8 + n])
    close(out[:, 8:8 + n], want, 1e-5)
    assert (out[:, :8] == 2).all() and (out[:, 8 + n:] == 2).all()
    R.gemm(a.cuda()[:, :k], w.cuda(), out[:, 8:8 + n], accumulate=True)
    close(out[:, 8:8 + n], 2 * want, 1e-5)
    act = torch.zeros(m, n + 16, device="cuda", dtype=dtype)
    R.gemm(a.cuda()[:, :k], w.cuda(), act[:, 8:8 + n], act="relu2")
    close(act[:, 8:8 + n], O.relu2(want), close_in(dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nb", [1, 2, 3, 4])
@pytest.mark.parametrize("k,kn", [(8, 5), (136, 136), (2048, 2041)])
def test_fused_decode_products(dtype, nb, k, kn):
    """Two matrices on one normalised row with norms of their own, an activation and an accumulated result; rows; joined rows."""
    from ollama_b200.ops import rows as R
    f32 = dtype == torch.float32
    x = rnd(nb, k, seed=1, scale=2)
    x[:, kn:] = 0
    g1, g2 = rnd(k, seed=2), rnd(k, seed=3)
    w1, w2 = rnd(37, k, seed=4).to(dtype), rnd(50, k, seed=5).to(dtype)
    o1, o2 = torch.full((nb, 48), 3.0, device="cuda"), torch.full((nb, 52), 3.0, device="cuda")
    xc, w1c, w2c, g1c, g2c = x.cuda(), w1.cuda(), w2.cuda(), g1.cuda(), g2.cuda()
    R.gemv([R.seg(w1c, 37, o1, g1c, accumulate=True), R.seg(w2c, 50, o2, g2c, act="relu2")], k, xc, nb, f32, R.SRC_NORM, 1e-3, kn)
    h = O.rms(x[:, :kn].double(), 1e-3)
    close(o1[:, :37], 3 + (h * g1[:kn]) @ w1[:, :kn].double().t(), 2e-5)
    close(o2[:, :50], O.relu2((h * g2[:kn]) @ w2[:, :kn].double().t()), 2e-5)
    assert (o1[:, 37:] == 3).all() and (o2[:, 50:] == 3).all()
    R.gemv([R.seg(w1c, 37, o1)], k, xc, nb, f32)
    close(o1[:, :37], x.double() @ w1.double().t(), 2e-5)
    y, w3 = rnd(nb, k, seed=6), rnd(21, 2 * k, seed=7).to(dtype)
    o3 = torch.zeros(nb, 24, device="cuda")
    R.gemv([R.seg(w3.cuda(), 21, o3)], 2 * k, xc, nb, f32, R.SRC_JOINED, x2=y.cuda(), k1=k)
    close(o3[:, :21], torch.cat([x, y], 1).double() @ w3.double().t(), 2e-5)


class Attn:
    """One attention layer over a paged cache: raw projections of a sequence, pages in a scattered order, kernels chosen by the caller."""

    def __init__(self, H, G, dim, vdim, chunk, n, cap=0.0, norm=True, n_rot=None, kind="tc", seed=0):
        self.H, self.G, self.dim, self.vdim, self.chunk, self.n, self.cap, self.kind = H, G, dim, vdim, chunk, n, cap, kind
        self.scale, self.eps = 1.0 / math.sqrt(dim), 1e-4
        self.n_rot = dim // 2 * 2 if n_rot is None else n_rot
        self.f32 = kind == "f32"
        hd = 64 if max(dim, vdim) <= 64 else 128
        self.hd, self.dk, self.dv = (hd, hd, hd) if kind == "tc" else (0, dim, vdim)
        nq, nk, nv = H * dim, G * dim, G * vdim
        self.nq, self.nk = nq, nk
        self.qkv = rnd(n, nq + nk + nv, seed=seed)
        self.qn, self.kn = (1 + 0.2 * rnd(nq, seed=seed + 1), 1 + 0.2 * rnd(nk, seed=seed + 2)) if norm else (None, None)
        self.freqs = O.rotary_freqs(5000.0, self.n_rot) if self.n_rot else torch.zeros(1, dtype=F64)
        self.pages = (n + 63) // 64
        total = self.pages + 3
        g = torch.Generator().manual_seed(seed + 3)
        self.table = torch.zeros(3, self.pages + 2, dtype=torch.int32)
        self.slot = 1
        self.table[1, :self.pages] = torch.randperm(total, generator=g)[:self.pages].to(torch.int32)
        self.table = self.table.cuda()
        dt = torch.float32 if self.f32 else torch.float16
        self.kc = torch.full((total, G, 64, self.dk), 7.0, device="cuda", dtype=dt)        # garbage an earlier owner may have left
        self.vc = torch.full((total, G, 64, self.dv), -9.0, device="cuda", dtype=dt)

    def heads(self):
        """Normalised and rotated q, k and v of the whole sequence (fp64)."""
        x = self.qkv.double()
        q, k, v = x[:, :self.nq], x[:, self.nq:self.nq + self.nk], x[:, self.nq + self.nk:]
        if self.qn is not None:
            q, k = O.norm_plain(q, self.qn.double(), self.eps), O.norm_plain(k, self.kn.double(), self.eps)
        q, k, v = q.reshape(self.n, self.H, self.dim), k.reshape(self.n, self.G, self.dim), v.reshape(self.n, self.G, self.vdim)
        if self.n_rot:
            pos = torch.arange(self.n)
            q, k = O.rotate(q, pos, self.freqs), O.rotate(k, pos, self.freqs)
        return q, k, v

    def aim(self, pairs, strength=6.0):
        """Make the query at position i point at the key at position j (all heads), for the (i, j) of ``pairs``: only without norm and rotation."""
        for i, j in pairs:
            k = self.qkv[j, self.nq:self.nq + self.nk].view(self.G, self.dim)
            k = k / k.norm(dim=-1, keepdim=True)
            self.qkv[j, self.nq:self.nq + self.nk] = (k * strength).reshape(-1)
            self.qkv[i, :self.nq] = (k.repeat_interleave(self.H // self.G, 0) * strength * math.sqrt(self.dim)).reshape(-1)

    def expected(self):
        q, k, v = self.heads()
        return O.attend(q, k, v, self.scale, self.cap, self.chunk).reshape(self.n, -1)

    def rows(self, lo, hi):
        from ollama_b200.ops import rows as R
        m = hi - lo
        pos, slots = torch.arange(lo, hi, dtype=torch.int32).cuda(), torch.full((m,), self.slot, dtype=torch.int32).cuda()
        dq = self.hd or self.dim
        q = torch.empty(m, self.H, dq, device="cuda")
        c = lambda t: None if t is None else t.cuda()
        R.paged_append(self.qkv[lo:hi].cuda(), heads=self.H, kv_heads=self.G, dim=self.dim, vdim=self.vdim, q_norm=c(self.qn), k_norm=c(self.kn), eps=self.eps,
                       freqs=self.freqs.cuda(), n_rot=self.n_rot, positions=pos, slots=slots, table=self.table, q_out=q, k_cache=self.kc, v_cache=self.vc)
        ldo = self.H * self.vdim + 8 - self.H * self.vdim % 8
        out = torch.full((m, ldo), 5.0, device="cuda", dtype=torch.float32 if self.f32 else torch.bfloat16)
        kw = dict(scale=self.scale, softcap=self.cap, chunk=self.chunk)
        if self.kind == "tc":
            tiles = torch.tensor([(r, min(128, m - r), self.slot, lo + r) for r in range(0, m, 128)], dtype=torch.int32).cuda()
            R.attn_prefill_paged(q, self.kc, self.vc, tiles, self.table, out, vdim=self.vdim, **kw)
        else:
            R.paged_attn(q, self.kc, self.vc, pos, slots, self.table, out, dim=self.dim, vdim=self.vdim, **kw)
        assert (out[:, self.H * self.vdim:] == 5).all()
        return out[:, :self.H * self.vdim]

    def decode(self, p, splits):
        from ollama_b200.ops import rows as R
        pos, slots = torch.tensor([p], dtype=torch.int32).cuda(), torch.tensor([self.slot], dtype=torch.int32).cuda()
        acc, ml = torch.empty(self.H * splits * self.hd, device="cuda"), torch.empty(self.H * splits * 2, device="cuda")
        out = torch.full((1, self.H * self.vdim + 3), 5.0, device="cuda")
        c = lambda t: None if t is None else t.cuda()
        ok = R.attn_decode_paged(self.qkv[p:p + 1].cuda(), self.kc, self.vc, pos, slots, self.table, out, 1, heads=self.H, dim=self.dim, vdim=self.vdim,
                                 q_norm=c(self.qn), k_norm=c(self.kn), eps=self.eps, freqs=self.freqs.cuda(), n_rot=self.n_rot, scale=self.scale, softcap=self.cap,
                                 chunk=self.chunk, n_splits=splits, n_ctx=max(self.n, 64), part_acc=acc, part_ml=ml)
        assert ok and (out[:, self.H * self.vdim:] == 5).all()
        return out[:, :self.H * self.vdim]


SHAPES = [  # H, G, dim, vdim, chunk
    (3, 1, 40, 24, 20), (2, 2, 12, 32, 33), (4, 2, 64, 64, 128), (8, 2, 128, 128, 100), (6, 3, 96, 72, 0), (2, 1, 2, 1, 1), (16, 1, 100, 128, 64), (2, 1, 128, 64, 1000),
]


@pytest.mark.parametrize("kind", ["tc", "f16", "f32"])
@pytest.mark.parametrize("shape", SHAPES)
def test_paged_attention_of_prompt_portions(shape, kind):
    H, G, dim, vdim, chunk = shape
    n = 290
    a = Attn(H, G, dim, vdim, chunk, n, cap=7.0 if chunk % 3 else 0.0, n_rot=dim // 2 // 2 * 2, kind=kind, seed=dim)
    want, tol = a.expected(), 2e-5 if kind == "f32" else 8e-3
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
def test_paged_decode_attention(shape, splits):
    H, G, dim, vdim, chunk = shape
    n = 270
    a = Attn(H, G, dim, vdim, chunk, n, cap=7.0 if chunk % 3 else 0.0, n_rot=dim // 2 // 2 * 2, seed=dim + 1)
    want = a.expected()
    at = 0
    for p in [0, 1, 19, 20, 21, 63, 64, 65, 99, 100, 127, 128, 129, 191, 192, 255, 256, 269]:
        if p > at:
            a.rows(at, p)
        close(a.decode(p, splits)[0], want[p], 3e-3)
        at = p + 1


@pytest.mark.parametrize("kind", ["tc", "f16", "f32"])
@pytest.mark.parametrize("chunk", [0, 96, 128, 160])
def test_a_single_key_stands_out_near_edges_and_far_away(chunk, kind):
    """Queries aimed at one key: inside the chunk it takes nearly all the weight, a token beyond the edge none of it."""
    n = 400
    edges = [c for c in range(chunk, n, chunk)] if chunk else []
    pairs = [(390, 0), (130, 64), (131, 63)] if not chunk else []
    for e in edges[:2]:
        last = min(e + chunk, n) - 1
        pairs += [(e + 1, e), (e + 2, e - 1), (last, e), (last - 1, e - 1)][:4]
    seen = set()
    pairs = [(i, j) for i, j in pairs if not (i in seen or seen.add(i))]
    a = Attn(4, 2, 48, 40, chunk, n, norm=False, n_rot=0, kind=kind, seed=3)
    a.aim(pairs)
    want = a.expected()
    v = a.heads()[2]
    for i, j in pairs:      # the inputs do what they are for
        hit = (want[i].view(4, 40) - v[j].repeat_interleave(2, 0)).abs().max()
        assert (hit < 0.05) == O.chunk_visible(i, j, chunk)
    got = a.rows(0, n)
    tol = 2e-5 if kind == "f32" else 8e-3
    close(got, want, tol)
    if kind == "tc":
        for i, _ in pairs:
            close(a.decode(i, 3)[0], want[i], 5e-3)


def test_rotation_is_exact_far_along_a_sequence():
    from ollama_b200.ops import rows as R
    H, dim, pos = 2, 32, torch.tensor([0, 1, 4095, 131071], dtype=torch.int32)
    qkv = rnd(4, (H + 2) * dim, seed=9)
    f = O.rotary_freqs(10.0, 32)
    table = torch.zeros(1, 2048, dtype=torch.int32).cuda()
    q, kc, vc = torch.empty(4, H, dim, device="cuda"), torch.zeros(1, 1, 64, dim, device="cuda"), torch.zeros(1, 1, 64, dim, device="cuda")
    R.paged_append(qkv.cuda(), heads=H, kv_heads=1, dim=dim, vdim=dim, q_norm=None, k_norm=None, eps=0.0, freqs=f.cuda(), n_rot=32, positions=pos.cuda(),
                   slots=torch.zeros(4, dtype=torch.int32).cuda(), table=table, q_out=q, k_cache=kc, v_cache=vc)
    close(q, O.rotate(qkv[:, :H * dim].double().view(4, H, dim), pos, f), 2e-6)


class Ssm:
    def __init__(self, inner, n, r, taps, T, dtype, seed=0):
        self.inner, self.n, self.r, self.taps, self.T, self.dtype = inner, n, r, taps, T, dtype
        self.x, self.z = rnd(T, inner, seed=seed).to(dtype).float(), rnd(T, inner, seed=seed + 1).to(dtype).float()
        self.conv_w, self.conv_b = rnd(taps, inner, seed=seed + 2) / math.sqrt(taps), 0.3 * rnd(inner, seed=seed + 3)
        self.A = -(0.02 + 3.0 * torch.rand(inner, n, generator=torch.Generator().manual_seed(seed)) ** 3)
        self.B, self.C = rnd(T, n, seed=seed + 4), rnd(T, n, seed=seed + 5)
        self.low, self.w_dt = rnd(T, r, seed=seed + 6), (rnd(inner, r, seed=seed + 7) / math.sqrt(r)).to(dtype)
        self.bias, self.d = -2.0 + rnd(inner, seed=seed + 8), rnd(inner, seed=seed + 9)
        self.a2 = (self.A.double() * (1.0 if dtype == torch.float32 else 1.4426950408889634)).float().cuda()
        self.r8 = -(-r // 8) * 8
        self.p = torch.zeros(T, self.r8 + 2 * n + 8 - (2 * n) % 8)
        self.p[:, :r], self.p[:, self.r8:self.r8 + n], self.p[:, self.r8 + n:self.r8 + 2 * n] = self.low, self.B, self.C
        self.wp = torch.zeros(inner, self.r8, dtype=dtype)
        self.wp[:, :r] = self.w_dt
        self.xz = torch.cat([self.x, self.z], 1).to(dtype)
        self.state, self.conv_state = torch.full((3, inner, n), 40.0, device="cuda"), torch.full((3, max(taps - 1, 1), inner), -30.0, device="cuda")

    def expected(self):
        u = O.silu(O.causal_conv(self.x.double(), self.conv_w.double().t(), self.conv_b.double()))
        self.u = u
        us = u.to(self.dtype).double()
        dt = O.softplus(self.low.double() @ self.w_dt.double().t() + self.bias.double())
        y = O.selective_scan(us if self.dtype != torch.float32 else u, dt, self.A.double(), self.B.double(), self.C.double(), self.d.double())
        return y * O.silu(self.z.double())

    def portions(self, slot, lo, hi):
        """Convolution and scan of rows lo .. hi - 1 as one portion beside an unrelated sequence in another slot."""
        from ollama_b200.ops import rows as R
        n = hi - lo
        pos = torch.cat([torch.arange(lo, hi), torch.arange(5)]).to(torch.int32).cuda()
        slots = torch.tensor([slot] * n + [2] * 5, dtype=torch.int32).cuda()
        offs = torch.cat([torch.arange(n), torch.arange(5)]).to(torch.int32).cuda()
        segs = torch.tensor([(0, n, slot, lo), (n, 5, 2, 0)], dtype=torch.int32).cuda()
        both = lambda t: torch.cat([t[lo:hi], t[:5].flip(0)]).contiguous().cuda()
        xz, p = both(self.xz), both(self.p)
        u = torch.empty(n + 5, self.inner, device="cuda", dtype=self.dtype)
        R.ssm_conv(xz, self.inner, self.conv_w.cuda(), self.conv_b.cuda(), self.conv_state, slots, pos, offs, u)
        dt = (p[:, :self.r].double() @ self.w_dt.double().cuda().t()).float().contiguous()
        out = torch.empty(n + 5, self.inner, device="cuda", dtype=self.dtype)
        R.ssm_scan(xz, self.inner, u, dt, p, self.r8, self.bias.cuda(), self.a2, self.d.cuda(), self.taps, self.state, self.conv_state, segs, out)
        return u[:n], out[:n]

    def step(self, slot, t, given):
        from ollama_b200.ops import rows as R
        pos, slots = torch.tensor([t], dtype=torch.int32).cuda(), torch.tensor([slot], dtype=torch.int32).cuda()
        out = torch.empty(1, self.inner, device="cuda")
        p = self.p[t:t + 1].cuda()
        dt = (p[:, :self.r].double() @ self.w_dt.double().cuda().t()).float().contiguous() if given else None
        R.ssm_step(self.xz[t:t + 1].cuda(), self.inner, (self.conv_w.cuda(), self.conv_b.cuda(), self.conv_state), p, self.r8, self.wp.cuda(), dt, self.bias.cuda(),
                   self.a2, self.d.cuda(), self.state, slots, pos, out, 1, self.dtype == torch.float32)
        return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("inner,n,r,taps", [(8, 1, 1, 1), (56, 10, 5, 4), (40, 16, 8, 2), (72, 33, 20, 3), (24, 70, 3, 5), (16, 200, 12, 4), (136, 32, 9, 3)])
def test_state_space_portions_and_steps(dtype, inner, n, r, taps):
    T = 140
    s = Ssm(inner, n, r, taps, T, dtype, seed=inner)
    want = s.expected()
    tol = 2e-5 if dtype == torch.float32 else 1.2e-2
    for slot, cuts in ((0, [T]), (1, [2, 2, 33, 1, 64, 31, T])):
        at, us, ys = 0, [], []
        for c in cuts:
            if at < T:
                u, y = s.portions(slot, at, min(at + c, T))
                us.append(u), ys.append(y)
                at += c
        close(torch.cat(us), s.u, close_in(dtype))
        close(torch.cat(ys), want, tol)
    for given in (False, True):      # a prompt, then token by token; and a sequence that is decoded from its first token
        s.portions(0, 0, 90)
        close(torch.cat([s.step(0, t, given) for t in range(90, 120)]), want[90:120], tol)
        close(torch.cat([s.step(1, t, given) for t in range(0, 30)]), want[:30], tol)


@pytest.mark.parametrize("given", [False, True])
def test_convolution_in_the_decode_product(given):
    """Rows 12, 2 and 0 of three sequences as outputs of a product (with an identity matrix): its epilogue convolves them with the slots' last
    inputs, and the step takes the result."""
    from ollama_b200.ops import rows as R
    s = Ssm(56, 10, 5, 4, 20, torch.bfloat16, seed=2)
    want = s.expected()
    s.portions(0, 0, 12)
    s.portions(1, 0, 2)
    at = [12, 2, 0]
    x = s.xz[at].float().cuda()
    eye = torch.eye(112, dtype=torch.bfloat16, device="cuda")
    slots, pos = torch.tensor([0, 1, 2], dtype=torch.int32).cuda(), torch.tensor(at, dtype=torch.int32).cuda()
    xz, u, out = torch.zeros(3, 112, device="cuda"), torch.full((3, 64), 9.0, device="cuda"), torch.zeros(3, 56, device="cuda")
    conv = (s.conv_w.cuda(), s.conv_b.cuda(), s.conv_state)
    R.gemv([R.seg(eye, 112, xz)], 112, x, 3, False, conv=conv, conv_out=u, slots=slots, positions=pos)
    assert torch.equal(xz, x) and (u[:, 56:] == 9).all()
    close(u[:, :56], s.u[at], 1e-5)
    R.ssm_step(xz, 56, conv, s.p[at].cuda(), s.r8, s.wp.cuda(), None, s.bias.cuda(), s.a2, s.d.cuda(), s.state, slots, pos, out, 3, u=u if given else None)
    close(out, want[at], 1e-2)
