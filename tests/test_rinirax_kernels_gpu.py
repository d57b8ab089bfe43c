"""Kernels behind Rinirax models, one mechanism at a time, each against the plain formulas in 64 bits.  Inputs are made so that a fault shows: in the attention tests one
key carries nearly all of a query's weight in one of the maps, in the recurrence tests slow gates keep the first tokens alive."""
import math

import pytest
import torch

import rinirax_oracle as O
from test_tirudra_kernels_gpu import F64, close, i32, rnd, up

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module", autouse=True)
def no_timeouts():
    from ollama_b200.ops import cuda as K
    K.need("stack")
    yield
    assert K.gemm_status() == 0


# -- average over depth ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("n,k", [(1, 52), (2, 1), (3, 37), (9, 264), (40, 2052), (7, 5000), (33, 4096), (12, 9000)])
@pytest.mark.parametrize("rows", [1, 3, 70])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 5e-3)])
def test_sum_over_depth_and_its_layer_norm(n, k, rows, dtype, tol):
    from ollama_b200.ops import rows as R
    kp, eps = up(k), 1e-4
    hist = torch.full((n + 2, rows, kp), 9.0).cuda()
    hist[:n, :, :k], hist[:n, :, k:] = rnd(n, rows, k, seed=n).cuda() + 3.0, 0.0         # a mean that a one-pass variance would suffer from
    w, g, b = rnd(n, seed=1).cuda(), rnd(kp, seed=2).cuda(), rnd(kp, seed=3).cuda()
    want = torch.einsum("j,jrk->rk", w.double(), hist[:n, :, :k].double()).cpu()
    h = torch.full((rows, kp), 7.0, device="cuda", dtype=dtype)
    x = R.depth_rows(hist, n, w, k, eps, g, b, h)
    assert x.data_ptr() == hist[n].data_ptr()
    close(x[:, :k], want, 1e-6)
    close(h[:, :k], O.layer_norm(want, g[:k].double().cpu(), b[:k].double().cpu(), eps), tol if k > 1 else 1.0)
    assert (h[:, k:] == 0).all() and (x[:, k:] == 0).all() and (hist[n + 1] == 9).all()
    hist[n] = 5.0
    R.depth_rows(hist, n, w, k, eps)
    close(hist[n, :, :k], want, 1e-6)


# -- gated recurrence -----------------------------------------------------------------------------------------------
def gru_rows(rows, width, dtype, seed=0):
    """(rows [z' | u | g], width padded to vectors) with gates from nearly closed to open."""
    wp = up(width)
    x = torch.zeros(rows, 3 * wp)
    x[:, :width] = rnd(rows, width, seed=seed, scale=1.5) + torch.linspace(-7.0, 2.0, width)
    x[:, wp:wp + width], x[:, 2 * wp:2 * wp + width] = rnd(rows, width, seed=seed + 1, scale=2.0), rnd(rows, width, seed=seed + 2)
    x[0, :width] = 3.0                       # the first token opens the gates
    x[0, wp:wp + width] = 40.0
    return x.to(dtype).cuda(), wp


def gru_want(x, width, wp):
    x = x.double().cpu()
    return O.gru_scan(x[:, :width], x[:, wp:wp + width]) * O.silu(x[:, 2 * wp:2 * wp + width])


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 5e-3)])
@pytest.mark.parametrize("width", [1, 33, 264])
@pytest.mark.parametrize("cuts", [[1], [5], [255, 1, 256, 2, 257], [700, 3], [2, 2, 2, 2100], [4300, 40]])
def test_recurrence_over_portions_and_single_tokens(dtype, tol, width, cuts):
    from ollama_b200.ops import rows as R
    n = sum(cuts) + 3
    x, wp = gru_rows(n, width, dtype)
    want = gru_want(x, width, wp)
    state, at, got = torch.full((3, wp), 77.0).cuda(), 0, []
    for c in cuts:
        out = torch.full((c, wp + 8), 5.0, device="cuda", dtype=dtype)
        R.gru_scan(x[at:at + c], wp, state, torch.tensor([[0, c, 2, at]], dtype=torch.int32).cuda(), c, out[:, :wp])
        assert (out[:, wp:] == 5).all()
        got.append(out[:, :width])
        at += c
    for i in range(3):
        out = torch.full((1, wp), 5.0, device="cuda", dtype=dtype)
        R.gru_step(x[at:at + 1], wp, state, i32(2), i32(at), out, exact=dtype == torch.float32)
        got.append(out[:, :width])
        at += 1
    close(torch.cat(got), want, tol)
    assert (state[:2] == 77).all()


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 5e-3)])
def test_recurrence_of_unequal_portions_side_by_side(dtype, tol):
    from ollama_b200.ops import rows as R
    width, lens = 40, [2, 900, 1, 256, 31]
    x, wp = gru_rows(sum(lens), width, dtype, seed=5)
    state = torch.full((9, wp), 7.0).cuda()
    segs, at = [], 0
    for i, n in enumerate(lens):
        segs.append((at, n, 8 - i, 0))
        at += n
    out = torch.empty(sum(lens), wp, device="cuda", dtype=dtype)
    R.gru_scan(x, wp, state, torch.tensor(segs, dtype=torch.int32).cuda(), max(lens), out)
    for a, n, _, _ in segs:
        close(out[a:a + n, :width], gru_want(x[a:a + n], width, wp), tol)


# -- differential attention -----------------------------------------------------------------------------------------
class Diff:
    """One sequence in slot 1 of a paged cache with scattered pages; rows of [q | k | v], rotation in the half-split order."""

    def __init__(self, H, G, dim, vdim, n, kind, dims=0, lam=0.4, seed=0):
        self.H, self.G, self.dim, self.vdim, self.n, self.lam, self.offset, self.eps, self.f32 = H, G, dim, vdim, n, lam, 0.3, 1e-3, kind == "f32"
        self.scale, self.nq, self.nk = 0.7 / math.sqrt(dim), 2 * H * dim, 2 * G * dim
        self.rows_in = rnd(n, up(self.nq + self.nk + G * vdim), seed=seed)
        self.freqs = O.rotation({"base": 60.0, "dims": dims})[0] if dims else torch.zeros(0, dtype=F64)
        big = max(2 * dim, vdim)
        self.hd = 0 if kind != "tc" else 64 if big <= 64 else 128
        pages = -(-n // 64)
        self.table = torch.zeros(2, pages + 1, dtype=torch.int32).cuda()
        self.table[1, :pages] = torch.randperm(pages + 3, generator=torch.Generator().manual_seed(seed))[:pages].to(torch.int32).cuda()
        dk, dv = (self.hd, self.hd) if self.hd else (up(2 * dim), up(vdim))
        dt = torch.float32 if self.f32 else torch.float16
        self.kc, self.vc = torch.full((pages + 3, G, 64, dk), 7.0, dtype=dt, device="cuda"), torch.full((pages + 3, G, 64, dv), -9.0, dtype=dt, device="cuda")

    def aim(self, pairs, strength=6.0):
        """The query at position i finds the key at position j and little else in map m, for the (i, j, m) of ``pairs`` (without rotation)."""
        for i, j, m in pairs:
            k = self.rows_in[j, self.nq:self.nq + self.nk].view(self.G, 2, self.dim)
            k[:, m] *= strength / k[:, m].norm(dim=-1, keepdim=True)
            q = self.rows_in[i, :self.nq].view(self.H, 2, self.dim)
            q[:, m] = (k[:, m] * math.sqrt(self.dim)).repeat_interleave(self.H // self.G, 0)

    def expected(self):
        x, n, pos = self.rows_in.double(), self.n, torch.arange(self.n)
        q, k = x[:, :self.nq].view(n, 2 * self.H, self.dim), x[:, self.nq:self.nq + self.nk].view(n, 2 * self.G, self.dim)
        if len(self.freqs):
            from tirudra_oracle import rotate_half
            q, k = (rotate_half(t, pos, self.freqs) for t in (q, k))
        q, k, v = q.view(n, self.H, 2, -1), k.view(n, self.G, 2, -1), x[:, self.nq + self.nk:self.nq + self.nk + self.G * self.vdim].view(n, self.G, self.vdim)
        a = [O.attend(q[:, :, m], k[:, :, m], v, self.scale, O.window_visible(n)) for m in range(2)]
        return O.diff_combine(*a, self.lam, self.offset, self.eps).reshape(n, -1)

    def _prep(self):
        from ollama_b200.ops import rows as R
        self.f = (self.freqs if len(self.freqs) else torch.zeros(1, dtype=F64)).cuda()
        self.d = R.DiffHeads(self.lam, 1.0 - self.offset, self.eps, 1)
        return R, dict(heads=2 * self.H, maps=2, dim=self.dim, vdim=self.vdim, q_norm=None, k_norm=None, eps=0.0, freqs=self.f, n_rot=2 * len(self.freqs))

    def rows(self, lo, hi, append=True):
        m, x = hi - lo, self.rows_in[lo:hi].cuda()
        x = x if append else x[:, :up(self.nq, 4)].contiguous()
        R, prep = self._prep()
        pos, slots = torch.arange(lo, hi, dtype=torch.int32).cuda(), torch.ones(m, dtype=torch.int32).cuda()
        q = torch.full((m, 2 * self.H, self.hd or 2 * self.dim), 3.0, device="cuda")
        R.paged_append(x, kv_heads=self.G, positions=pos, slots=slots, table=self.table, q_out=q, k_cache=self.kc, v_cache=self.vc, append=append, **prep)
        out = torch.full((m, up(self.H * self.vdim + 1)), 5.0, device="cuda", dtype=torch.float32 if self.f32 else torch.bfloat16)
        if self.hd:
            tiles = torch.tensor([(r, min(64, m - r), 1, lo + r) for r in range(0, m, 64)], dtype=torch.int32).cuda()
            R.attn_prefill_paged(q, self.kc, self.vc, tiles, self.table, out, vdim=self.vdim, scale=self.scale, diff=self.d)
        else:
            both = torch.empty(m, 2 * self.H * self.vdim, device="cuda")
            R.paged_attn(q, self.kc, self.vc, pos, slots, self.table, both, dim=2 * self.dim, vdim=self.vdim, scale=self.scale)
            R.diff_rows(both, self.H, self.vdim, self.d, out)
        assert (out[:, self.H * self.vdim:] == 5).all()
        return out[:, :self.H * self.vdim]

    def decode(self, p, splits, append=True):
        x = self.rows_in[p:p + 1].cuda()
        x = x if append else x[:, :up(self.nq, 4)].contiguous()
        R, prep = self._prep()
        acc, ml = torch.empty(2 * self.H * splits * self.hd, device="cuda"), torch.empty(2 * self.H * splits * 2, device="cuda")
        out = torch.full((1, self.H * self.vdim + 3), 5.0, device="cuda")
        assert R.attn_decode_paged(x, self.kc, self.vc, i32(p), i32(1), self.table, out, 1, softcap=0.0, chunk=0, n_splits=splits, n_ctx=max(self.n, 64), part_acc=acc, part_ml=ml,
                                   scale=self.scale, append=append, diff=self.d, **prep)
        assert (out[:, self.H * self.vdim:] == 5).all()
        return out[:, :self.H * self.vdim]


SHAPES = [(3, 1, 20, 36, 8), (2, 2, 12, 32, 0), (4, 2, 32, 64, 32), (8, 1, 64, 128, 64), (6, 3, 48, 90, 0), (1, 1, 2, 1, 2), (8, 8, 30, 30, 6), (5, 1, 33, 100, 10)]
TOL = {"tc": 1.2e-2, "f16": 1.2e-2, "f32": 2e-5}


def pairs_for(n):
    return [(n - 1, 0, 0), (n - 2, 0, 1), (n - 3, 63, 0), (n - 4, 64, 1), (130, 128, 0), (129, 127, 1), (128, 128, 1), (65, 1, 0), (64, 64, 0)]


@pytest.mark.parametrize("kind", ["tc", "f16", "f32"])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("rotated", [False, True])
def test_differential_attention_of_portions_and_decoded_tokens(shape, kind, rotated):
    H, G, dim, vdim, dims = shape
    n = 331
    a = Diff(H, G, dim, vdim, n, kind, dims if rotated else 0)
    a.aim(pairs_for(n))
    want = a.expected()
    lo, tol = 0, TOL[kind] * (20 if vdim == 1 else 1)      # a head of one value is little more than a sign
    for size in (200, 1, 2, 64, 63, 1):
        close(a.rows(lo, lo + size), want[lo:lo + size], tol)
        lo += size
    if a.hd:
        for splits in (1, 3, 11):
            a.kc[a.table[1, n // 64].long(), :, (n - 1) % 64] = 7.0                # the token's own row is written by the launch
            close(a.decode(n - 1, splits), want[n - 1:], tol)
    # the same queries on keys and values that are there already
    close(a.rows(0, 190, append=False), want[:190], tol)
    if a.hd:
        kc = a.kc.clone()
        for p in (0, 63, 64, 129, n - 1):
            close(a.decode(p, 4, append=False), want[p:p + 1], tol)
        assert torch.equal(kc, a.kc)


def test_more_maps_than_a_decode_tile_has_rows_are_left_to_the_plain_kernel():
    a = Diff(9, 1, 16, 16, 70, "tc")
    R, prep = a._prep()
    x, one = a.rows_in[:1].cuda(), torch.empty(1).cuda()
    assert not R.attn_decode_paged(x, a.kc, a.vc, i32(0), i32(1), a.table, torch.zeros(1, 9 * 16).cuda(), 1, softcap=0.0, chunk=0, n_splits=1, n_ctx=64, part_acc=one, part_ml=one,
                                   scale=1.0, diff=a.d, **prep)


# -- latent attention under a window ---------------------------------------------------------------------------------
@pytest.mark.parametrize("window", [1, 2, 37, 64, 65, 128, 200, 1000])
@pytest.mark.parametrize("heads,rank,rot,splits", [(3, 36, 8, 1), (20, 300, 64, 3), (16, 128, 16, 7)])
def test_latent_scores_inside_a_window(window, heads, rank, rot, splits):
    from ollama_b200.ops import latent as A
    cp, T = up(rank, 16), 333
    w = up(cp + rot, 32)
    rows = torch.zeros(T, w)
    rows[:, :rank], rows[:, cp:cp + rot] = rnd(T, rank), rnd(T, rot, seed=1)
    at = [0, 5, 63, 64, 127, 128, 191, 200, 331, 332]
    n = len(at)
    q = torch.zeros(n, heads, w)
    q[..., :rank], q[..., cp:cp + rot] = 0.3 * rnd(n, heads, rank, seed=4), 0.3 * rnd(n, heads, rot, seed=5)
    rows[:, 0], q[..., 0] = 0.0, 7.0
    for p in at:                             # standing-out keys just inside and just outside
        for j in (p - window, p - window + 1):
            if j >= 0:
                rows[j, 0] = 7.0
    perm = torch.randperm(8, generator=torch.Generator().manual_seed(heads))[:6]
    cache = torch.full((8, 1, 64, w), 3.0)
    for j in range(T):
        cache[perm[j // 64], 0, j % 64] = rows[j]
    table = torch.zeros(2, 6, dtype=torch.int32)
    table[1] = perm
    qh, ch = q.half(), rows.half().double()
    acc, ml = torch.full((n, heads, splits, cp), math.nan, device="cuda"), torch.empty(n, heads, splits, 2, device="cuda")
    assert A.attn_latent(qh.cuda(), n, cache.half().cuda(), acc, ml, heads=heads, cp=cp, scale=0.9, splits=splits, positions=i32(*at), slots=i32(*[1] * n), table=table.cuda(), window=window)
    acc, ml = acc.double().cpu(), ml.double().cpu()
    for i, p in enumerate(at):
        lo = max(0, p - window + 1)
        want = torch.softmax(torch.einsum("hw,tw->ht", qh[i].double(), ch[lo:p + 1]) * 0.9, -1) @ ch[lo:p + 1, :cp]
        used = ml[i, :, :, 1] > 0
        c = torch.where(used, torch.exp(ml[i, :, :, 0] - ml[i, :, :, 0].max(-1, keepdim=True)[0]), 0.0)
        got = (torch.where(used[..., None], acc[i], 0.0) * c[..., None]).sum(1) / (c * ml[i, :, :, 1]).sum(-1, keepdim=True)
        close(got, want, 3e-3)


@pytest.mark.parametrize("window", [1, 37, 64, 127, 128, 129, 300, 2000])
@pytest.mark.parametrize("heads,dim,rot,vdim", [(2, 20, 8, 28), (3, 128, 64, 128), (4, 64, 0, 64)])
def test_prompt_tiles_inside_a_window(window, heads, dim, rot, vdim):
    """Portions of two sequences, the second far into its text: its buffer begins with a multiple of 128 before its first window."""
    from ollama_b200.ops import latent as A
    dp, rp, vp = up(dim, 64), up(rot, 64), up(vdim, 64)
    lens = [(0, 200), (500, 131)]                                # past, new tokens
    firsts = [max(0, p - window + 1) & ~127 for p, _ in lens]
    total = sum(p + n - f for (p, n), f in zip(lens, firsts))
    kv = torch.zeros(total, heads * (dp + vp), dtype=torch.float16)
    k, v = kv[:, :heads * dp].view(total, heads, dp), kv[:, heads * dp:].view(total, heads, vp)
    k[..., :dim], v[..., :vdim] = 0.5 * rnd(total, heads, dim).half(), rnd(total, heads, vdim, seed=1).half()
    sh = torch.zeros(total, max(rp, 8), dtype=torch.float16)
    sh[:, :rot] = rnd(total, rot, seed=2).half()
    rows = sum(n for _, n in lens)
    q = torch.zeros(rows, heads, dp + rp, dtype=torch.float16)
    q[..., :dim] = 0.5 * rnd(rows, heads, dim, seed=3).half()
    q[..., dp:dp + rot] = 0.3 * rnd(rows, heads, rot, seed=4).half()
    q[..., 0], k[..., 0] = 7.0, 0.0
    base, row0, tiles = 0, 0, []
    for (past, n), first in zip(lens, firsts):
        for p in (past + n - 1, past + 64, past + 128):
            for j in (p - window, p - window + 1):
                if first <= j < past + n:
                    k[base + j - first, :, 0] = 7.0
        tiles += [(row0 + t, min(128, n - t), base - first, past + t) for t in range(0, n, 128)]
        base, row0 = base + past + n - first, row0 + n
    out = torch.full((rows, heads * vdim + 4), 9.0, dtype=torch.bfloat16, device="cuda")
    A.attn_prefill_parts(q.cuda(), kv.cuda(), sh.cuda(), torch.tensor(tiles, dtype=torch.int32).cuda(), out, heads=heads, dp=dp, vp=vp, rp=rp, vdim=vdim, scale=0.8, window=window)
    base = row0 = 0
    for (past, n), first in zip(lens, firsts):
        T = past + n - first
        i, j = torch.arange(past, past + n)[:, None], torch.arange(first, past + n)[None]
        seen = (j <= i) & (i - j < window)
        for h in range(heads):
            s = q[row0:row0 + n, h, :dp].double() @ k[base:base + T, h].double().t()
            if rot:
                s += q[row0:row0 + n, h, dp:].double() @ sh[base:base + T, :rp].double().t()
            close(out[row0:row0 + n, h * vdim:(h + 1) * vdim], torch.softmax((s * 0.8).masked_fill(~seen, -math.inf), -1) @ v[base:base + T, h, :vdim].double(), 1e-2)
        base, row0 = base + T, row0 + n
    assert (out[:, heads * vdim:] == 9.0).all()


def test_gathered_latents_begin_where_they_are_seen():
    from ollama_b200.ops import latent as A
    cp, rot, w = 32, 6, 64
    cache = rnd(4, 1, 64, w).half().cuda()
    table = torch.tensor([[2, 0, 3], [1, 1, 1]], dtype=torch.int32).cuda()
    seqs = torch.tensor([(-128 + 3, 170, 0, 128), (45, 5, 1, 0)], dtype=torch.int32).cuda()
    c, r = torch.full((50, cp), 9.0, dtype=torch.bfloat16, device="cuda"), torch.full((50, 8), 9.0, dtype=torch.float16, device="cuda")
    A.latent_gather(cache, cp, rot, seqs, 42, table, c, r)
    assert torch.equal(c[3:45], cache[3, 0, :42, :cp].bfloat16()) and torch.equal(r[3:45, :rot], cache[3, 0, :42, cp:cp + rot])
    assert torch.equal(c[45:], cache[1, 0, :5, :cp].bfloat16()) and (c[:3] == 9).all() and (r[3:, rot:] == 0).all()


# -- experts and activation ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,groups,keep,ff,width", [(1, 1, 1, 1, 1, 8), (12, 3, 3, 2, 28, 52), (6, 6, 3, 3, 16, 37), (256, 8, 8, 4, 40, 136), (48, 2, 48, 5, 24, 64), (10, 5, 2, 1, 9, 40), (480, 16, 40, 7, 8, 24)])
@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("rows", [1, 3, 4, 70])
def test_experts_of_the_best_groups_beside_another_product(E, top, groups, keep, ff, width, f32, rows):
    """Both forms (few rows, sorted rows): sigmoid scores, corrections that make every choice score negative, the chosen weights, and a mixer's last product beside them."""
    from ollama_b200.engine import blocks as B
    from ollama_b200.engine.stack import _Rows
    from ollama_b200.models.stack import DESIGNS, Expert, ExpertMLP
    dt = torch.float32 if f32 else torch.bfloat16

    def t(*s, seed, scale=1.0):
        return rnd(*s, seed=seed, scale=scale).to(dt)
    w = {"router": t(E, width, seed=1, scale=2 / math.sqrt(width)), "correction": rnd(E, seed=2, scale=0.5) - 1.6}
    for e in range(E):
        for i, (name, s) in enumerate((("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))):
            w[f"e{e}.{name}"] = t(*s, seed=10 * e + i, scale=1.5 * s[1] ** -0.5)
    names = {"ffn_gate_inp.weight": w["router"], "exp_probs_b.bias": w["correction"]}
    for name in ("gate", "up", "down"):
        names[f"ffn_{name}_exps.weight"] = torch.stack([w[f"e{e}.{name}"] for e in range(E)])
    src = B.WeightSource(lambda name: names[name].float().cuda(), "cuda", dt, width)

    class Engine:
        class stack:
            eps, residual_mult, design = 1e-5, 1.0, DESIGNS["Rinirax"]
        wp, pdl, _n, gemv_rows, act_dtype = src.wp, True, 0, 4, dt
    Engine.f32, Engine.stack.width = f32, width

    class Meta:
        tokens = torch.zeros(rows, dtype=torch.int32).cuda()
    x = torch.zeros(rows, src.wp).cuda()
    x[:, :width] = rnd(rows, width, seed=6).cuda()
    start = x[:, :width].double().cpu()
    ffn = B.ExpertFFN(src, "", ExpertMLP(E, top, Expert(ff), groups=groups, keep=keep, scale=1.7, **DESIGNS["Rinirax"].experts), None, f32)
    s = B.Step(Engine(), _Rows(rows, "cuda"), Meta(), x, None, rows <= 4)
    h = torch.zeros(rows, src.wp, device="cuda", dtype=s.act)
    h[:, :width] = rnd(rows, width, seed=7).cuda().to(dt).to(s.act)
    h64 = h[:, :width].double().cpu()
    z = torch.zeros(rows, ffn.router.w.shape[0], device="cuda")
    s.product(h, ffn.router, z)
    close(z[:, :E], h64 @ w["router"].double().t(), 1e-5)
    other, cols = torch.zeros(src.wp, 24, device="cuda", dtype=dt), rnd(rows, 24, seed=9).cuda()
    other[:width] = t(width, 24, seed=8, scale=0.2).cuda()
    if s.small:
        ffn.mix(s, h, z, beside=B.Mat(other), fill=lambda out: out.copy_(cols))
    else:
        ffn.mix(s, h, z)
        s.add(cols.to(s.act), B.Mat(other))
    cfg = {"router": {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}, "scale": 1.7}}
    want = start + O.moe_ff(h64, lambda name: w[name].double(), cfg) + cols.double().cpu() @ other[:width].double().cpu().t()
    close(s.x[:, :width], want, 3e-5 if f32 else 1.5e-2)
    assert (s.x[:, width:] == 0).all()


@pytest.mark.parametrize("m", [1, 4, 5, 33, 200, 1200])
@pytest.mark.parametrize("n,k", [(8, 40), (104, 72), (1000, 2048), (2600, 264)])
@pytest.mark.parametrize("f32", [False, True])
def test_activation_with_two_numbers_behind_every_kind_of_product(m, n, k, f32):
    from ollama_b200.ops import rows as R
    dt = torch.float32 if f32 else torch.bfloat16
    x, w = rnd(m, k, seed=1).to(dt).cuda(), (2.5 * rnd(n, k, seed=2) / math.sqrt(k)).to(dt).cuda()
    p, q = 0.37, 0.9
    z = x.double() @ w.double().t()
    neg = torch.clamp(z, max=0.0)
    want = torch.where(z > 0, p * z * z, q * (torch.expm1(neg) - neg)) + 0.5 * z
    wide = torch.full((m, n + 16), 9.0, device="cuda", dtype=dt)
    R.gemm(x, w, wide[:, 8:8 + n], act="xielu", nums=(p, q))
    close(wide[:, 8:8 + n], want, 5e-6 if f32 else 6e-3)
    assert (wide[:, :8] == 9).all() and (wide[:, 8 + n:] == 9).all()
    if not f32:
        out = torch.empty(m, n, device="cuda")
        R.gemm(x, w, out, act="xielu", nums=(p, q))
        close(out, want, 1e-5)
    if m <= 4:
        out = torch.full((m, n), 9.0, device="cuda")
        R.gemv([R.seg(w, n, out, act="xielu", nums=(p, q))], k, x.float(), m, f32)
        close(out, want, 1e-5)
    assert torch.allclose(want.cpu(), O.xielu(z.cpu(), torch.log(torch.expm1(torch.tensor(p, dtype=F64))), torch.log(torch.expm1(torch.tensor(q - 0.5, dtype=F64)))))
