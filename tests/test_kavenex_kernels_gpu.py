"""Kernels behind Kavenex models, each against the plain formulas in 64 bits."""
import math

import pytest
import torch

import kavenex_oracle as O

pytestmark = pytest.mark.gpu
F64 = torch.float64


@pytest.fixture(scope="module")
def ops():
    from ollama_b200.ops import cuda as K
    from ollama_b200.ops import latent as A
    from ollama_b200.ops import rows as R
    yield K, A, R
    assert K.gemm_status() == 0


def rnd(*s, seed=0, dtype=torch.float32, scale=1.0):
    return (torch.randn(*s, generator=torch.Generator().manual_seed(seed + sum(s))) * scale).to(dtype).cuda()


def close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    err = (got - want).abs().max() / want.abs().max().clamp(min=1e-9)
    assert torch.isfinite(got).all() and err < tol, float(err)


def up(n, m=8):
    return -(-n // m) * m


@pytest.mark.parametrize("k", [1, 37, 52, 2048, 4100])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 5e-3)])
def test_layer_norm_with_the_update_before_it(ops, k, dtype, tol):
    K, A, R = ops
    kp, rows, eps = up(k), 5, 1e-5
    x = torch.zeros(rows, kp).cuda()
    x[:, :k] = rnd(rows, k) + 4.0                                # a mean well away from zero
    y, x0 = rnd(rows, kp, seed=1), rnd(rows, kp, seed=2)
    vec = [torch.cat([rnd(k, seed=3 + i), torch.zeros(kp - k).cuda()]) for i in range(6)]
    w1, b1, w2, b2, wy, step = vec
    want = x[:, :k].double() + 0.7 * O.norm_plain(y[:, :k].double(), wy[:k].double(), eps) + x0[:, :k].double() + step[:k].double()
    o1, o2 = torch.full((rows, kp), 9.0, device="cuda", dtype=dtype), torch.full((rows, kp), 9.0, device="cuda", dtype=dtype)
    R.norm_rows(x, k, eps, w1, o1, w2, o2, b1, b2, y=y, wy=wy, mult=0.7, x0=x0, step=step)
    close(x[:, :k], want, 1e-6)
    close(o1[:, :k], O.layer_norm(want, w1[:k].double(), b1[:k].double(), eps), tol)
    close(o2[:, :k], O.layer_norm(want, w2[:k].double(), b2[:k].double(), eps), tol)
    assert (o1[:, k:] == 0).all() and (x[:, k:] == 0).all()
    before = x.clone()
    R.norm_rows(x, k, eps, None, None, step=step)                # the update alone
    close(x[:, :k], before[:, :k].double() + step[:k].double(), 1e-6)


@pytest.mark.parametrize("nb", [1, 2, 3, 4])
@pytest.mark.parametrize("k,n", [(8, 2), (52, 34), (2048, 600), (4096, 30)])
def test_decode_product_with_folded_layer_norm(ops, nb, k, n):
    K, A, R = ops
    kp, eps = up(k), 1e-5
    x = torch.zeros(nb, kp).cuda()
    x[:, :k] = rnd(nb, k) * 2 + 1.5
    g, b = torch.zeros(kp).cuda(), torch.zeros(kp).cuda()
    g[:k], b[:k] = rnd(k, seed=1), rnd(k, seed=2)
    w = torch.zeros(n, kp, dtype=torch.bfloat16, device="cuda")
    w[:, :k] = rnd(n, k, seed=3, scale=k ** -0.5)
    bias = rnd(n, seed=4)
    rs, rc = w.float() @ g, w.float() @ b + bias
    h64 = O.layer_norm(x[:, :k].double(), g[:k].double(), b[:k].double(), eps)
    want = h64 @ w[:, :k].double().t() + bias.double()
    out, h = torch.zeros(nb, n).cuda(), torch.full((nb, kp), 9.0, device="cuda")
    R.gemv([R.seg(w, n, out, g, rs=rs, rc=rc)], kp, x, nb, False, R.SRC_LAYER, eps, k, h=h, hb=b)
    close(out, want, 2e-5)
    close(h[:, :k], h64, 1e-5)
    assert (h[:, k:] == 0).all()
    gu = torch.zeros(nb, n // 2).cuda()
    R.gemv([R.seg(w, n, gu, g, act="glu:gelu_tanh", rs=rs, rc=rc)], kp, x, nb, False, R.SRC_LAYER, eps, k)
    close(gu, O.gelu_tanh(want[:, 0::2]) * want[:, 1::2], 3e-5)


@pytest.mark.parametrize("f32", [False, True])
def test_decode_product_epilogues(ops, f32):
    K, A, R = ops
    nb, k, n, dt = 3, 264, 46, torch.float32 if f32 else torch.bfloat16
    x, w, table, tok = rnd(nb, k), rnd(n, k, dtype=dt, scale=0.1), rnd(9, 48, dtype=dt, seed=5), torch.tensor([8, 0, 3], dtype=torch.int32).cuda()
    p = x.double() @ w.double().t()
    out = torch.zeros(nb, 48).cuda()
    R.gemv([R.seg(w, n, out, act="gelu_tanh", mul=table)], k, x, nb, f32, mul_row=tok)
    close(out[:, :n], O.gelu_tanh(p) * table[tok.long()].double()[:, :n], 1e-5)
    acc = rnd(nb, n, seed=6)
    want = acc.double() - 0.3 * p
    R.gemv([R.seg(w, n, acc, accumulate=True, alpha=-0.3)], k, x, nb, f32)
    close(acc, want, 1e-5)
    h = torch.zeros(nb, n // 2).cuda()
    R.gemv([R.seg(w, n, h, act="glu:swiglu_oai", limit=0.6)], k, x, nb, f32)
    g, u = p[:, 0::2].clamp(max=0.6), p[:, 1::2].clamp(-0.6, 0.6)
    close(h, g * torch.sigmoid(1.702 * g) * (u + 1), 1e-5)


@pytest.mark.parametrize("m,n,k", [(5, 64, 2048), (70, 24, 40), (200, 256, 512), (300, 520, 1032)])
@pytest.mark.parametrize("f32", [False, True])
def test_products_of_many_rows(ops, m, n, k, f32):
    """Every epilogue, in one launch and (few rows, long rows) split along k."""
    K, A, R = ops
    dt, tol = (torch.float32, 1e-5) if f32 else (torch.bfloat16, 6e-3)
    a, w = rnd(m, k, dtype=dt), rnd(n, k, dtype=dt, scale=k ** -0.5)
    bias, table, tok = rnd(n, seed=7), rnd(11, n, dtype=dt, seed=8), torch.randint(0, 11, (m,), dtype=torch.int32).cuda()
    p = a.double() @ w.double().t() + bias.double()
    types = [torch.float32] if f32 else [torch.float32, torch.bfloat16, torch.float16]
    for t in types:
        out = torch.zeros(m, n, device="cuda", dtype=t)
        R.gemm(a, w, out, bias=bias, act="gelu_tanh", mul=table, mul_row=tok, alpha=1.7)
        close(out, 1.7 * O.gelu_tanh(p) * table[tok.long()].double(), tol if t != torch.float32 else 2e-5)
    acc = rnd(m, n, seed=9)
    want = acc.double() + 0.4 * p
    copy = None if f32 else torch.zeros(m, n, device="cuda", dtype=dt)
    R.gemm(a, w, acc, bias=bias, accumulate=True, alpha=0.4, copy=copy)
    close(acc, want, 2e-5)
    assert f32 or torch.equal(copy, acc.to(dt))
    if n % 8 == 0:
        h = torch.zeros(m, n // 2, device="cuda", dtype=dt)
        R.gemm(a, w, h, bias=bias, act="glu:gelu_tanh")
        close(h, O.gelu_tanh(p[:, 0::2]) * p[:, 1::2], tol)


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("E,top,ff,sff,width", [(1, 1, 1, 0, 8), (6, 2, 28, 20, 52), (9, 4, 16, 0, 37), (300, 16, 40, 130, 264)])
@pytest.mark.parametrize("rows", [1, 3, 4, 70])
def test_experts(ops, f32, E, top, ff, sff, width, rows):
    """Both forms (few rows, sorted rows): the router's choice, limits that bind, the shared expert and the residual."""
    from ollama_b200.engine import blocks as B
    from ollama_b200.models.stack import Expert, ExpertMLP
    K, A, R = ops
    dt = torch.float32 if f32 else torch.bfloat16
    w = {"router": rnd(E, width, seed=1, dtype=dt), "router.b": rnd(E, seed=2)}
    for e in range(E):
        for i, (n, s) in enumerate((("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))):
            w[f"e{e}.{n}"] = rnd(*s, seed=10 * e + i, dtype=dt, scale=1.5 * s[1] ** -0.5)
    for i, (n, s) in enumerate((("gate", (sff, width)), ("up", (sff, width)), ("down", (width, sff)))):
        if sff:
            w[f"shared.{n}"] = rnd(*s, seed=900 + i, dtype=dt, scale=1.5 * s[1] ** -0.5)
    names = {"ffn_gate_inp.weight": w["router"], "ffn_gate_inp.bias": w["router.b"]}
    for n in ("gate", "up", "down"):
        names[f"ffn_{n}_exps.weight"] = torch.stack([w[f"e{e}.{n}"] for e in range(E)])
        if sff:
            names[f"ffn_{n}_shexp.weight"] = w[f"shared.{n}"]
    src = B.WeightSource(lambda n: names[n].float(), "cuda", dt, width)
    norm = B.Norm(torch.zeros(src.wp).cuda(), torch.zeros(src.wp).cuda())
    norm.g[:width], norm.b[:width] = 1.0 + 0.2 * rnd(width, seed=3), rnd(width, seed=4)

    class Engine:
        class stack:
            eps, residual_mult = 1e-5, -0.6
        wp, pdl, _n, gemv_rows = src.wp, True, 0, 4
        act_dtype = dt
    Engine.f32, Engine.stack.width = f32, width
    from ollama_b200.engine.stack import _Rows
    x = torch.zeros(rows, src.wp).cuda()
    x[:, :width] = rnd(rows, width, seed=5)
    m = ExpertMLP(E, top, Expert(ff, 0.8), Expert(sff, 0.5) if sff else None)
    ffn = B.ExpertFFN(src, "", m, norm, f32)

    class Meta:
        tokens = torch.zeros(rows, dtype=torch.int32).cuda()
    h = O.layer_norm(x[:, :width].double(), norm.g[:width].double(), norm.b[:width].double(), 1e-5)
    if not f32 and rows > 4:
        h = h.to(torch.bfloat16).double()                        # what the products read there: no test of a close call
    cfg = {"router": {"experts": E, "top": top}, "expert": {"limit": 0.8}, "shared": {"limit": 0.5} if sff else None}
    want = x[:, :width].double() - 0.6 * O.moe_ff(h, lambda n: w[n].double(), cfg)
    ffn.run(B.Step(Engine(), _Rows(rows, "cuda"), Meta(), x, None, rows <= 4))
    close(x[:, :width], want, 1e-5 if f32 else 1e-2)
    assert (x[:, width:] == 0).all()


def needle(q, c, at, r):
    """Let the query rows ``q`` find the cache rows at positions ``at`` and nothing else: scores there stand out by tens."""
    c[at] = 0.0
    c[at, r] = 6.0
    q[..., r] = 6.0


def cache_of(rows, w, table_row, n_pages, dtype):
    """Rows [n, w] of one sequence in pages."""
    cache = torch.full((n_pages, 1, 64, w), 30.0, dtype=dtype, device="cuda")      # what is not the sequence's must not matter
    for p in range(0, len(rows), 64):
        part = rows[p:p + 64]
        cache[table_row[p // 64], 0, :len(part)] = part.to(dtype)
    return cache


@pytest.mark.parametrize("heads,rank,rot", [(1, 1, 2), (3, 36, 8), (16, 128, 64), (17, 96, 32), (40, 512, 64), (16, 512, 128), (5, 200, 0)])
@pytest.mark.parametrize("splits", [1, 3, 128])
def test_latent_scores_at_every_kind_of_place(ops, heads, rank, rot, splits):
    """Single standing-out keys first, last, at page borders and far away; queries at several positions; a value product behind it, both ways."""
    K, A, R = ops
    cp, vdim = up(rank, 16), 19
    w = up(cp + rot, 32)
    T = 333
    rows = torch.zeros(T, w).cuda()
    rows[:, :rank] = rnd(T, rank)
    rows[:, cp:cp + rot] = rnd(T, rot, seed=1) if rot else 0
    perm = torch.randperm(12, generator=torch.Generator().manual_seed(heads)).tolist()
    uv = torch.zeros(heads * vdim, cp, dtype=torch.bfloat16, device="cuda")
    uv[:, :rank] = rnd(heads * vdim, rank, seed=3, scale=rank ** -0.5)
    places, at = [0, 1, 62, 63, 64, 65, 127, 128, 200, 331, 332], [0, 5, 63, 64, 127, 128, 191, 200, 332, 332, 332]
    n = len(at)
    q = torch.zeros(n, heads, w).cuda()
    q[..., :rank] = 0.3 * rnd(n, heads, rank, seed=4)
    q[..., cp:cp + rot] = 0.3 * rnd(n, heads, rot, seed=5) if rot else 0
    needle(q, rows, [p for p in places if p < T], 0)
    rows[:, 1 % rank] = rnd(T, seed=6)
    table = torch.zeros(2, 6, dtype=torch.int32)
    table[1] = torch.tensor(perm[:6])
    table = table.cuda()
    cache = cache_of(rows, w, perm, 12, torch.float16)
    pos, slots = torch.tensor(at, dtype=torch.int32).cuda(), torch.ones(n, dtype=torch.int32).cuda()
    qh, ch = q.half(), rows.half().double()
    want_lat = torch.zeros(n, heads, cp, dtype=F64).cuda()
    for i, p in enumerate(at):
        s = torch.softmax(torch.einsum("hw,tw->ht", qh[i].double(), ch[:p + 1]) * 0.9, -1)
        want_lat[i] = s @ ch[:p + 1, :cp]
    want = torch.einsum("nhc,hvc->nhv", want_lat, uv.double().view(heads, vdim, cp)).reshape(n, -1)
    acc, ml = torch.full((n, heads, splits, cp), math.nan, device="cuda"), torch.empty(n, heads, splits, 2, device="cuda")
    assert A.attn_latent(qh, n, cache, acc, ml, heads=heads, cp=cp, scale=0.9, splits=splits, positions=pos, slots=slots, table=table)
    for merged in (None, torch.empty(n, heads, cp, dtype=torch.bfloat16, device="cuda")):
        out = torch.zeros(n, up(heads * vdim)).cuda()
        A.latent_merge(acc, ml, n, uv, out, heads=heads, splits=splits, cp=cp, vdim=vdim, merged=merged)
        close(out[:, :heads * vdim], want, 2e-3 if merged is None else 8e-3)
    # the listed rows of a larger step, in another order
    order = torch.tensor([7, 2, 9], dtype=torch.int32).cuda()
    acc, ml, out = acc[:3], ml[:3], torch.zeros(n, up(heads * vdim)).cuda()
    assert A.attn_latent(qh[order.long()].contiguous(), 3, cache, acc, ml, heads=heads, cp=cp, scale=0.9, splits=splits, positions=pos, slots=slots, table=table, rows=order)
    A.latent_merge(acc, ml, 3, uv, out, heads=heads, splits=splits, cp=cp, vdim=vdim, rows=order)
    close(out[order.long(), :heads * vdim], want[order.long()], 2e-3)
    assert (out[0] == 0).all()


@pytest.mark.parametrize("rank,cache32", [(36, True), (600, True), (36, False)])
def test_absorbed_queries_and_cache_rows(ops, rank, cache32):
    K, A, R = ops
    H, d, rot, n, eps = 3, 21, 6, 6, 1e-5
    cp = up(rank, 16)
    w = up(cp + rot, 32)
    for wt in (torch.float32, torch.bfloat16):
        qkv = rnd(n, H * (d + rot) + rank + rot + 5)
        norm, uk = rnd(rank, seed=1), torch.zeros(H, d, cp, dtype=wt, device="cuda")
        uk[..., :rank] = rnd(H, d, rank, seed=2)
        freqs = torch.tensor([90.0 ** (-2 * i / rot) for i in range(rot // 2)], dtype=F64).cuda()
        pos = torch.tensor([0, 63, 64, 100, 65, 3], dtype=torch.int32).cuda()
        slots = torch.tensor([0, 0, 0, 0, 1, 1], dtype=torch.int32).cuda()
        table = torch.tensor([[3, 1], [0, 4]], dtype=torch.int32).cuda()
        for inter in (True, False):
            cache = torch.full((5, 1, 64, w), 7.0, device="cuda", dtype=torch.float32 if cache32 else torch.float16)
            q = torch.zeros(n, H, w, device="cuda", dtype=cache.dtype)
            A.latent_step(qkv, qkv[:, H * (d + rot):], n, heads=H, dim=d, rot=rot, rank=rank, norm=norm, eps=eps, freqs=freqs, interleaved=inter, positions=pos, slots=slots, table=table,
                          cache=cache, cp=cp, uk=uk, q_out=q)
            tol = 1e-5 if cache32 else 1e-3
            x = qkv.double().cpu()

            def turn(v):           # [n, heads, rot]
                if inter:
                    return O.rotate_pairs(v, pos.cpu(), 90.0)
                half = torch.cat([v[..., i::rot // 2] for i in range(rot // 2)], -1)      # (i, i + rot / 2) side by side
                y = O.rotate_pairs(half, pos.cpu(), 90.0)
                return torch.cat([y[..., 0::2], y[..., 1::2]], -1)
            qs = x[:, :H * (d + rot)].view(n, H, d + rot)
            close(q[..., :cp], torch.einsum("nhd,hdc->nhc", qs[..., :d], uk.double().cpu()), tol)
            close(q[..., cp:cp + rot], turn(qs[..., d:]), tol)
            c = x[:, H * (d + rot):H * (d + rot) + rank]
            k = x[:, None, H * (d + rot) + rank:H * (d + rot) + rank + rot]
            got = torch.stack([cache[table[s, p // 64], 0, p % 64] for s, p in zip(slots.tolist(), pos.tolist())])
            close(got[:, :rank], O.norm_plain(c, norm.double().cpu(), eps), tol)
            close(got[:, cp:cp + rot], turn(k)[:, 0], tol)
            assert (got[:, rank:cp] == 0).all() and (got[:, cp + rot:] == 0).all() and (q[..., cp + rot:] == 0).all()
            assert int((cache != 7.0).any(-1).sum()) == n                       # nothing else was written
            if not cache32:                                                     # the long form: queries as they are, the same cache rows
                again, dp, rp = torch.full_like(cache, 7.0), 24, 10
                q = torch.full((n, H, dp + rp), 9.0, device="cuda", dtype=torch.float16)
                A.latent_step(qkv, qkv[:, H * (d + rot):], n, heads=H, dim=d, rot=rot, rank=rank, norm=norm, eps=eps, freqs=freqs, interleaved=inter, positions=pos, slots=slots, table=table,
                              cache=again, cp=cp, q_out=q, dp=dp, rp=rp)
                assert torch.equal(again, cache)
                close(q[..., :d], qs[..., :d], tol)
                close(q[..., dp:dp + rot], turn(qs[..., d:]), tol)
                assert (q[..., d:dp] == 0).all() and (q[..., dp + rot:] == 0).all()


@pytest.mark.parametrize("heads,dim,rot,vdim", [(2, 20, 8, 28), (3, 128, 64, 128), (1, 64, 64, 100), (4, 100, 40, 64), (2, 64, 0, 64)])
def test_prompt_tiles_over_keys_in_two_parts(ops, heads, dim, rot, vdim):
    """Portions of two sequences, one with a past; single standing-out keys first, at tile borders and far away."""
    K, A, R = ops
    dp, rp, vp = up(dim, 64), up(rot, 64), up(vdim, 64)
    assert A.parts_supported(dp, rp, vp)
    lens = [(0, 200), (300, 131)]                                # past, new tokens
    total = sum(p + n for p, n in lens)
    kv = torch.zeros(total, heads * (dp + vp), dtype=torch.float16, device="cuda")
    k, v = kv[:, :heads * dp].view(total, heads, dp), kv[:, heads * dp:].view(total, heads, vp)
    k[..., :dim], v[..., :vdim] = 0.5 * rnd(total, heads, dim).half(), rnd(total, heads, vdim, seed=1).half()
    sh = torch.zeros(total, max(rp, 8), dtype=torch.float16, device="cuda")
    if rot:
        sh[:, :rot] = rnd(total, rot, seed=2).half()
    rows = sum(n for _, n in lens)
    q = torch.zeros(rows, heads, dp + rp, dtype=torch.float16, device="cuda")
    q[..., :dim] = 0.5 * rnd(rows, heads, dim, seed=3).half()
    if rot:
        q[..., dp:dp + rot] = 0.3 * rnd(rows, heads, rot, seed=4).half()
    q[..., 0] = 7.0
    k[..., 0] = 0.0
    base, row0, tiles = 0, 0, []
    for past, n in lens:
        for p in (0, 127, 128, 255, 256, 300, past + n - 1):
            if p < past + n:
                k[base + p, :, 0] = 7.0
        tiles += [(row0 + t, min(128, n - t), base, past + t) for t in range(0, n, 128)]
        base, row0 = base + past + n, row0 + n
    out = torch.full((rows, heads * vdim + 4), 9.0, dtype=torch.bfloat16, device="cuda")
    A.attn_prefill_parts(q, kv, sh, torch.tensor(tiles, dtype=torch.int32).cuda(), out, heads=heads, dp=dp, vp=vp, rp=rp, vdim=vdim, scale=0.8)
    base = row0 = 0
    for past, n in lens:
        T = past + n
        for h in range(heads):
            s = q[row0:row0 + n, h, :dp].double() @ k[base:base + T, h].double().t()
            if rot:
                s += q[row0:row0 + n, h, dp:].double() @ sh[base:base + T, :rp].double().t()
            s = (s * 0.8).masked_fill(torch.ones(n, T).triu(past + 1).bool().cuda(), -math.inf)
            close(out[row0:row0 + n, h * vdim:(h + 1) * vdim], torch.softmax(s, -1) @ v[base:base + T, h, :vdim].double(), 1e-2)
        base, row0 = base + T, row0 + n
    assert (out[:, heads * vdim:] == 9.0).all()


def test_wrong_shapes_are_errors(ops):
    K, A, R = ops
    x = torch.zeros(1, 8).cuda()
    with pytest.raises(K.CudaKernelError):
        R.gemv([R.seg(torch.zeros(3, 8, dtype=torch.bfloat16).cuda(), 3, torch.zeros(1, 4).cuda(), act="glu:gelu_tanh")], 8, x, 1, False)      # odd gated rows
    with pytest.raises(K.CudaKernelError):
        A.latent_merge(torch.zeros(1, 1, 2, 16).cuda(), None, 1, torch.zeros(4, 16).cuda(), torch.zeros(1, 8).cuda(), heads=1, splits=2, cp=16, vdim=4)
    q = torch.zeros(1, 2, 1024, dtype=torch.float16).cuda()
    i = torch.zeros(1, dtype=torch.int32).cuda()
    assert not A.attn_latent(q, 1, torch.zeros(1, 1, 64, 1024, dtype=torch.float16).cuda(), torch.zeros(1, 2, 1, 960).cuda(), torch.zeros(1, 2, 1, 2).cuda(), heads=2, cp=960,
                             scale=1.0, splits=1, positions=i, slots=i, table=torch.zeros(1, 1, dtype=torch.int32).cuda())
