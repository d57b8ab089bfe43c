"""Attention over heads of keys and values, and the state-space mixer with one decay per head, of stack models whose layers' parts follow one another
(engine/blocks.py)."""
from __future__ import annotations

import torch

from .. import envconfig
from ..models.stack import AttentionMixer, Mamba2Mixer
from ..ops import rows as O
from ..ops import ssd as D
from .blocks import Mat, Norm, Step, WeightSource, up


MIN_SPLIT = 128                  # keys


class HeadAttention:
    """The projections of queries, keys, values and gate are one product; with a convolution the first three go through it, and the slot keeps their last inputs.
    Interleaved rotary pairs are brought into the half-split order at load, by the order of the q and k rows, which leaves the scores as they are.  ``norm`` None: the
    layer's parts share one, and the layer calls :meth:`project` and :meth:`mix`."""

    def __init__(self, src: WeightSource, p: str, m: AttentionMixer, norm: Norm | None, f32: bool, post: Norm | None):
        w, nq, nk, nv = src.width, m.n_q, m.n_k, m.n_v
        self.m, self.norm, self.post, self.f32, self.n_out = m, norm, post, f32, m.heads * m.vdim
        self.n8 = up(nq + nk + nv)                                       # the gate starts here
        n_in = self.n8 + up(m.n_gate)
        w_in, bias, self.conv_w = src.zeros(n_in, src.wp), torch.zeros(n_in, device=src.device) if m.bias else None, None
        if m.conv:
            self.conv_w = torch.zeros(m.conv, self.n8, device=src.device)
        for at, k, name in ((0, nq, "q"), (nq, nk, "k"), (nq + nk, nv, "v")):
            if not k:
                continue
            rows = self._half_split(k, src.device) if name in "qk" else slice(None)
            w_in[at:at + k, :w] = src.tensor(f"{p}attn_{name}.weight", k, w)[rows]
            if name in m.bias:
                bias[at:at + k] = src.tensor(f"{p}attn_{name}.bias", k).float()[rows]
            if m.conv:
                self.conv_w[:, at:at + k] = src.tensor(f"{p}attn_{name}_conv1d.weight", k, m.conv).float()[rows].t()
        if m.n_gate:
            w_in[self.n8:self.n8 + m.n_gate, :w] = src.tensor(p + "attn_gate.weight", m.n_gate, w)
        self.w_in = Mat(w_in, bias)
        self.w_o = Mat(src.pack([(0, 0, p + "attn_output.weight", (w, m.heads * m.vdim))], src.wp, up(m.heads * m.vdim)))
        self.q_norm = self.k_norm = None
        if m.qk_norm:
            n = (nq, nk) if m.qk_norm == "row" else (m.dim, m.dim)
            self.q_norm, self.k_norm = src.vec(p + "attn_q_norm.weight", n[0]), src.vec(p + "attn_k_norm.weight", n[1])
        self.v_off = nq if m.keys_as_values else nq + nk
        self.diff = O.NO_DIFF
        if m.maps > 1:
            dots = [(src.tensor(f"{p}attn_lambda_q{i}.weight", m.dim).double() * src.tensor(f"{p}attn_lambda_k{i}.weight", m.dim).double()).sum() for i in (1, 2)]
            self.diff = O.DiffHeads(float(dots[0].exp() - dots[1].exp()) + m.diff, 1.0 - m.diff, src.eps, 1)
        self.n_rot, self.magnitude = (m.rot.dims, m.rot.magnitude) if m.rot else (0, 1.0)
        self.freqs = torch.tensor(m.rot.freqs() if m.rot else [0.0], dtype=torch.float64, device=src.device)
        # the tensor-core kernels take cache rows of 64 or 128 f16 values
        big = max(m.maps * m.dim, m.vdim)
        self.hd = 0 if f32 or big > 128 else 64 if big <= 64 else 128
        self.dk, self.dv = (self.hd, self.hd) if self.hd else (up(m.maps * m.dim), up(m.vdim))

    def _half_split(self, n: int, device) -> torch.Tensor | slice:
        """Order of the rows of an [n, ...] q or k projection in which pairs (2i, 2i + 1) of a map stand dims / 2 apart."""
        m = self.m
        if m.rot is None or not m.rot.interleaved:
            return slice(None)
        one = [*range(0, m.rot.dims, 2), *range(1, m.rot.dims, 2), *range(m.rot.dims, m.dim)]
        return (torch.arange(0, n, m.dim)[:, None] + torch.tensor(one)[None]).reshape(-1).to(device)

    def product_weights(self) -> tuple[int, int, float]:
        return self.w_in.w.numel() + self.w_o.w.numel(), 0, 0.0

    def make_cache(self, cache, kv: tuple[torch.Tensor, ...] | None = None) -> tuple[torch.Tensor, ...]:
        """``kv``: the memory of the layer run whose keys and values are used."""
        ty = torch.float32 if self.f32 else torch.float16
        mem = (cache.add_pages(self.m.kv_heads, self.dk, ty), cache.add_pages(self.m.kv_heads, self.dv, ty)) if kv is None else kv[:2]
        return mem if self.conv_w is None else (*mem, cache.add_state(max(self.m.conv - 1, 1), self.n8))

    def splits(self, nb: int, n_ctx: int, sms: int) -> tuple[int, int]:
        """(parts of the keys for a decode step of ``nb`` sequences, most keys a query sees)."""
        keys = min(n_ctx, self.m.chunk or (self.m.window + self.m.keep + 128 if self.m.window else n_ctx))
        room = sms // (self.m.kv_heads * nb)          # shorter parts than usual as long as SMs would stand idle
        return max(1, min(envconfig.attn_splits(), max(keys // envconfig.attn_split_len(), min(keys // MIN_SPLIT, room)))), keys

    def run(self, s: Step, mem: tuple[torch.Tensor, ...]) -> None:
        h = s.rows(self.norm)
        out = s.buf("mix", self.w_o.w.shape[1], zero=True)
        self.mix(s, self.project(s, h, mem), mem, out)
        s.result(out, self.w_o, self.post)

    def project(self, s: Step, h: torch.Tensor, mem: tuple[torch.Tensor, ...], **beside) -> tuple[torch.Tensor, torch.Tensor]:
        """(projections, the same behind their convolution); ``beside``: see Step.enter."""
        proj = s.buf("in", self.w_in.w.shape[0], torch.float32)
        if self.conv_w is None:
            s.enter(h, self.w_in, proj, **beside)
            return proj, proj
        u, conv = s.buf("u", self.n8, torch.float32), (self.conv_w, None, mem[2])
        if s.small:                           # the convolution follows in the product's epilogue
            s.enter(h, self.w_in, proj, conv=conv, conv_out=u, conv_silu=False, conv_shift=True, **beside)
            return proj, u
        s.enter(h, self.w_in, proj, **beside)
        O.ssm_conv(proj, self.n8, *conv, s.m.slots, s.m.positions, s.m.offs, u, silu=False, shift=s.decode, pdl=s.pdl)
        if not s.decode:
            O.conv_keep(proj, self.n8, self.m.conv, mem[2], s.m.segs)
        s.launched(1 + (not s.decode))
        return proj, u

    def mix(self, s: Step, projected: tuple[torch.Tensor, torch.Tensor], mem: tuple[torch.Tensor, ...], out: torch.Tensor) -> None:
        proj, qkv = projected
        self._attend(s, qkv, O.head_gate(proj[:, self.n8:], self.m.gate) if self.m.gate else O.NO_GATE, mem[0], mem[1], out)

    def _attend(self, s: Step, qkv, gate, kc, vc, out) -> None:
        m, be, nb, dev = self.m, s.be, s.nb, qkv.device
        table, at = be.cache.table, {"positions": s.m.positions, "slots": s.m.slots}
        heads, diff = m.maps * m.heads, self.diff         # heads of the kernels
        prep = dict(heads=heads, maps=m.maps, append=m.kv_from is None, dim=m.dim, vdim=m.vdim, q_norm=self.q_norm, k_norm=self.k_norm, eps=be.stack.eps, freqs=self.freqs, n_rot=self.n_rot,
                    head_norm=m.qk_norm == "head", v_off=self.v_off, mscale=self.magnitude, pdl=s.pdl)
        mask = dict(scale=m.scale, softcap=m.softcap, chunk=m.chunk, window=m.window, keep=m.keep, gate=gate)
        s.launched(2)
        if s.decode and self.hd:
            n, keys = self.splits(nb, be.n_ctx, be.sms)
            acc, ml = torch.empty(nb, heads, n, self.hd, device=dev), torch.empty(nb, heads, n, 2, device=dev)
            if O.attn_decode_paged(qkv, kc, vc, table=table, out=out, nb=nb, n_splits=n, n_ctx=keys, part_acc=acc, part_ml=ml, diff=diff, **at, **prep, **mask):
                return
        q = s.buf("q", heads * (self.hd or m.maps * m.dim), torch.float32).view(nb, heads, -1)
        O.paged_append(qkv, kv_heads=m.kv_heads, table=table, q_out=q, k_cache=kc, v_cache=vc, **at, **prep)
        if self.hd and s.m.tiles is not None:
            O.attn_prefill_paged(q, kc, vc, s.m.half_tiles if diff.on else s.m.tiles, table, out, vdim=m.vdim, diff=diff, **mask)
            return
        res = s.buf("maps", heads * m.vdim, torch.float32) if diff.on else out
        O.paged_attn(q, kc, vc, table=table, out=res, dim=m.maps * m.dim, vdim=m.vdim, pdl=s.pdl, **at, **mask)
        if diff.on:
            O.diff_rows(res, m.heads, m.vdim, diff, out, pdl=s.pdl)
            s.launched()


class StateSpaceHeads:
    """Mamba-2.  Heads, and the B and C of a group, are padded with zero columns so that the kernels read whole vectors: the input product's rows, the convolution's
    channels, the norm and the output product's columns are laid out that way at load."""

    def __init__(self, src: WeightSource, p: str, m: Mamba2Mixer, norm: Norm, f32: bool, post: Norm | None):
        w, H, G, P, N = src.width, m.heads, m.groups, m.vdim, m.state
        self.m, self.norm, self.post = m, norm, post
        self.vp, self.np = up(P), up(N, 16)
        if self.np > D.MAX_STATE:
            raise NotImplementedError(f"{N} state dimensions")
        self.inner, bc = H * self.vp, G * self.np
        self.off_b, self.off_c, self.ch = self.inner, self.inner + bc, self.inner + 2 * bc

        def heads(t: torch.Tensor, n: int, size: int, padded: int) -> torch.Tensor:
            """[n * size, ...] -> [n * padded, ...] with zeros behind every ``size``."""
            out = torch.zeros(n, padded, *t.shape[1:], device=t.device, dtype=t.dtype)
            out[:, :size] = t.view(n, size, *t.shape[1:])
            return out.view(n * padded, *t.shape[1:])

        def channels(t: torch.Tensor) -> torch.Tensor:
            x, b, c = torch.split(t, [m.inner, G * N, G * N])
            return torch.cat([heads(x, H, P, self.vp), heads(b, G, N, self.np), heads(c, G, N, self.np)])

        z, xbc, dt = torch.split(src.tensor(p + "ssm_in.weight", m.inner + m.channels + H, w), [m.inner, m.channels, H])
        n_in = self.inner + self.ch
        w_in = src.zeros(n_in + up(H), src.wp)                           # z | x B C | step sizes
        w_in[:self.inner, :w], w_in[self.inner:n_in, :w], w_in[n_in:n_in + H, :w] = heads(z, H, P, self.vp), channels(xbc), dt
        self.w_all, self.w_in, self.w_dt = w_in, Mat(w_in[:n_in]), Mat(w_in[n_in:])
        self.conv_w = channels(src.tensor(p + "ssm_conv1d.weight", m.channels, m.conv).float()).t().contiguous()
        self.conv_b = channels(src.tensor(p + "ssm_conv1d.bias", m.channels).float())
        self.dt_bias, self.a, self.d = src.vec(p + "ssm_dt.bias", H), src.vec(p + "ssm_a", H), src.vec(p + "ssm_d", H)
        self.g = heads(src.tensor(p + "ssm_norm.weight", m.inner).float(), H, P, self.vp)
        w_o = src.zeros(src.wp, self.inner)
        w_o[:w] = heads(src.tensor(p + "ssm_out.weight", w, m.inner).t(), H, P, self.vp).t()
        self.w_o = Mat(w_o)

    def product_weights(self) -> tuple[int, int, float]:
        return sum(a.w.numel() for a in (self.w_in, self.w_dt, self.w_o)), 0, 0.0

    def make_cache(self, cache) -> tuple[torch.Tensor, torch.Tensor]:
        return cache.add_state(self.m.heads, self.vp, self.np), cache.add_state(max(self.m.conv - 1, 1), self.ch)

    def run(self, s: Step, mem: tuple[torch.Tensor, torch.Tensor]) -> None:
        (state, conv_state), m, be, f32 = mem, self.m, s.be, torch.float32
        zx = s.buf("zx", self.w_in.w.shape[0])
        z, xbc, u, dt = zx[:, :self.inner], zx[:, self.inner:], s.buf("xbc", self.ch), s.buf("dt", self.w_dt.w.shape[0], f32)
        conv, h = (self.conv_w, self.conv_b, conv_state), s.rows(self.norm)
        if s.small:                           # the convolution follows in the product's epilogue
            w = self.w_in.w
            O.gemv([O.seg(w[self.inner:], self.ch, xbc), O.seg(w, self.inner, z), O.seg(self.w_dt.w, dt.shape[1], dt)], be.wp, h, s.nb, be.f32, conv=conv, conv_out=u,
                   conv_shift=True, slots=s.m.slots, positions=s.m.positions, pdl=s.pdl)
            s.launched()
        else:
            if be.f32:
                s.product(h, self.w_in, zx)
                s.product(h, self.w_dt, dt)
            else:
                O.gemm(h, self.w_all, zx, tail=dt)
                s.launched()
            O.ssm_conv(xbc, self.ch, *conv, s.m.slots, s.m.positions, s.m.offs, u, shift=s.decode, pdl=s.pdl)
            if not s.decode:
                O.conv_keep(xbc, self.ch, m.conv, conv_state, s.m.segs)
            s.launched(1 + (not s.decode))
        out = s.buf("mix", self.inner, zero=True)
        args = (u, self.off_b, self.off_c, z, dt, self.dt_bias, self.a, self.d, m.groups, state)
        if s.decode:
            D.ssd_step(*args, s.m.slots, s.m.positions, out, pdl=s.pdl)
        else:
            D.ssd_scan(*args, s.m.segs, out, pdl=s.pdl)
        s.launched()
        if s.small and m.norm_groups == 1 and self.post is not None:        # one root mean square per row: the product applies it to its results
            y = s.buf("y", be.wp, f32)
            O.gemv([O.seg(self.w_o.w, be.wp, y, self.g)], self.inner, out, s.nb, be.f32, O.SRC_NORM, be.stack.eps, m.inner, pdl=s.pdl)
            s.leave(y, self.post)
        else:
            D.group_norm(out, m.heads, m.vdim, self.vp, m.norm_groups, self.g, be.stack.eps, pdl=s.pdl)
            s.result(out, self.w_o, self.post)
        s.launched()
