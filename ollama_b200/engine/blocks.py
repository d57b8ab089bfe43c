"""Parts of stack models' layers that run one after the other (engine/stack.py): latent attention, gated and mixture-of-experts feed-forwards,
inputs of a layer's own per token.  Further mixers are in engine/mixers.py.

Each class holds a layer's weights, laid out for the kernels, and adds its result to the residual rows of a :class:`Step`.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from ..models.stack import DenseMLP, Expert, ExpertMLP, GruMixer, LatentMixer
from ..ops import cuda as K
from ..ops import latent as A
from ..ops.cuda import ExpertGroups
from ..ops import rows as O
from .cache import PAGE

LONG_PORTION = 64                # prompt portions of this many tokens multiply keys and values out; shorter ones stay in the latent space
MAX_SPLITS = 128
MERGE_ROWS = 6                   # more rows than this merge their splits and multiply the values in two launches


def up(n: int, m: int = 8) -> int:
    return -(-n // m) * m


class WeightSource:
    """Named tensors of a model as zero-padded matrices and vectors on the device."""

    def __init__(self, get, device, act_dtype, width: int, eps: float = 0.0):
        self._get, self.device, self.act_dtype, self.width, self.wp, self.eps = get, device, act_dtype, width, up(width), eps

    def tensor(self, name: str, *shape: int) -> torch.Tensor:
        t = self._get(name)
        if tuple(t.shape) != tuple(shape):
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {tuple(shape)}")
        return t

    def vec(self, name: str, n: int) -> torch.Tensor:
        t = torch.zeros(up(n), device=self.device)
        v = self._get(name).float()
        if v.numel() != n:
            raise ValueError(f"{name}: {v.numel()} values, expected {n}")
        t[:n] = v.reshape(-1)
        return t

    def zeros(self, *shape: int) -> torch.Tensor:
        return torch.zeros(*shape, device=self.device, dtype=self.act_dtype)

    def pack(self, parts, n_rows: int, cols: int) -> torch.Tensor:
        """[n_rows, cols] in the compute type; ``parts``: (row, column, name, shape)."""
        w = self.zeros(n_rows, cols)
        for r0, c0, name, shape in parts:
            w[r0:r0 + shape[0], c0:c0 + shape[1]] = self.tensor(name, *shape)
        return w

    def gate_up(self, gate: str, up_name: str, ff: int, lead: tuple[int, ...] = ()) -> torch.Tensor:
        """[..., 2 * padded ff, wp]: rows 2i and 2i + 1 are gate and up of column i."""
        w = self.zeros(*lead, 2 * up(ff), self.wp)
        w[..., 0:2 * ff:2, :self.width] = self.tensor(gate, *lead, ff, self.width)
        w[..., 1:2 * ff:2, :self.width] = self.tensor(up_name, *lead, ff, self.width)
        return w


@dataclass
class Norm:
    """Layer norm, or without a bias an RMS norm."""
    g: torch.Tensor
    b: torch.Tensor | None


@dataclass
class Mat:
    """Matrix of a product; ``rs`` and ``rc`` fold a layer norm before it in (see kernels/gemv_rows.cu)."""
    w: torch.Tensor
    bias: torch.Tensor | None = None
    rs: torch.Tensor | None = None
    rc: torch.Tensor | None = None

    def fold(self, norm: Norm) -> "Mat":
        w = self.w.float()
        self.rs, self.rc = w @ norm.g, w @ norm.b
        if self.bias is not None:
            self.rc += self.bias
        return self


def make_norm(src: WeightSource, name: str, kind: str = "layer") -> Norm:
    return Norm(src.vec(name + ".weight", src.width), src.vec(name + ".bias", src.width) if kind == "layer" else None)


@dataclass
class LongPortions:
    """Rows of a step whose keys and values are multiplied out: query tiles, the sequences' places in the scratch buffer, and the other rows.  Under a window the
    buffer begins with a sequence's first visible position, so that the row of position 0 may be negative."""
    tiles: torch.Tensor               # [n, 4]: first row, rows, buffer row of the sequence's position 0, position
    seqs: torch.Tensor                # [n, 4]: buffer row of position 0, end of the positions, slot, first position
    total: int
    longest: int                      # positions of one sequence in the buffer
    rest: torch.Tensor | None         # step rows that stay in the latent space


class Step:
    """The rows of one step on their way through the layers.

    A layer may leave an update of the residual ``pending`` (a normalised branch, the vectors that join a pass of a loop); the next norm
    applies it in its own pass over the rows.
    """

    def __init__(self, be, B, m, x: torch.Tensor, x0: torch.Tensor | None, decode: bool, hist: torch.Tensor | None = None):
        self.be, self.B, self.m, self.x, self.x0, self.decode = be, B, m, x, x0, decode
        self.hist = hist                               # [blocks, rows, columns]: embedding output and layer results, where layers read an average of them
        self.nb = x.shape[0]
        self.small = decode and self.nb <= be.gemv_rows
        self.folded = self.small and not be.f32        # norms inside the products; 32-bit models form them first
        self.act = torch.float32 if self.small else be.act_dtype
        self.pdl = be.pdl and decode
        self.pending: dict = {}
        self.copy = None                               # bf16 copy of the rows, made by the last product before a per-token input
        self.last = False                              # the block that runs is a layer's last before its per-token input

    def buf(self, name: str, cols: int, dtype=None, zero: bool = False) -> torch.Tensor:
        return self.B.get(name, cols, dtype or self.act, self.nb, zero)

    def launched(self, n: int = 1) -> None:
        self.be._n += n

    def flush(self) -> None:
        if self.pending:
            O.norm_rows(self.x, self.be.stack.width, self.be.stack.eps, None, None, pdl=self.pdl, **self.pending)
            self.pending = {}
            self.launched()

    def average(self, n: int, w: torch.Tensor, norm: Norm | None) -> torch.Tensor | None:
        """The stream becomes the sum of the first ``n`` blocks of the history with weights ``w`` (and block ``n``, which the layer adds to); returns its norm."""
        h = self.buf("h", self.be.wp) if norm is not None else None
        g, b = (norm.g, norm.b) if norm is not None else (None, None)
        self.x = O.depth_rows(self.hist, n, w, self.be.stack.width, self.be.stack.eps, g, b, h, pdl=self.pdl)
        self.launched()
        return h

    def enter(self, h: torch.Tensor, mat: Mat, out: torch.Tensor, segs=(), joined: Mat | None = None, tail: torch.Tensor | None = None, **conv) -> None:
        """out = mat h + bias.  Beside it, in the same launch: the products ``segs`` for a few rows, for many rows the last columns of ``joined``, which begins with
        ``mat``, as fp32 rows ``tail``."""
        if self.small:
            O.gemv([O.seg(mat.w, out.shape[1], out, rc=mat.bias), *segs], mat.w.shape[1], h, self.nb, self.be.f32, slots=self.m.slots, positions=self.m.positions,
                   pdl=self.pdl, **conv)
        else:
            m = joined or mat
            O.gemm(h, m.w, out, bias=m.bias, tail=tail)
        self.launched()

    def product(self, h: torch.Tensor, mat: Mat, out: torch.Tensor, **kw) -> None:
        """out (+)= f(mat h + bias) [times the tokens' rows of a table ``mul``]."""
        if self.small:
            O.gemv([O.seg(mat.w, mat.w.shape[0], out, rc=mat.bias, **kw)], mat.w.shape[1], h, self.nb, self.be.f32, mul_row=self.m.tokens, pdl=self.pdl)
        else:
            O.gemm(h, mat.w, out, bias=mat.bias, mul_row=self.m.tokens, **kw)
        self.launched()

    def add(self, h: torch.Tensor, mat: Mat) -> None:
        """x += residual multiplier * mat h."""
        kw = {}
        if self.last and not self.small and self.act == torch.bfloat16:
            kw["copy"] = self.copy = self.buf("copy", self.be.wp)
        self.product(h, mat, self.x, accumulate=True, alpha=self.be.stack.residual_mult, **kw)

    def rows(self, norm: Norm) -> torch.Tensor:
        """norm(x), after what is pending."""
        h = self.buf("h", self.be.wp)
        O.norm_rows(self.x, self.be.stack.width, self.be.stack.eps, norm.g, h, b1=norm.b, pdl=self.pdl, **self.pending)
        self.pending = {}
        self.launched()
        return h

    def result(self, h: torch.Tensor, mat: Mat, post: Norm | None) -> None:
        """Adds mat h to the stream, under the norm ``post`` where there is one."""
        if post is None:
            self.add(h, mat)
            return
        y = self.buf("y", self.be.wp, torch.float32)
        self.product(h, mat, y)
        self.leave(y, post)

    def leave(self, y: torch.Tensor, post: Norm) -> None:
        self.pending = {"y": y, "wy": post.g, "mult": self.be.stack.residual_mult}

    def normed(self, norm: Norm, mat: Mat, out: torch.Tensor, keep: bool = False, **kw) -> torch.Tensor | None:
        """out = f(mat norm(x) + bias); returns the normalised rows where they exist (always with ``keep``)."""
        be, st = self.be, self.be.stack
        if self.folded and norm.b is not None:
            h = self.buf("h", be.wp) if keep else None
            self.flush()
            O.gemv([O.seg(mat.w, mat.w.shape[0], out, norm.g, rs=mat.rs, rc=mat.rc, **kw)], be.wp, self.x, self.nb, False, O.SRC_LAYER, st.eps, st.width, h=h,
                   hb=norm.b, pdl=self.pdl)
            self.launched()
            return h
        h = self.rows(norm)
        self.product(h, mat, out, **kw)
        return h


class LatentAttention:
    """The input product gives queries, latent and rotated key part; with a latent of the queries' own the queries follow in a product of their own.  ``norm`` None: the
    layer's parts share one, and the layer calls :meth:`project` and :meth:`mix`."""

    def __init__(self, src: WeightSource, p: str, m: LatentMixer, norm: Norm | None, f32: bool):
        H, w = m.heads, src.width
        self.m, self.norm, self.f32, self.n_out = m, norm, f32, H * m.vdim
        nq = H * (m.dim + m.rot_dim)
        self.w_uq = self.q_norm = None
        if m.q_rank:
            self.off_c, name = up(m.q_rank), "attn_q_a"
            self.q_norm = src.vec(p + "attn_q_a_norm.weight", m.q_rank)
            self.w_uq = Mat(src.pack([(0, 0, p + "attn_q_b.weight", (nq, m.q_rank))], up(nq), self.off_c))
        else:
            self.off_c, name = nq, "attn_q"
        n_in = self.off_c + m.kv_rank + m.rot_dim
        self.w_in = Mat(src.pack([(0, 0, f"{p}{name}.weight", (m.q_rank or nq, w)), (self.off_c, 0, p + "attn_kv_a_mqa.weight", (m.kv_rank + m.rot_dim, w))], up(n_in), src.wp))
        self.w_o = Mat(src.pack([(0, 0, p + "attn_output.weight", (w, H * m.vdim))], src.wp, up(H * m.vdim)))
        self.c_norm = src.vec(p + "attn_kv_a_norm.weight", m.kv_rank)
        self.cp = up(m.kv_rank, 16)
        self.row = up(self.cp + m.rot_dim, 32)           # values of a cache row
        # the tensor-core kernel takes latents of up to 512 values in f16; wider ones and 32-bit models keep an fp32 cache
        self.cache_type = torch.float32 if f32 or self.cp > 512 or self.row > 640 else torch.float16
        uk, uv = src.tensor(p + "attn_k_b.weight", H * m.dim, m.kv_rank), src.tensor(p + "attn_v_b.weight", H * m.vdim, m.kv_rank)
        self.uk, self.uv = src.zeros(H, m.dim, self.cp), src.zeros(H * m.vdim, self.cp)
        self.uk[..., :m.kv_rank] = uk.view(H, m.dim, m.kv_rank)
        self.uv[:, :m.kv_rank] = uv
        self.freqs = torch.tensor(m.rot.freqs() if m.rot else [0.0], dtype=torch.float64, device=src.device)
        self.interleaved, self.magnitude = (m.rot.interleaved, m.rot.magnitude) if m.rot else (False, 1.0)
        self.dp, self.rp, self.vp = up(m.dim, 64), up(m.rot_dim, 64), up(m.vdim, 64)
        self.w_kv = None
        if self.cache_type == torch.float16 and A.parts_supported(self.dp, self.rp, self.vp):
            self.w_kv = src.zeros(H * (self.dp + self.vp), self.cp)      # rows: every head's keys, then every head's values
            self.w_kv[:H * self.dp].view(H, self.dp, self.cp)[:, :m.dim] = self.uk
            self.w_kv[H * self.dp:].view(H, self.vp, self.cp)[:, :m.vdim] = self.uv.view(H, m.vdim, self.cp)
        if not f32 and norm is not None:
            self.w_in.fold(norm)

    def product_weights(self) -> tuple[int, int, float]:
        return sum(t.numel() for t in (self.w_in.w, self.uk, self.uv, self.w_o.w, *((self.w_uq.w,) if self.w_uq else ()))), 0, 0.0

    def make_cache(self, cache) -> tuple[torch.Tensor]:
        return (cache.add_pages(1, self.row, self.cache_type),)

    def run(self, s: Step, mem: tuple[torch.Tensor]) -> None:
        qkv = s.buf("in", self.w_in.w.shape[0], torch.float32)
        s.normed(self.norm, self.w_in, qkv)
        out = s.buf("mix", self.w_o.w.shape[1], zero=True)
        self.mix(s, qkv, mem, out)
        s.add(out, self.w_o)

    def project(self, s: Step, h: torch.Tensor, mem, **beside) -> torch.Tensor:
        proj = s.buf("in", self.w_in.w.shape[0], torch.float32)
        s.enter(h, self.w_in, proj, **beside)
        return proj

    def mix(self, s: Step, proj: torch.Tensor, mem: tuple[torch.Tensor], out: torch.Tensor) -> None:
        (cache,), lp = mem, (s.m.long or {}).get(self.m.window)
        qc = (self._queries(s, proj), proj[:, self.off_c:])
        if lp is None or self.w_kv is None or s.decode:
            self._latent(s, qc, cache, out, s.nb, None, True)
        else:
            self._long(s, qc, cache, out, lp)
            if lp.rest is not None:
                self._latent(s, qc, cache, out, lp.rest.numel(), lp.rest, False)

    def _queries(self, s: Step, proj: torch.Tensor) -> torch.Tensor:
        m, eps = self.m, s.be.stack.eps
        if self.w_uq is None:
            return proj
        n, w = self.off_c, self.w_uq.w
        q = s.buf("latent_q", w.shape[0], torch.float32)
        if s.small:
            O.gemv([O.seg(w, q.shape[1], q, self.q_norm)], n, proj, s.nb, s.be.f32, O.SRC_NORM, eps, m.q_rank, pdl=s.pdl)
        else:
            c = s.buf("latent_cq", n)
            O.norm_rows(proj, m.q_rank, eps, self.q_norm, c, pdl=s.pdl)
            O.gemm(c, w, q)
            s.launched()
        s.launched()
        return q

    def _step_args(self, s: Step) -> dict:
        m = self.m
        return dict(heads=m.heads, dim=m.dim, rot=m.rot_dim, rank=m.kv_rank, norm=self.c_norm, eps=s.be.stack.eps, freqs=self.freqs, interleaved=self.interleaved,
                    positions=s.m.positions, slots=s.m.slots, table=s.be.cache.table, cp=self.cp, mscale=self.magnitude, pdl=s.pdl)

    def splits(self, n: int, n_ctx: int, sms: int) -> int:
        """Parts of the keys for ``n`` queries: as many CTAs as are resident (wide rows: one per SM), none shorter than a page."""
        groups = -(-self.m.heads // (16 if self.m.heads <= 16 else 32))
        keys = min(n_ctx, self.m.window + PAGE - 1) if self.m.window else n_ctx
        return max(1, min(-(-keys // PAGE), (1 if self.row > 256 else 2) * sms // (groups * n), MAX_SPLITS))

    def _latent(self, s: Step, qc, cache, out, n: int, rows, append: bool) -> None:
        """Attention of ``n`` rows in the latent space."""
        m, dev, table = self.m, out.device, s.be.cache.table
        q = torch.empty(n, m.heads, self.row, device=dev, dtype=cache.dtype)
        A.latent_step(*qc, n, cache=cache, rows=rows, append=append, uk=self.uk, q_out=q, **self._step_args(s))
        at = dict(positions=s.m.positions, slots=s.m.slots, table=table, window=m.window, pdl=s.pdl)
        splits, ml = self.splits(n, s.be.n_ctx, s.be.sms), None
        if cache.dtype == torch.float16:
            acc, ml = torch.empty(n, m.heads, splits, self.cp, device=dev), torch.empty(n, m.heads, splits, 2, device=dev)
            if not A.attn_latent(q, n, cache, acc, ml, heads=m.heads, cp=self.cp, scale=m.scale, splits=splits, rows=rows, **at):
                raise ValueError(f"latent attention of {m.heads} heads on rows of {self.row}")
        else:
            splits, acc = 1, torch.empty(n, m.heads * self.cp, device=dev)
            O.paged_attn(q, cache, cache, dim=self.row, vdim=self.cp, scale=m.scale, out=acc, **at)
        merged = torch.empty(n, m.heads, self.cp, device=dev, dtype=torch.bfloat16) if ml is not None and n > MERGE_ROWS and self.uv.dtype == torch.bfloat16 else None
        A.latent_merge(acc, ml, n, self.uv, out, heads=m.heads, splits=splits, cp=self.cp, vdim=m.vdim, rows=rows, merged=merged, pdl=s.pdl)
        s.launched(3 + (merged is not None))

    def _long(self, s: Step, qc, cache, out, lp: LongPortions) -> None:
        """Attention of the query tiles of ``lp`` over keys and values multiplied out of the latents; cache rows of the whole step."""
        m, dev, H = self.m, out.device, self.m.heads
        q = torch.empty(s.nb, H, self.dp + self.rp, device=dev, dtype=torch.float16)
        A.latent_step(*qc, s.nb, cache=cache, q_out=q, dp=self.dp, rp=self.rp, **self._step_args(s))
        c = torch.empty(lp.total, self.cp, device=dev, dtype=torch.bfloat16)
        r = torch.empty(lp.total, max(self.rp, 8), device=dev, dtype=torch.float16)
        A.latent_gather(cache, self.cp, m.rot_dim, lp.seqs, lp.longest, s.be.cache.table, c, r)
        kv = torch.empty(lp.total, self.w_kv.shape[0], device=dev, dtype=torch.float16)
        O.gemm(c, self.w_kv, kv)
        A.attn_prefill_parts(q, kv, r, lp.tiles, out, heads=H, dp=self.dp, vp=self.vp, rp=self.rp, vdim=m.vdim, scale=m.scale, window=m.window)
        s.launched(4)


class GatedRecurrence:
    """Channels padded to whole vectors; the input product's rows are update gate, candidate and output gate."""

    def __init__(self, src: WeightSource, p: str, m: GruMixer, f32: bool):
        n, w, wp = m.width, src.width, up(m.width)
        self.m, self.wp, self.f32, self.n_out = m, wp, f32, wp
        bias = torch.zeros(3 * wp, device=src.device)
        bias[:n], bias[wp:wp + n] = src.vec(p + "gru_z.bias", n)[:n], src.vec(p + "gru_x.bias", n)[:n]
        self.w_in = Mat(src.pack([(i * wp, 0, f"{p}gru_{name}.weight", (n, w)) for i, name in enumerate(("z", "x", "gate"))], 3 * wp, src.wp), bias)
        self.w_o = Mat(src.pack([(0, 0, p + "gru_out.weight", (w, n))], src.wp, wp))

    def product_weights(self) -> tuple[int, int, float]:
        return self.w_in.w.numel() + self.w_o.w.numel(), 0, 0.0

    def make_cache(self, cache) -> tuple[torch.Tensor]:
        return (cache.add_state(self.wp),)

    def project(self, s: Step, h: torch.Tensor, mem, **beside) -> torch.Tensor:
        proj = s.buf("gru", 3 * self.wp)
        s.enter(h, self.w_in, proj, **beside)
        return proj

    def mix(self, s: Step, proj: torch.Tensor, mem: tuple[torch.Tensor], out: torch.Tensor) -> None:
        if s.decode:
            O.gru_step(proj, self.wp, mem[0], s.m.slots, s.m.positions, out, self.f32, pdl=s.pdl)
        else:
            O.gru_scan(proj, self.wp, mem[0], s.m.segs, s.m.longest, out)
        s.launched()


class DenseFFN:
    """Two matrices with an activation of single values between them, which may have two numbers of the layer's own."""

    def __init__(self, src: WeightSource, p: str, m: DenseMLP):
        self.act, self.ffp, self.nums = m.act, up(m.ff), O.NO_NUMS
        if m.act == "xielu":
            a, b = torch.nn.functional.softplus(src.tensor(p + "ffn_act.weight", 2).double()).tolist()
            self.nums = (a, 0.5 + b)
        self.up = Mat(src.pack([(0, 0, p + "ffn_up.weight", (m.ff, src.width))], self.ffp, src.wp))
        self.down = Mat(src.pack([(0, 0, p + "ffn_down.weight", (src.width, m.ff))], src.wp, self.ffp))

    def product_weights(self) -> tuple[int, int, float]:
        return self.up.w.numel() + self.down.w.numel(), 0, 0.0


class GatedFFN:
    def __init__(self, src: WeightSource, p: str, m: DenseMLP, norm: Norm, f32: bool, names=("ffn_gate", "ffn_up", "ffn_down")):
        gate, up_name, down = (p + n + ".weight" for n in names)
        self.norm, self.act, self.ffp = norm, "glu:" + m.act, up(m.ff)
        self.w_gu = Mat(src.gate_up(gate, up_name, m.ff))
        self.w_down = Mat(src.pack([(0, 0, down, (src.width, m.ff))], src.wp, self.ffp))
        if not f32:
            self.w_gu.fold(norm)

    def product_weights(self) -> tuple[int, int, float]:
        return self.w_gu.w.numel() + self.w_down.w.numel(), 0, 0.0

    def run(self, s: Step) -> None:
        f = s.buf("ff", self.ffp, zero=True)
        s.normed(self.norm, self.w_gu, f, act=self.act)
        s.add(f, self.w_down)


@dataclass
class _Shared:
    e: Expert
    gu: Mat
    down: Mat
    gu_router: Mat


class ExpertFFN:
    """Mixture of experts; the experts stand stacked in one matrix each for gate / up and down.  The router's last row is the shared expert's gate where it has one."""

    def __init__(self, src: WeightSource, p: str, m: ExpertMLP, norm: Norm | None, f32: bool, post: Norm | None = None):
        w, E, n = src.width, m.experts, m.outputs
        self.groups = ExpertGroups(m.groups, m.keep, m.scale) if m.scoring == "sigmoid" else A.NO_GROUPS
        self.m, self.norm, self.post, self.ffp, self.act = m, norm, post, up(m.expert.ff), "glu:" + m.act
        parts = [(0, 0, p + "ffn_gate_inp.weight", (n, w))]
        if m.shared is not None and m.shared_gate:
            parts.append((n, 0, p + "ffn_gate_inp_shexp.weight", (1, w)))
        router, bias = src.pack(parts, up(n + len(parts) - 1), src.wp), src.vec(p + "ffn_gate_inp.bias", E) if m.router_bias else None
        self.correction = src.vec(p + "exp_probs_b.bias", n) if m.correction else None
        self.gu = src.gate_up(p + "ffn_gate_exps.weight", p + "ffn_up_exps.weight", m.expert.ff, (E,))
        self.down = src.zeros(E, src.wp, self.ffp)
        self.down[:, :w, :m.expert.ff] = src.tensor(p + "ffn_down_exps.weight", E, w, m.expert.ff)
        self.shared = None
        if m.shared is not None:              # its gate / up and the router stand below one another: one product of many rows gives both
            ff = m.shared.ff
            gu = torch.cat([src.gate_up(p + "ffn_gate_shexp.weight", p + "ffn_up_shexp.weight", ff), router])
            n_gu = 2 * up(ff)
            router = gu[n_gu:]
            both = Mat(gu, torch.cat([torch.zeros(n_gu, device=src.device), bias]) if bias is not None else None)
            self.shared = _Shared(m.shared, Mat(gu[:n_gu]), Mat(src.pack([(0, 0, p + "ffn_down_shexp.weight", (w, ff))], src.wp, up(ff))), both)
        self.router = Mat(router, bias)
        if not f32 and norm is not None and norm.b is not None:
            self.router.fold(norm)

    def product_weights(self) -> tuple[int, int, float]:
        sh = self.shared
        return (self.router.w.numel() + (sh.gu.w.numel() + sh.down.w.numel() if sh else 0), self.gu.numel() + self.down.numel(), self.m.top / self.m.outputs)

    def run(self, s: Step) -> None:
        m, sh, fs = self.m, self.shared, None
        z = s.buf("router", self.router.w.shape[0], torch.float32)
        both = sh is not None and not s.small and s.act == torch.bfloat16
        if both:
            h, fs = s.rows(self.norm), s.buf("shared", up(sh.e.ff), zero=True)
            O.gemm(h, sh.gu_router.w, fs, act=self.act, limit=sh.e.limit, bias=sh.gu_router.bias, tail=z)
            s.launched()
        else:
            h = s.normed(self.norm, self.router, z, keep=True)
        self.mix(s, h, z, fs)

    def mix(self, s: Step, h: torch.Tensor, z: torch.Tensor, fs: torch.Tensor | None = None, beside: Mat | None = None, fill=None) -> None:
        """The experts' part behind the router's product ``z``.  ``fs``: the shared expert's hidden columns where they exist already.  ``beside``: another part of the layer whose
        last product is added in the same launch (a few rows; layers without a shared expert), ``fill(out)`` forms the columns it is multiplied with."""
        m, sh, post, mult = self.m, self.shared, self.post, s.be.stack.residual_mult
        both = fs is not None
        gate = z[:, m.outputs:m.outputs + 1] if sh and m.shared_gate else None
        out = s.x if post is None else s.buf("y", s.be.wp, torch.float32)
        if post is not None:
            mult = 1.0
        if s.small:
            tail = sh.down if sh else beside
            sfp = tail.w.shape[1] if tail else 0
            a = s.buf("experts", m.top * self.ffp + sfp, zero=True)
            ids, wts = s.buf("ids", m.top, torch.int32), s.buf("weights", m.top)
            if fill is not None:
                fill(a[:, m.top * self.ffp:])
            A.moe_up_rows(z, h, s.nb, self.gu, 2 * m.expert.ff, a, ids, wts, experts=m.experts, top=m.top, ffp=self.ffp, limit=m.expert.limit, act=self.act, outputs=m.outputs,
                          correction=self.correction, groups=self.groups, ws=sh.gu.w if sh else None, ns=2 * sh.e.ff if sh else 0, limit_s=sh.e.limit if sh else math.inf, pdl=s.pdl)
            A.moe_down_rows(a, s.nb, ids, wts, self.down, out, top=m.top, n=s.be.stack.width, mult=mult, ws=tail.w if tail else None, store=post is not None, h=h, gate=gate,
                            pdl=s.pdl)
            s.launched(2)
        else:
            ids, lids, wts = A.moe_route(z, m.outputs, m.top, m.experts, self.correction, self.groups)
            row, tile_expert, rows = K.moe_plan(lids, m.experts)
            xs = K.moe_gather(h, row, m.top, rows)
            f = torch.empty(rows, self.ffp, device=h.device, dtype=s.act)
            O.gemm(xs, self.gu.view(-1, self.gu.shape[2]), f, act=self.act, limit=m.expert.limit, experts=m.experts, tile_expert=tile_expert)
            y = torch.empty(rows, s.be.wp, device=h.device)
            O.gemm(f, self.down.view(-1, self.ffp), y, experts=m.experts, tile_expert=tile_expert)
            more, late = {"ids": ids, "n_experts": m.experts, "h": h} if m.identity else {}, post is None and gate is None
            if sh:
                if not both:
                    fs = s.buf("shared", up(sh.e.ff), zero=True)
                    s.product(h, sh.gu, fs, act=self.act, limit=sh.e.limit)
                if not late:
                    more["shared"], more["gate"] = s.buf("shared_y", s.be.wp, torch.float32), gate
                    s.product(fs, sh.down, more["shared"])
            K.moe_scatter_combine(y, row, wts, s.nb, m.top, out=out, accumulate=post is None, mult=mult, **more)
            s.launched(6)
            if sh and late:
                s.add(fs, sh.down)
        if post is not None:
            s.leave(out, post)


class SideInput:
    """g = gelu(gate x) * e[token]; x += multiplier * rmsnorm(proj g) * w, after a layer's feed-forward."""

    def __init__(self, src: WeightSource, p: str, dim: int, table: torch.Tensor):
        self.dim, self.dimp, self.e = dim, up(dim), table      # table [vocab, dimp]: this layer's part of every token's row
        self.gate = Mat(src.pack([(0, 0, p + "inp_gate.weight", (dim, src.width))], self.dimp, src.wp))
        self.proj = Mat(src.pack([(0, 0, p + "proj.weight", (src.width, dim))], src.wp, self.dimp))
        self.w = src.vec(p + "post_norm.weight", src.width)

    def product_weights(self) -> tuple[int, int, float]:
        return self.gate.w.numel() + self.proj.w.numel(), 0, 0.0

    def run(self, s: Step) -> None:
        h, s.copy = s.copy if s.copy is not None else s.x, None
        if h.dtype != s.act:
            h = s.buf("copy", s.be.wp)
            O.join_rows(s.x, s.be.wp, h, pdl=s.pdl)
            s.launched()
        g, y = s.buf("side_g", self.dimp), s.buf("side_y", s.be.wp, torch.float32)
        s.product(h, self.gate, g, act="gelu_tanh", mul=self.e)
        s.product(g, self.proj, y)
        s.pending = {"y": y, "wy": self.w, "mult": s.be.stack.residual_mult}
