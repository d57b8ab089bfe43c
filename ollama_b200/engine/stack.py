"""Engine of stack models (models/stack.py): decoders whose layers have mixers of different kinds, run on a paged cache.

A step is a set of rows: portions of prompts and single tokens of several sequences side by side.  Rows of all sequences share the
matrix products; attention reads each sequence's pages, the state-space scan each sequence's state.  A parallel block with two norms costs

    norm pair -> [q|k|v] product, feed-forward product with the activation in its epilogue -> attention
              -> one product over [attention output | feed-forward hidden] with the residual add in its epilogue

because W_o a + W_down f is one product over joined columns.  Layers whose mixer and feed-forward follow one another (engine/blocks.py, engine/mixers.py)
take each norm into the product behind it, or into one pass with what is still to be added to the stream.  Layers whose parts read one norm (engine/shared.py) share
their first and last products.  Decode steps of up to four sequences fuse the norms into a
multi-matrix GEMV (kernels/gemv_rows.cu), norm + rotation + cache append into the attention kernel, and the convolution and step-size
projection into the products around the recurrence: four launches per layer plus the merge of the attention splits.  Larger steps and
prompts multiply on the tcgen05 GEMM.  ``dtype`` "float32" runs weights, activations, cache and products in 32 bits.

Matrices are padded with zeros to multiples of eight rows and columns, activation rows likewise, so that any model size meets the
alignment of the tensor-core kernels.
"""
from __future__ import annotations

import logging
from typing import Sequence

import numpy as np
import torch

from .. import envconfig
from ..gguf.reader import GGUFFile
from ..models.config import ModelConfig, config_from_gguf
from ..models.stack import AttentionMixer, DenseMLP, ExpertMLP, LatentMixer, LayerRun, Mamba2Mixer, MambaMixer
from ..models.weights import QWeight, load_tensor
from ..ops import cuda as K
from ..ops import reference as R
from ..ops import rows as O
from .blocks import LONG_PORTION, ExpertFFN, GatedFFN, LatentAttention, LongPortions, Mat, Norm, SideInput, Step, WeightSource, make_norm, up
from .cache import CacheFull, PagedCache
from .mixers import HeadAttention, StateSpaceHeads
from .shared import DepthAverage, SharedNormLayer
from .steps import StepEngine

MAX_DECODE_ROWS = 32
LOGIT_ROWS = 256                 # rows per pass of the output head
LOG2E = 1.4426950408889634


_up8 = up


class _Layer:
    pass


class _Rows:
    """Named row buffers of a step; the buffers of decode steps live as long as their CUDA graphs."""

    def __init__(self, rows: int, device):
        self.rows, self.device, self.bufs = rows, device, {}

    def get(self, name: str, cols: int, dtype, nb: int, zero: bool = False) -> torch.Tensor:
        key = (name, cols, dtype)
        t = self.bufs.get(key)
        if t is None:
            t = self.bufs[key] = (torch.zeros if zero else torch.empty)(self.rows, cols, device=self.device, dtype=dtype)
        return t[:nb]


class _Meta:
    """Device arrays that describe the rows of a step."""

    def __init__(self, tokens, positions, slots, offs=None, segs=None, tiles=None, half_tiles=None, long: dict[int, LongPortions] | None = None,
                 longest: int = 1):
        self.tokens, self.positions, self.slots, self.offs, self.segs, self.tiles, self.half_tiles = tokens, positions, slots, offs, segs, tiles, half_tiles
        self.long, self.longest = long, longest      # by window (0: none); rows of the longest portion


class StackBackend(StepEngine):
    name = "b200"
    supports_embeds = False
    supports_shift = False           # chunk borders and recurrent states do not move with the tokens: the runner evaluates them again

    def __init__(self, g: GGUFFile | None, device: str = "cuda", opts=None, cfg: ModelConfig | None = None, tensors: dict[str, QWeight] | None = None,
                 dtype: str | None = None):
        self.device = torch.device(device if device != "cuda" else f"cuda:{torch.cuda.current_device()}")
        self.cfg = cfg if cfg is not None else config_from_gguf(g)
        self.stack = self.cfg.stack
        K.need("stack")
        dtype = dtype or getattr(opts, "dtype", None) or "bfloat16"
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"unknown compute type {dtype!r}")
        self.f32 = dtype == "float32"
        self.act_dtype = torch.float32 if self.f32 else torch.bfloat16
        kv_type = (getattr(opts, "kv_cache_type", None) or "f16").lower()
        if kv_type != "f16":
            logging.getLogger("ollama_b200.engine").warning("K/V cache type %s is stored as f16 (stack models have no quantised cache)", kv_type)
        self._init_steps()
        self.supports_verify = not self.cfg.recurrent
        self.max_batch = MAX_DECODE_ROWS
        self.gemv_rows = O.GEMV_MAX_ROWS      # steps of more sequences multiply on the tensor-core GEMM
        self.sms = torch.cuda.get_device_properties(self.device).multi_processor_count
        self.runs = self.stack.runs()
        self._load(g, tensors)

    # -- loading ------------------------------------------------------------------------------------
    def _load(self, g: GGUFFile | None, tensors) -> None:
        st, dev = self.stack, self.device
        width, self.wp = st.width, _up8(st.width)

        def get(name: str) -> torch.Tensor:
            return (tensors[name] if tensors is not None else load_tensor(g, name)).dequant().to(dev)

        src = WeightSource(get, dev, self.act_dtype, width, st.eps)
        vec, pack = src.vec, src.pack
        wp = self.wp
        self.embd = K.DevWeight(K.WT_F32 if self.f32 else K.WT_BF16, st.vocab, wp, [pack([(0, 0, "token_embd.weight", (st.vocab, width))], st.vocab, wp)])
        self.head = pack([(0, 0, "output.weight", (st.vocab, width))], _up8(st.vocab), wp)
        self.loop_in = self.loop_step = self.side_table = self.depth = None
        self.layers: list[_Layer] = []
        if not st.design.paired:
            self._load_sequential(src)
            torch.cuda.synchronize(dev)
            return
        self.out_norm = vec("output_norm.weight", width)
        if st.loop is not None:
            w = get("loop_in.weight")
            if tuple(w.shape) != (width, 2 * width):
                raise ValueError(f"loop_in.weight: shape {tuple(w.shape)}")
            self.loop_in = torch.zeros(wp, 2 * wp, device=dev, dtype=self.act_dtype)
            self.loop_in[:width, :width] = w[:, :width]
            self.loop_in[:width, wp:wp + width] = w[:, width:]
        for i, sl in enumerate(st.layers):
            L, p, m = _Layer(), f"blk.{i}.", sl.mixer
            L.mixer, L.mlp = m, sl.mlp
            L.norm1 = vec(p + "attn_norm.weight", width)
            L.ffp = 0
            L.norm2 = L.up = None
            if sl.mlp is not None:
                L.ffp = _up8(sl.mlp.ff)
                L.norm2 = vec(p + "ffn_norm.weight", width)
                L.up = pack([(0, 0, p + "ffn_up.weight", (sl.mlp.ff, width))], L.ffp, wp)
            if isinstance(m, AttentionMixer):
                nq, nk, nv = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
                L.n_qkv, L.mixp, L.mix_out = nq + nk + nv, _up8(m.heads * m.vdim), m.heads * m.vdim
                L.w_in = pack([(0, 0, p + "attn_q.weight", (nq, width)), (nq, 0, p + "attn_k.weight", (nk, width)),
                               (nq + nk, 0, p + "attn_v.weight", (nv, width))], _up8(L.n_qkv), wp)
                L.q_norm, L.k_norm = vec(p + "attn_q_norm.weight", nq), vec(p + "attn_k_norm.weight", nk)
                L.n_rot = m.rot.dims if m.rot else 0
                L.freqs = torch.tensor(m.rot.freqs() if m.rot else [0.0], dtype=torch.float64, device=dev)
                # the tensor-core kernels take cache rows of 64 or 128 f16 values
                big = max(m.dim, m.vdim)
                L.hd = 0 if self.f32 or big > 128 else 64 if big <= 64 else 128
                L.dk, L.dv = (L.hd, L.hd) if L.hd else (_up8(m.dim), _up8(m.vdim))
                out_name = "attn_output.weight"
            else:
                n, r, self_inner = m.state, m.dt_rank, m.inner
                L.inner, L.r8 = _up8(self_inner), _up8(r)
                L.mixp, L.mix_out = L.inner, self_inner
                w = get(p + "ssm_in.weight")
                if tuple(w.shape) != (2 * self_inner, width):
                    raise ValueError(f"{p}ssm_in.weight: shape {tuple(w.shape)}")
                L.w_in = torch.zeros(2 * L.inner, wp, device=dev, dtype=self.act_dtype)
                L.w_in[:self_inner, :width] = w[:self_inner]
                L.w_in[L.inner:L.inner + self_inner, :width] = w[self_inner:]
                L.np = _up8(L.r8 + 2 * n)
                w = get(p + "ssm_x.weight")
                if tuple(w.shape) != (r + 2 * n, self_inner):
                    raise ValueError(f"{p}ssm_x.weight: shape {tuple(w.shape)}")
                L.w_x = torch.zeros(L.np, L.inner, device=dev, dtype=self.act_dtype)      # rows: step size (padded) | B | C
                L.w_x[:r, :self_inner] = w[:r]
                L.w_x[L.r8:L.r8 + 2 * n, :self_inner] = w[r:]
                L.w_dt = pack([(0, 0, p + "ssm_dt.weight", (self_inner, r))], L.inner, L.r8)
                L.dt_bias, L.d = vec(p + "ssm_dt.bias", self_inner), vec(p + "ssm_d", self_inner)
                L.a2 = torch.zeros(L.inner, n, device=dev)
                L.a2[:self_inner] = (get(p + "ssm_a").double() * (1.0 if self.f32 else LOG2E)).float()
                L.conv_w = torch.zeros(m.conv, L.inner, device=dev)
                L.conv_w[:, :self_inner] = get(p + "ssm_conv1d.weight").float().t()
                L.conv_b = vec(p + "ssm_conv1d.bias", self_inner)
                out_name = "ssm_out.weight"
            parts = [(0, 0, p + out_name, (width, L.mix_out))]
            if sl.mlp is not None:
                parts.append((0, L.mixp, p + "ffn_down.weight", (width, sl.mlp.ff)))
            L.w_out = pack(parts, wp, L.mixp + L.ffp)
            self.layers.append(L)
        torch.cuda.synchronize(dev)

    def _load_sequential(self, src: WeightSource) -> None:
        """Layers made of the parts in blocks.py and mixers.py: mixer and feed-forward follow one another, each behind a norm and, in some designs, under another
        one, or read one norm."""
        st, f32 = self.stack, self.f32
        norm = st.design.norm
        self.out_norm = make_norm(src, "output_norm", norm)
        self.out_mat = Mat(self.head)
        if not f32 and norm == "layer":
            self.out_mat.fold(self.out_norm)
        if st.loop is not None:
            self.loop_step = torch.zeros(st.loop[2], src.wp, device=src.device)
            self.loop_step[:, :st.width] = src.tensor("loop_step.weight", st.loop[2], st.width).float()
        if st.side_dim:
            n, d = len(st.layers), st.side_dim
            self.side_table = src.zeros(st.vocab, n, _up8(d))
            self.side_table[..., :d] = src.tensor("per_layer_token_embd.weight", st.vocab, n * d).view(st.vocab, n, d)
        self.depth = DepthAverage(src, len(st.layers)) if st.design.depth_average else None
        for i, sl in enumerate(st.layers):
            L, p = _Layer(), f"blk.{i}."
            if st.design.shared_norm:
                self.layers.append(SharedNormLayer(src, p, sl, norm, f32))
                continue
            pre = make_norm(src, p + "attn_norm", norm)
            post = make_norm(src, p + "post_attention_norm", norm) if st.design.post_norm else None
            if isinstance(sl.mixer, LatentMixer):
                L.mix = LatentAttention(src, p, sl.mixer, pre, f32)
            elif isinstance(sl.mixer, (AttentionMixer, Mamba2Mixer)):
                L.mix = (HeadAttention if isinstance(sl.mixer, AttentionMixer) else StateSpaceHeads)(src, p, sl.mixer, pre, f32, post)
            else:
                raise NotImplementedError(f"{type(sl.mixer).__name__} in a sequential layer")
            L.ff = L.side = None
            if sl.mlp is not None:
                pre = make_norm(src, p + "ffn_norm", norm)
                post = make_norm(src, p + "post_ffw_norm", norm) if st.design.post_norm else None
                if isinstance(sl.mlp, ExpertMLP):
                    L.ff = ExpertFFN(src, p, sl.mlp, pre, f32, post)
                elif post is None:
                    L.ff = GatedFFN(src, p, sl.mlp, pre, f32)
                else:
                    raise NotImplementedError("a dense feed-forward under a norm of its own")
            if st.side_dim:
                L.side = SideInput(src, p, st.side_dim, self.side_table[:, i])
            self.layers.append(L)

    def _weights(self):
        """Every weight tensor on the device, once."""
        seen: set[int] = set()

        def walk(o):
            if isinstance(o, torch.Tensor):
                if o.untyped_storage().data_ptr() not in seen:           # matrices of several parts may be windows of one
                    seen.add(o.untyped_storage().data_ptr())
                    yield o
            elif isinstance(o, (list, tuple)):
                for v in o:
                    yield from walk(v)
            elif hasattr(o, "__dict__") and type(o).__module__.startswith(__package__):
                yield from walk(list(vars(o).values()))
        yield from walk([self.embd.planes[0], self.head, self.loop_in, self.loop_step, self.side_table, self.out_norm, self.layers, self.depth])

    def weight_bytes(self) -> int:
        return sum(t.untyped_storage().nbytes() for t in self._weights())

    def product_weights(self) -> tuple[int, int, float]:
        """Matrix weights over all layer runs and the head: (those every token is multiplied with, those of the routed experts, the share of
        the routed ones that a token picks)."""
        dense, routed, share = self.head.numel(), 0, 0.0
        for r in self.runs:
            L = self.layers[r.layer]
            if self.stack.design.paired:
                dense += sum(t.numel() for t in (L.w_in, L.up, L.w_out, getattr(L, "w_x", None), getattr(L, "w_dt", None)) if t is not None)
                dense += self.loop_in.numel() if r.joins else 0
                continue
            d, e, p = (sum(v) for v in zip(*(b.product_weights() for b in (L.mix, L.ff, L.side) if b is not None)))
            dense, routed, share = dense + d, routed + e, max(share, p)
        return dense, routed, share

    def kv_bytes(self) -> int:
        return self.cache.nbytes() if getattr(self, "cache", None) is not None else 0

    # -- buffers --------------------------------------------------------------------------------------
    def alloc(self, n_slots: int, n_ctx: int, pool_tokens: int | None = None) -> None:
        """``pool_tokens``: positions the page pool holds for all slots together (default: every slot can fill its context)."""
        dev = self.device
        self.n_slots, self.n_ctx = n_slots, n_ctx
        self.cache = PagedCache(n_slots, n_ctx, pool_tokens, dev)
        kv_dt = torch.float32 if self.f32 else torch.float16
        self.mem: list[tuple[torch.Tensor, torch.Tensor]] = []        # per layer run: (keys, values) or (state, convolution inputs)
        for r in self.runs:
            L = self.layers[r.layer]
            if not self.stack.design.paired:
                j = getattr(L.mix.m, "kv_from", None)
                kv = {} if j is None else {"kv": next(self.mem[k] for k in reversed(range(len(self.mem))) if self.runs[k].layer == j)}
                self.mem.append(L.mix.make_cache(self.cache, **kv))
            elif isinstance(L.mixer, AttentionMixer):
                self.mem.append((self.cache.add_pages(L.mixer.kv_heads, L.dk, kv_dt), self.cache.add_pages(L.mixer.kv_heads, L.dv, kv_dt)))
            else:
                self.mem.append((self.cache.add_state(L.inner, L.mixer.state), self.cache.add_state(max(L.mixer.conv - 1, 1), L.inner)))
        MB, i32 = self.max_batch, torch.int32
        b = self.buf = _Layer()
        b.rows = _Rows(MB, dev)
        b.all_logits = torch.zeros(MB, _up8(self.stack.vocab), device=dev)
        b.logits = b.all_logits[:, :self.stack.vocab]
        b.meta = torch.zeros(3, MB, device=dev, dtype=i32)          # tokens | positions | slots of the decode batch
        b.tokens, b.positions, b.slots = b.meta[0], b.meta[1], b.meta[2]
        b.offs = torch.zeros(MB, device=dev, dtype=i32)
        b.sampled = torch.zeros(MB, device=dev, dtype=i32)
        b.host_in, b.host_out = torch.zeros(3, MB, dtype=i32).pin_memory(), torch.zeros(MB, dtype=i32).pin_memory()
        b.host_np, b.host_out_np = b.host_in.numpy(), b.host_out.numpy()
        att = [L for L in self.layers if self.stack.design.paired and isinstance(L.mixer, AttentionMixer) and L.hd]
        for L in att:       # split-K width of decode attention, by the most keys a query of the layer can see
            L.keys = min(n_ctx, L.mixer.chunk or n_ctx)
            L.n_splits = max(1, min(envconfig.attn_splits(), L.keys // envconfig.attn_split_len()))
        b.part_acc = torch.zeros(max([MB * L.mixer.heads * L.n_splits * L.hd for L in att], default=1), device=dev)
        b.part_ml = torch.zeros(max([MB * L.mixer.heads * L.n_splits * 2 for L in att], default=1), device=dev)
        self._graphs.clear()
        self._warm.clear()

    def close(self) -> None:
        self._graphs.clear()
        self.mem, self.cache, self.buf = [], None, None

    def admit(self, slot: int, n_tokens: int, idle: Sequence[int]) -> tuple[bool, list[int]]:
        """Reserve pages for ``n_tokens`` positions of ``slot``, giving up what the ``idle`` slots still hold, in their order, as far as
        needed.  Returns whether that sufficed and the slots that were emptied."""
        dropped: list[int] = []
        for s in [None, *idle]:
            if s is not None:
                self.cache.release(s)
                dropped.append(s)
            try:
                self.cache.reserve(slot, n_tokens)
                return True, dropped
            except CacheFull:
                continue
        return False, dropped

    def free_slot(self, slot: int) -> None:
        """The sequence in ``slot`` has ended: its pages go back to the pool."""
        self.cache.release(slot)

    def _reserve(self, slots, ends) -> None:
        for s, e in zip(slots, ends):
            self.cache.reserve(s, e)
        self.h2d_bytes += self.cache.sync()

    # -- one layer run ----------------------------------------------------------------------------------
    def _mm(self, a, w, out, **kw) -> None:
        O.gemm(a, w, out, **kw)
        self._n += 1

    def _layer(self, i: int, x: torch.Tensor, x0: torch.Tensor, B: _Rows, m: _Meta, decode: bool) -> torch.Tensor:
        """Layer run ``i`` on the residual rows ``x``; returns the residual (another buffer where the run begins a pass of the loop)."""
        run = self.runs[i]
        L, wp, eps, nb, f32 = self.layers[run.layer], self.wp, self.stack.eps, x.shape[0], torch.float32
        small = decode and nb <= self.gemv_rows
        AT = f32 if small else self.act_dtype
        pdl = self.pdl and decode
        if run.joins:
            y = B.get("x1" if x.data_ptr() == B.get("x", wp, f32, nb, True).data_ptr() else "x", wp, f32, nb, True)
            if small:
                O.gemv([O.seg(self.loop_in, self.stack.width, y)], 2 * wp, x, nb, self.f32, O.SRC_JOINED, x2=x0, k1=wp, pdl=pdl)
            else:
                j = B.get("joined", 2 * wp, AT, nb)
                O.join_rows(x, wp, j, x0, wp, wp, pdl=pdl)
                self._mm(j, self.loop_in, y)
            self._n += 1
            x = y
        n_in = L.w_in.shape[0]
        act = L.mlp.act if L.mlp else ""
        cat = B.get("cat", L.mixp + L.ffp, AT, nb, True)
        h_in = B.get("in", n_in, f32 if isinstance(L.mixer, AttentionMixer) else AT, nb)
        if small:
            segs = [O.seg(L.w_in, n_in, h_in, L.norm1)]
            if L.ffp:
                segs.append(O.seg(L.up, L.ffp, cat[:, L.mixp:], L.norm2, act))
            if isinstance(L.mixer, MambaMixer):      # the convolution follows in the product's epilogue
                u = B.get("u", L.inner, f32, nb)
                O.gemv(segs, wp, x, nb, self.f32, O.SRC_NORM, eps, self.stack.width, conv=(L.conv_w, L.conv_b, self.mem[i][1]), conv_out=u, slots=m.slots,
                       positions=m.positions, pdl=pdl)
            else:
                O.gemv(segs, wp, x, nb, self.f32, O.SRC_NORM, eps, self.stack.width, pdl=pdl)
        else:
            h1, h2 = B.get("h1", wp, AT, nb), B.get("h2", wp, AT, nb) if L.ffp else None
            O.norm_rows(x, self.stack.width, eps, L.norm1, h1, L.norm2, h2, pdl=pdl)
            self._mm(h1, L.w_in, h_in)
            if L.ffp:
                self._mm(h2, L.up, cat[:, L.mixp:], act=act)
        self._n += 1
        if isinstance(L.mixer, AttentionMixer):
            self._attention(L, self.mem[i], h_in, cat, B, m, decode, pdl)
        else:
            self._mamba(L, self.mem[i], h_in, cat, B, m, decode, small, pdl)
        if small:
            O.gemv([O.seg(L.w_out, self.stack.width, x, accumulate=True)], cat.shape[1], cat, nb, self.f32, pdl=pdl)
            self._n += 1
        else:
            self._mm(cat, L.w_out, x, accumulate=True)
        return x

    def _attention(self, L, mem, qkv, out, B, m, decode, pdl) -> None:
        mx, (kc, vc), b, nb = L.mixer, mem, self.buf, qkv.shape[0]
        table = self.cache.table
        if decode and L.hd and O.attn_decode_paged(
                qkv, kc, vc, m.positions, m.slots, table, out, nb, heads=mx.heads, dim=mx.dim, vdim=mx.vdim, q_norm=L.q_norm, k_norm=L.k_norm,
                eps=self.stack.eps, freqs=L.freqs, n_rot=L.n_rot, scale=mx.scale, softcap=mx.softcap, chunk=mx.chunk, n_splits=L.n_splits, n_ctx=L.keys,
                part_acc=b.part_acc, part_ml=b.part_ml, pdl=pdl):
            self._n += 2
            return
        dq = L.hd or mx.dim
        q = B.get("q", mx.heads * dq, torch.float32, nb).view(nb, mx.heads, dq)
        O.paged_append(qkv, heads=mx.heads, kv_heads=mx.kv_heads, dim=mx.dim, vdim=mx.vdim, q_norm=L.q_norm, k_norm=L.k_norm, eps=self.stack.eps,
                       freqs=L.freqs, n_rot=L.n_rot, positions=m.positions, slots=m.slots, table=table, q_out=q, k_cache=kc, v_cache=vc, pdl=pdl)
        if L.hd and m.tiles is not None:
            O.attn_prefill_paged(q, kc, vc, m.tiles, table, out, vdim=mx.vdim, scale=mx.scale, softcap=mx.softcap, chunk=mx.chunk)
        else:
            O.paged_attn(q, kc, vc, m.positions, m.slots, table, out, dim=mx.dim, vdim=mx.vdim, scale=mx.scale, softcap=mx.softcap, chunk=mx.chunk, pdl=pdl)
        self._n += 2

    def _mamba(self, L, mem, xz, out, B, m, decode, small, pdl) -> None:
        (state, conv_state), nb, f32 = mem, xz.shape[0], torch.float32
        p = B.get("p", L.np, f32, nb)
        conv = (L.conv_w, L.conv_b, conv_state)
        if small:
            u = B.get("u", L.inner, f32, nb)
            O.gemv([O.seg(L.w_x, L.np, p)], L.inner, u, nb, self.f32, pdl=pdl)
            O.ssm_step(xz, L.inner, conv, p, L.r8, L.w_dt, None, L.dt_bias, L.a2, L.d, state, m.slots, m.positions, out, nb, self.f32, u, pdl=pdl)
            self._n += 2
            return
        u, dl, dt = B.get("u", L.inner, xz.dtype, nb), B.get("dl", L.r8, xz.dtype, nb), B.get("dt", L.inner, f32, nb)
        O.ssm_conv(xz, L.inner, L.conv_w, L.conv_b, conv_state, m.slots, m.positions, m.offs, u, pdl=pdl)
        self._mm(u, L.w_x, p)
        O.join_rows(p, L.r8, dl, pdl=pdl)
        self._mm(dl, L.w_dt, dt)
        if decode:
            O.ssm_step(xz, L.inner, conv, p, L.r8, L.w_dt, dt, L.dt_bias, L.a2, L.d, state, m.slots, m.positions, out, nb, self.f32, pdl=pdl)
        else:
            O.ssm_scan(xz, L.inner, u, dt, p, L.r8, L.dt_bias, L.a2, L.d, L.mixer.conv, state, conv_state, m.segs, out)
        self._n += 3

    def _run_rows(self, B: _Rows, m: _Meta, nb: int, decode: bool, tap=None) -> torch.Tensor:
        """All layer runs on ``nb`` rows; ``tap(i, x)``: called after every run (inspection)."""
        hist = None
        if self.depth is not None:
            n = len(self.runs) + 2
            hist = B.get("hist", n * self.wp, torch.float32, nb).view(n, nb, self.wp)
        x = B.get("x", self.wp, torch.float32, nb, True) if hist is None else hist[0]
        K.embed(self.embd, m.tokens[:nb], self.stack.embed_scale, out=x)
        self._n += 1
        x0 = x
        if self.stack.loop is not None:
            x0 = B.get("x0", self.wp, torch.float32, nb, True)
            x0.copy_(x)
        if hist is not None:
            return self._run_depth(Step(self, B, m, x, x0, decode, hist), tap)
        if not self.stack.design.paired:
            return self._run_sequential(Step(self, B, m, x, x0, decode), tap)
        for i in range(len(self.runs)):
            x = self._layer(i, x, x0, B, m, decode)
            if tap is not None:
                tap(i, x[:, :self.stack.width])
        return x

    def _join(self, run: LayerRun | None, s: Step) -> dict:
        """What a layer run adds to the stream before it begins: a pass of the loop starts with a vector of its own and, but for the first, with the
        embedding output."""
        if run is None or not run.joins:
            return {}
        return {"step": self.loop_step[run.turn], **({"x0": s.x0} if run.turn else {})}

    def _run_sequential(self, s: Step, tap=None) -> torch.Tensor:
        s.pending = self._join(self.runs[0], s)
        for i, run in enumerate(self.runs):
            L, nxt = self.layers[run.layer], self.runs[i + 1] if i + 1 < len(self.runs) else None
            s.last = L.side is not None and L.ff is None
            L.mix.run(s, self.mem[i])
            if L.ff is not None:
                s.last = L.side is not None
                L.ff.run(s)
            if L.side is not None:
                L.side.run(s)
            if tap is not None:                # the stream of this layer run, before anything is added for the next one
                s.flush()
                tap(i, s.x[:, :self.stack.width])
            s.pending.update(self._join(nxt, s))
        s.flush()
        return s.x

    def _run_depth(self, s: Step, tap=None) -> torch.Tensor:
        """Layers that read a weighted sum of the embedding output and all earlier results; the output reads one too."""
        w, n = self.depth.w, len(self.runs)
        for i in range(n + 1):
            h = s.average(i + 1, w[i], self.layers[self.runs[i].layer].norm if i < n else None)
            if tap is not None and i > 0:
                tap(i - 1, s.x[:, :self.stack.width])
            if i < n:
                self.layers[self.runs[i].layer].run(s, self.mem[i], h)
        return s.x

    def _head_rows(self, x: torch.Tensor, out: torch.Tensor, pdl: bool = False) -> None:
        """Logits (before the soft cap) of hidden rows ``x`` into the rows of ``out`` [rows, padded vocabulary]."""
        nb, st = x.shape[0], self.stack
        scale = st.logit_scale
        if isinstance(self.out_norm, Norm):
            if nb <= self.gemv_rows and self.out_norm.b is None:
                O.gemv([O.seg(self.head, st.vocab, out, self.out_norm.g, alpha=scale)], self.wp, x, nb, self.f32, O.SRC_NORM, st.eps, st.width, pdl=pdl)
            elif nb <= self.gemv_rows and not self.f32:
                m = self.out_mat
                O.gemv([O.seg(m.w, m.w.shape[0], out, self.out_norm.g, rs=m.rs, rc=m.rc, alpha=scale)], self.wp, x, nb, False, O.SRC_LAYER, st.eps, st.width, pdl=pdl)
            else:
                h = torch.empty(nb, self.wp, device=self.device, dtype=self.act_dtype)
                O.norm_rows(x, st.width, st.eps, self.out_norm.g, h, b1=self.out_norm.b, pdl=pdl)
                self._mm(h, self.head, out, alpha=scale)
        elif nb <= self.gemv_rows:
            O.gemv([O.seg(self.head, st.vocab, out, self.out_norm, alpha=scale)], self.wp, x, nb, self.f32, O.SRC_NORM, st.eps, st.width, pdl=pdl)
        else:
            h = torch.empty(nb, self.wp, device=self.device, dtype=self.act_dtype)
            O.norm_rows(x, st.width, st.eps, self.out_norm, h, pdl=pdl)
            self._mm(h, self.head, out, alpha=scale)
        self._n += 1

    # -- decode ---------------------------------------------------------------------------------------
    def _stage(self, slots, tokens, positions) -> int:
        self._reserve(slots, [p + 1 for p in positions])
        return super()._stage(slots, tokens, positions)

    def _decode_kernels(self, nb: int, want_argmax) -> None:
        b = self.buf
        self._n = 0
        m = _Meta(b.tokens[:nb], b.positions[:nb], b.slots[:nb], b.offs[:nb])
        x = self._run_rows(b.rows, m, nb, decode=True)
        self._head_rows(x, b.all_logits[:nb], pdl=self.pdl)
        if want_argmax:
            loop = want_argmax == "loop"
            K.argmax(b.logits[:nb], out=b.sampled, tokens=b.tokens if loop else None, positions=b.positions if loop else None)
            self._n += 1
        self.launches_per_step = self._n

    @torch.no_grad()
    def decode_loop(self, slots, tokens, positions, n_steps, first_tokens=None):
        if len(slots) <= self.max_batch:
            self._reserve(slots, [p + n_steps for p in positions])
        return super().decode_loop(slots, tokens, positions, n_steps, first_tokens)

    # -- prompt rows and mixed steps ----------------------------------------------------------------------
    @torch.no_grad()
    def _forward_rows(self, segs: Sequence[tuple[int, Sequence[int], int]], x=None, embeds=None, spans=(), tap=None) -> torch.Tensor:
        """Rows of several sequences, each portion ``(slot, tokens, position of the first)``; returns the hidden rows in order."""
        dev = self.device
        self._reserve([s for s, _, _ in segs], [p0 + len(t) for _, t, p0 in segs])
        total = sum(len(t) for _, t, _ in segs)
        cols = np.empty((4, total), np.int32)           # tokens | positions | slots | offset in the portion
        seg_rows, tiles, at = [], [], 0
        windows = sorted({L.mixer.window for L in self.stack.layers if isinstance(L.mixer, LatentMixer)})
        longs = {w: ([], [], []) for w in windows}          # tiles, sequences, positions of each
        halves, rest = any(isinstance(L.mixer, AttentionMixer) and L.mixer.maps > 1 for L in self.stack.layers), []
        half_tiles = []
        for slot, toks, p0 in segs:
            n = len(toks)
            cols[0, at:at + n] = toks
            cols[1, at:at + n] = np.arange(p0, p0 + n)
            cols[2, at:at + n] = slot
            cols[3, at:at + n] = np.arange(n)
            seg_rows.append((at, n, slot, p0))
            tiles += [(at + r, min(128, n - r), slot, p0 + r) for r in range(0, n, 128)]
            if halves:
                half_tiles += [(at + r, min(64, n - r), slot, p0 + r) for r in range(0, n, 64)]
            if n < LONG_PORTION:
                rest += range(at, at + n)
            else:
                for w, (lt, seqs, count) in longs.items():
                    first = max(0, p0 - w + 1) & ~127 if w else 0       # keys are visited in tiles of 128 positions
                    row0 = sum(count) - first
                    lt += [(at + r, min(128, n - r), row0, p0 + r) for r in range(0, n, 128)]
                    seqs.append((row0, p0 + n, slot, first))
                    count.append(p0 + n - first)
            at += n
        np.maximum(cols[0], 0, out=cols[0])
        meta = torch.from_numpy(cols).to(dev)
        lists = [seg_rows, tiles, half_tiles, *(t for lt, seqs, _ in longs.values() for t in (lt, seqs))]
        geom = torch.tensor([r for t in lists for r in t], dtype=torch.int32).to(dev)
        self.h2d_bytes += 4 * (meta.numel() + geom.numel())
        parts = list(torch.split(geom, [len(t) for t in lists]))
        long = None
        if windows and len(rest) < total:
            rows = torch.tensor(rest, dtype=torch.int32).to(dev) if rest else None
            self.h2d_bytes += 4 * len(rest)
            long = {w: LongPortions(parts[3 + 2 * i], parts[4 + 2 * i], sum(count), max(count), rows) for i, (w, (_, _, count)) in enumerate(longs.items())}
        m = _Meta(meta[0], meta[1], meta[2], meta[3], *parts[:2], parts[2] if halves else None, long, max(len(t) for _, t, _ in segs))
        self._n = 0
        out = self._run_rows(_Rows(at, dev), m, at, decode=False, tap=tap)
        self.kernel_launches += self._n
        return out

    def _final_norm(self, x: torch.Tensor) -> torch.Tensor:
        w = self.stack.width
        if isinstance(self.out_norm, Norm):
            if self.out_norm.b is None:
                return R.rmsnorm(x[:, :w], self.out_norm.g[:w], self.stack.eps)
            return torch.nn.functional.layer_norm(x[:, :w], (w,), self.out_norm.g[:w], self.out_norm.b[:w], self.stack.eps)
        return R.rmsnorm(x[:, :w], self.out_norm[:w], self.stack.eps)

    def _logits(self, x: torch.Tensor) -> torch.Tensor:
        self._n = 0
        x = x.contiguous()
        out = torch.empty(x.shape[0], _up8(self.stack.vocab), device=self.device)
        for r in range(0, x.shape[0], LOGIT_ROWS):
            self._head_rows(x[r:r + LOGIT_ROWS], out[r:r + LOGIT_ROWS])
        self.kernel_launches += self._n
        return R.softcap(out[:, :self.stack.vocab], self.cfg.final_softcap)

    @torch.no_grad()
    def step(self, segs: Sequence[tuple[int, Sequence[int], int]], want: Sequence[Sequence[int]]) -> torch.Tensor | None:
        """One batch: portions of prompts beside single tokens, ``(slot, tokens, position of the first)`` each; ``want``: per portion the
        indices of the rows to return logits for.  Returns [rows, vocab] in that order, or None without any."""
        if all(len(t) == 1 for _, t, _ in segs) and len(segs) <= self.max_batch:
            rows = [i for i, w in enumerate(want) for _ in w]
            lg = self.decode([s for s, _, _ in segs], [max(int(t[0]), 0) for _, t, _ in segs], [p for _, _, p in segs])
            return lg[rows] if rows else None
        x = self._forward_rows(segs)
        rows, at = [], 0
        for (_, toks, _), w in zip(segs, want):
            rows += [at + int(j) for j in w]
            at += len(toks)
        return self._logits(x[torch.tensor(rows, device=self.device)]) if rows else None

    # -- slots --------------------------------------------------------------------------------------------
    @torch.no_grad()
    def copy_rows(self, src: int, dst: int, n: int) -> None:
        """The first ``n`` positions of slot ``src`` (for recurrent models: all it holds) become those of slot ``dst``."""
        self.cache.copy(src, dst, n)
        self.h2d_bytes += self.cache.sync()
