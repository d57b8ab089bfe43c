"""Bindings of the row kernels behind stack models: norms, fused decode products, products of many rows, paged attention and the selective
state-space mixer (kernels/norm_rows.cu, gemv_rows.cu, gemm_tc.cu, gemm_f32.cu, attn_paged.cu, ssm.cu, depth.cu, gru.cu)."""
from __future__ import annotations

import ctypes as C
import functools
import math

import torch

from .cuda import AttnDecodeArgs, AttnPrefillArgs, AttnRopeArgs, _check, lib, ptr, stream

P, I, F = C.c_void_p, C.c_int, C.c_float
GLU_BASE = 16
ACT = {"": 0, "relu2": 1, "gelu_tanh": 2, "xielu": 3, "glu:silu": GLU_BASE, "glu:gelu_tanh": GLU_BASE + 1, "glu:swiglu_oai": GLU_BASE + 2}
OUT_TYPE = {torch.float32: 0, torch.bfloat16: 1, torch.float16: 2}
SRC_ROWS, SRC_NORM, SRC_JOINED, SRC_LAYER = range(4)
GEMV_MAX_ROWS = 4
NO_NUMS = (0.0, 0.0)


def _st(name: str, fields: list) -> type:
    return type(name, (C.Structure,), {"_fields_": fields})


NormRowsArgs = _st("NormRowsArgs", [("x", P), ("ldx", I), ("k", I), ("ldo", I), ("eps", F), ("w1", P), ("w2", P), ("o1", P), ("o2", P), ("f32", I),
                                    ("b1", P), ("b2", P), ("y", P), ("wy", P), ("x0", P), ("step", P), ("ldy", I), ("mult", F)])
JoinRowsArgs = _st("JoinRowsArgs", [("a", P), ("b", P), ("lda", I), ("n_a", I), ("ldb", I), ("n_b", I), ("out", P), ("ldo", I), ("off_b", I), ("f32", I)])
RowSeg = _st("RowSeg", [("w", P), ("g", P), ("rs", P), ("rc", P), ("out", P), ("n", I), ("ldw", I), ("ldo", I), ("act", I), ("accumulate", I), ("alpha", F),
                        ("limit", F), ("mul", P), ("ldm", I), ("act_p", F), ("act_q", F)])
GemmRowsArgs = _st("GemmRowsArgs", [("a", P), ("b", P), ("out", P), ("bias", P), ("mul", P), ("mul_row", P), ("tile_expert", P), ("copy", P), ("ws", P),
                                    ("ws_floats", C.c_longlong), ("m", I), ("n", I), ("k", I), ("lda", I), ("ldb", I), ("ldo", I), ("out_type", I), ("act", I),
                                    ("accumulate", I), ("experts", I), ("ldm", I), ("alpha", F), ("limit", F), ("tail", P), ("tail_col", I), ("ld_tail", I),
                                    ("act_p", F), ("act_q", F)])
GemvRowsArgs = _st("GemvRowsArgs", [("seg", RowSeg * 4), ("nseg", I), ("nb", I), ("k", I), ("src", I), ("f32", I), ("x", P), ("ldx", I), ("x2", P),
                                    ("ldx2", I), ("k1", I), ("eps", F), ("kn", I), ("conv_seg", I), ("conv_n", I), ("taps", I), ("conv_w", P),
                                    ("conv_b", P), ("conv_state", P), ("conv_silu", I), ("conv_shift", I), ("conv_out", P), ("ldu", I), ("slots", P), ("positions", P),
                                    ("h", P), ("ldh", I), ("hb", P), ("mul_row", P)])
PagedAppendArgs = _st("PagedAppendArgs", [("qkv", P), ("ldq", I), ("n_heads", I), ("n_kv_heads", I), ("dim", I), ("vdim", I), ("q_norm", P), ("k_norm", P),
                                          ("eps", F), ("freqs", P), ("n_rot", I), ("positions", P), ("slots", P), ("page_table", P), ("max_pages", I),
                                          ("q_out", P), ("dq", I), ("k_cache", P), ("v_cache", P), ("dk", I), ("dv", I), ("cache32", I),
                                          ("head_norm", I), ("v_off", I), ("mscale", F), ("maps", I), ("no_append", I)])
HeadGate = _st("HeadGate", [("g", P), ("ld", I), ("kind", I)])
DiffHeads = _st("DiffHeads", [("lam", F), ("scale", F), ("eps", F), ("on", I)])
PagedAttnArgs = _st("PagedAttnArgs", [("q", P), ("dq", I), ("n_heads", I), ("n_kv_heads", I), ("dim", I), ("vdim", I), ("k_cache", P), ("v_cache", P),
                                      ("dk", I), ("dv", I), ("cache32", I), ("positions", P), ("slots", P), ("page_table", P), ("max_pages", I),
                                      ("chunk", I), ("scale", F), ("softcap", F), ("out", P), ("ldo", I), ("out16", I), ("window", I), ("keep", I), ("gate", HeadGate)])
AttnPagedArgs = _st("AttnPagedArgs", [("tiles", P), ("page_table", P), ("max_pages", I), ("chunk", I), ("vdim", I), ("ldo", I), ("window", I), ("keep", I), ("gate", HeadGate),
                                      ("diff", DiffHeads)])
SsmConvArgs = _st("SsmConvArgs", [("xz", P), ("ldx", I), ("inner", I), ("taps", I), ("w", P), ("b", P), ("state", P), ("slots", P), ("positions", P),
                                  ("offs", P), ("u", P), ("ldu", I), ("silu", I), ("shift", I)])
ConvKeepArgs = _st("ConvKeepArgs", [("xz", P), ("ldx", I), ("inner", I), ("taps", I), ("state", P), ("seg", P)])
SsmScanArgs = _st("SsmScanArgs", [("xz", P), ("ldx", I), ("off_z", I), ("u", P), ("ldu", I), ("dt", P), ("lddt", I), ("bc", P), ("ldbc", I), ("off_b", I),
                                  ("dt_bias", P), ("a2", P), ("d", P), ("inner", I), ("n_state", I), ("taps", I), ("state", P), ("conv_state", P), ("seg", P),
                                  ("out", P), ("ldo", I)])
SsmStepArgs = _st("SsmStepArgs", [("xz", P), ("ldx", I), ("off_z", I), ("xz16", I), ("conv_w", P), ("conv_b", P), ("conv_state", P), ("taps", I),
                                  ("inner", I), ("n_state", I), ("p", P), ("ldp", I), ("off_b", I), ("w_dt", P), ("rank", I), ("w32", I), ("dt", P),
                                  ("lddt", I), ("dt_bias", P), ("a2", P), ("d", P), ("state", P), ("slots", P), ("positions", P), ("out", P), ("ldo", I),
                                  ("out16", I), ("exact", I), ("u", P), ("ldu", I)])
DepthRowsArgs = _st("DepthRowsArgs", [("hist", P), ("stride", C.c_longlong), ("w", P), ("n", I), ("k", I), ("ldx", I), ("x", P), ("g", P), ("b", P), ("h", P), ("ldo", I),
                                      ("f32", I), ("eps", F)])
GruArgs = _st("GruArgs", [("x", P), ("ldx", I), ("off_u", I), ("off_g", I), ("width", I), ("state", P), ("seg", P), ("slots", P), ("positions", P), ("out", P), ("ldo", I)])


def _is32(t: torch.Tensor) -> int:
    return int(t.dtype == torch.float32)


def _call(name: str, args, *more) -> None:
    _check(getattr(lib(), name)(C.byref(args), *more, stream()), name)


def norm_rows(x: torch.Tensor, k: int, eps: float, w1: torch.Tensor | None, o1: torch.Tensor | None, w2: torch.Tensor | None = None,
              o2: torch.Tensor | None = None, b1: torch.Tensor | None = None, b2: torch.Tensor | None = None, y: torch.Tensor | None = None,
              wy: torch.Tensor | None = None, mult: float = 1.0, x0: torch.Tensor | None = None, step: torch.Tensor | None = None, pdl: bool = False) -> None:
    """o1 = norm(x) * w1 and, in the same pass, o2 = norm(x) * w2, for the first ``k`` columns; pad columns of the results are zeroed.  With biases
    a layer norm, else an RMS norm.  Before it x += mult * rmsnorm(y) * wy + x0 + step, in place, of the terms that are given; ``o1`` None: only that."""
    if x0 is not None and x0.stride(0) != x.stride(0):
        raise ValueError("norm_rows: row pitch of the joined rows")
    a = NormRowsArgs(ptr(x), x.stride(0), k, o1.stride(0) if o1 is not None else 0, eps, ptr(w1), ptr(w2), ptr(o1), ptr(o2), _is32(o1) if o1 is not None else 0,
                     ptr(b1), ptr(b2), ptr(y), ptr(wy), ptr(x0), ptr(step), y.stride(0) if y is not None else 0, mult)
    _call("b2_norm_rows", a, x.shape[0], int(pdl))


def join_rows(a: torch.Tensor, n_a: int, out: torch.Tensor, b: torch.Tensor | None = None, n_b: int = 0, off_b: int = 0, pdl: bool = False) -> None:
    """Columns 0 .. n_a - 1 of ``a`` and, from column ``off_b`` on, ``n_b`` columns of ``b``; zeros elsewhere; in the result's element type."""
    args = JoinRowsArgs(ptr(a), ptr(b), a.stride(0), n_a, b.stride(0) if b is not None else 0, n_b, ptr(out), out.stride(0), off_b, _is32(out))
    _call("b2_join_rows", args, a.shape[0], int(pdl))


def seg(w: torch.Tensor, n: int, out: torch.Tensor, g: torch.Tensor | None = None, act: str = "", accumulate: bool = False, alpha: float = 1.0,
        limit: float = math.inf, nums: tuple[float, float] = NO_NUMS, rs: torch.Tensor | None = None, rc: torch.Tensor | None = None,
        mul: torch.Tensor | None = None) -> RowSeg:
    """One matrix of :func:`gemv`: the first ``n`` rows of ``w`` into the rows of ``out``, as out (+)= alpha * act(... + rc) [* mul[mul_row]].  ``rs``: the rows' sums of
    w * g (layer norm).  ``nums``: the two numbers of the "xielu" activation.  Gated activations ("glu:...") take rows 2i and 2i + 1 as gate and up of column i."""
    s = RowSeg(ptr(w), ptr(g), ptr(rs), ptr(rc), ptr(out), n, w.stride(0), out.stride(0), ACT[act], int(accumulate), alpha, limit, ptr(mul),
               mul.stride(0) if mul is not None else 0, *nums)
    s.keep = (w, g, rs, rc, out, mul)     # the structure holds addresses only
    return s


def gemv(segs: list, k: int, x: torch.Tensor, nb: int, f32: bool, src: int = SRC_ROWS, eps: float = 0.0, kn: int = 0, x2: torch.Tensor | None = None,
         k1: int = 0, conv=None, conv_out: torch.Tensor | None = None, slots: torch.Tensor | None = None, positions: torch.Tensor | None = None,
         h: torch.Tensor | None = None, hb: torch.Tensor | None = None, mul_row: torch.Tensor | None = None,
         conv_silu: bool = True, conv_shift: bool = False, pdl: bool = False) -> None:
    """Products of up to four matrices with up to four source rows.  ``conv`` = (weights [taps, n], bias [n] or None, state [slots, taps - 1, n]): the first n
    results of the first matrix also run through that convolution, and with ``conv_silu`` SiLU, into ``conv_out``; ``conv_shift``: they enter the state.  ``h``: the normalised
    rows for the first matrix are stored too (``hb``: a layer norm's bias)."""
    a = GemvRowsArgs()
    for i, s in enumerate(segs):
        a.seg[i] = s
    a.nseg, a.nb, a.k, a.src, a.f32, a.x, a.ldx, a.eps, a.kn, a.conv_seg = len(segs), nb, k, src, int(f32), ptr(x), x.stride(0), eps, kn, -1
    a.mul_row = ptr(mul_row)
    if h is not None:
        a.h, a.ldh, a.hb = ptr(h), h.stride(0), ptr(hb)
    if x2 is not None:
        a.x2, a.ldx2, a.k1 = ptr(x2), x2.stride(0), k1
    if conv is not None:
        a.conv_seg, a.conv_n, a.taps = 0, conv[0].shape[1], conv[0].shape[0]
        a.conv_w, a.conv_b, a.conv_state, a.conv_out, a.ldu = ptr(conv[0]), ptr(conv[1]), ptr(conv[2]), ptr(conv_out), conv_out.stride(0)
        a.slots, a.positions, a.conv_silu, a.conv_shift = ptr(slots), ptr(positions), int(conv_silu), int(conv_shift)
    _call("b2_gemv_rows", a, int(pdl))


def gemm(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, act: str = "", accumulate: bool = False, k: int | None = None, alpha: float = 1.0,
         limit: float = math.inf, nums: tuple[float, float] = NO_NUMS, bias: torch.Tensor | None = None, mul: torch.Tensor | None = None, mul_row: torch.Tensor | None = None,
         experts: int = 0, tile_expert: torch.Tensor | None = None, copy: torch.Tensor | None = None, tail: torch.Tensor | None = None) -> None:
    """out (+)= alpha * act(a[:, :k] @ w[:, :k]^T + bias) [* mul[mul_row]]; bf16 operands on tcgen05 (result bf16, f16 or fp32), fp32 operands in full
    32 bits.  ``copy``: bf16 rows of out's pitch that receive an fp32 result too.
    ``a``, ``out`` and ``mul`` may be column windows of wider buffers.  Gated activations ("glu:...") halve the columns.  ``experts``: w holds
    that many stacked matrices and a's tiles of 128 rows belong to ``tile_expert``.  ``tail``: fp32 rows that receive the last columns' sums, as they are, instead of
    ``out`` (bf16 operands)."""
    n = w.shape[0] // max(experts, 1)
    m, k, nt = a.shape[0], w.shape[1] if k is None else k, tail.shape[1] if tail is not None else 0
    cols = (n - nt) // 2 if act.startswith("glu:") else n - nt
    if a.dtype != w.dtype or out.shape[0] != m or out.shape[1] != cols or a.shape[1] < k or a.stride(1) != 1 or out.stride(1) != 1:
        raise ValueError(f"gemm: {tuple(a.shape)} {a.dtype} x {tuple(w.shape)} {w.dtype} -> {tuple(out.shape)}")
    if nt and (tail.shape[0] != m or tail.dtype != torch.float32 or tail.stride(1) != 1):
        raise ValueError(f"gemm: tail {tuple(tail.shape)} {tail.dtype}")
    if copy is not None and (copy.stride(0) != out.stride(0) or copy.shape != out.shape or copy.dtype != torch.bfloat16):
        raise ValueError(f"gemm: copy {tuple(copy.shape)} {copy.dtype}")
    f32 = a.dtype == torch.float32
    size = 0 if f32 or experts else _split_floats(m, n, k)
    ws = torch.empty(size, device=a.device) if size else None
    g = GemmRowsArgs(ptr(a), ptr(w), ptr(out), ptr(bias), ptr(mul), ptr(mul_row), ptr(tile_expert), ptr(copy), ptr(ws), size, m, n, k, a.stride(0), w.stride(0), out.stride(0),
                     OUT_TYPE[out.dtype], ACT[act], int(accumulate), experts, mul.stride(0) if mul is not None else 0, alpha, limit, ptr(tail), n - nt,
                     tail.stride(0) if nt else 0, *nums)
    _call("b2_gemm_rows_f32" if f32 else "b2_gemm_rows", g)


@functools.lru_cache(maxsize=4096)
def _split_floats(m: int, n: int, k: int) -> int:
    f = lib().b2_gemm_rows_scratch
    f.restype, f.argtypes = C.c_longlong, [I, I, I]
    return int(f(m, n, k))


NO_GATE = HeadGate(None, 0, 0)
NO_DIFF = DiffHeads(0.0, 0.0, 0.0, 0)


def head_gate(g: torch.Tensor, kind: str) -> HeadGate:
    """Rows ``g`` of gate values, before the sigmoid: "element" one for each result column, "head" one for each head."""
    return HeadGate(ptr(g), g.stride(0), {"element": 1, "head": 2}[kind])


def paged_append(qkv, *, heads, kv_heads, dim, vdim, q_norm, k_norm, eps, freqs, n_rot, positions, slots, table, q_out, k_cache, v_cache, head_norm=False, v_off=None,
                 mscale=1.0, maps=1, append=True, pdl=False) -> None:
    """Norm over the whole q / k projections (``head_norm``: over each head), rotation, q to padded fp32 rows [rows, H, dq], k and v (columns from ``v_off`` on) into
    the paged caches.  ``maps`` 2: differential attention, ``heads`` counts maps, a key head is two keys side by side and a query row has zeros beside its map's
    columns.  ``append`` False: queries only."""
    v_off = (heads + maps * kv_heads) * dim if v_off is None else v_off
    a = PagedAppendArgs(ptr(qkv), qkv.stride(0), heads, kv_heads, dim, vdim, ptr(q_norm), ptr(k_norm), eps, ptr(freqs), n_rot, ptr(positions), ptr(slots),
                        ptr(table), table.shape[1], ptr(q_out), q_out.shape[2], ptr(k_cache), ptr(v_cache), k_cache.shape[3], v_cache.shape[3], _is32(k_cache),
                        int(head_norm), v_off, mscale, maps, int(not append))
    _call("b2_paged_append", a, qkv.shape[0], int(pdl))


def paged_attn(q, k_cache, v_cache, positions, slots, table, out, *, dim, vdim, scale, softcap=0.0, chunk=0, window=0, keep=0, gate=NO_GATE, pdl=False) -> None:
    """Attention of any head size over a paged cache: q [rows, H, dq] fp32 -> out[row, h * vdim ...]."""
    a = PagedAttnArgs(ptr(q), q.shape[2], q.shape[1], k_cache.shape[1], dim, vdim, ptr(k_cache), ptr(v_cache), k_cache.shape[3], v_cache.shape[3], _is32(k_cache),
                      ptr(positions), ptr(slots), ptr(table), table.shape[1], chunk, scale, softcap, ptr(out), out.stride(0), 1 - _is32(out), window, keep, gate)
    _call("b2_paged_attn", a, q.shape[0], int(pdl))


def attn_prefill_paged(q, k_cache, v_cache, tiles, table, out, *, vdim, scale, softcap=0.0, chunk=0, window=0, keep=0, gate=NO_GATE, diff=NO_DIFF) -> None:
    """tcgen05 attention of query tiles ([n, 4] int32: first row, rows, slot, position) over a paged f16 cache of row length 64 or 128.  ``diff``: differential
    attention, the heads of ``q`` are maps and the tiles have up to 64 rows."""
    a = AttnPrefillArgs(ptr(q), ptr(k_cache), ptr(v_cache), ptr(out), None, q.shape[0], q.shape[1], k_cache.shape[1], 0, 0, 0, 0, 1, 0, scale, softcap, None, None)
    pg = AttnPagedArgs(ptr(tiles), ptr(table), table.shape[1], chunk, vdim, out.stride(0), window, keep, gate, diff)
    _check(lib().b2_attn_prefill_paged(C.byref(a), C.byref(pg), q.shape[2], tiles.shape[0], k_cache.shape[0], stream()), "attn_prefill_paged")


def attn_decode_paged(qkv, k_cache, v_cache, positions, slots, table, out, nb, *, heads, dim, vdim, q_norm, k_norm, eps, freqs, n_rot, scale, softcap,
                      chunk, n_splits, n_ctx, part_acc, part_ml, window=0, keep=0, head_norm=False, v_off=None, mscale=1.0, gate=NO_GATE, maps=1,
                      append=True, diff=NO_DIFF, pdl=False) -> bool:
    """Decode attention on raw projections: norms, rotation, cache append, split-K attention, merge, difference of maps and gate (``maps`` and ``append``:
    :func:`paged_append`).  False: shape not taken, nothing launched."""
    hd, G = k_cache.shape[3], k_cache.shape[1]
    v_off = (heads + maps * G) * dim if v_off is None else v_off
    a = AttnDecodeArgs(None, ptr(k_cache), ptr(v_cache), ptr(positions), ptr(slots), heads, G, n_ctx, n_splits, scale, softcap, window,
                       ptr(part_acc), ptr(part_ml), None, None, ptr(table), table.shape[1], chunk, keep)
    r = AttnRopeArgs(ptr(qkv), None, mscale, n_rot, 1, ptr(q_norm), ptr(k_norm), eps, qkv.stride(0), dim, vdim, ptr(freqs), int(head_norm), v_off, maps, int(not append))
    f = lib().b2_attn_decode_paged
    f.argtypes = [P, P, I, I, P, I, I, P, P, I, P]
    rc = f(C.addressof(a), C.addressof(r), nb, hd, ptr(out), out.stride(0), 1 - _is32(out), C.addressof(gate), C.addressof(diff), int(pdl), stream())
    if rc == 801:
        return False
    _check(rc, "attn_decode_paged")
    return True


def diff_rows(x: torch.Tensor, heads: int, vdim: int, diff, out: torch.Tensor, pdl: bool = False) -> None:
    """Results of both maps, ``x`` [rows, heads * 2 * vdim] fp32 -> the heads' results of differential attention."""
    f = lib().b2_diff_rows
    f.argtypes = [P, I, I, I, P, P, I, I, I, P]
    _check(f(ptr(x), x.shape[0], heads, vdim, C.addressof(diff), ptr(out), out.stride(0), 1 - _is32(out), int(pdl), stream()), "diff_rows")


def depth_rows(hist: torch.Tensor, n: int, w: torch.Tensor, k: int, eps: float, g: torch.Tensor | None = None, b: torch.Tensor | None = None,
               h: torch.Tensor | None = None, pdl: bool = False) -> torch.Tensor:
    """x = the sum of the first ``n`` blocks of ``hist`` [blocks, rows, columns] with weights ``w``, written to block ``n`` and returned; ``h`` = its layer norm."""
    x = hist[n]
    a = DepthRowsArgs(ptr(hist), hist.stride(0), ptr(w), n, k, hist.shape[2], ptr(x), ptr(g), ptr(b), ptr(h), h.stride(0) if h is not None else 0,
                      _is32(h) if h is not None else 0, eps)
    _call("b2_depth_rows", a, x.shape[0], int(pdl))
    return x


def gru_scan(x: torch.Tensor, off: int, state: torch.Tensor, segs: torch.Tensor, longest: int, out: torch.Tensor, pdl: bool = False) -> None:
    """Rows [z | u | gate], ``off`` columns apart, of prompt portions ``segs`` ([n, 4] int32: first row, rows, slot, position; ``longest``: the most rows of one) through the gated recurrence."""
    a = GruArgs(ptr(x), x.stride(0), off, 2 * off, state.shape[1], ptr(state), ptr(segs), None, None, ptr(out), out.stride(0))
    _call("b2_gru_scan", a, segs.shape[0], longest, _is32(x), int(pdl))


def gru_step(x: torch.Tensor, off: int, state: torch.Tensor, slots, positions, out: torch.Tensor, exact: bool = False, pdl: bool = False) -> None:
    """One token per sequence."""
    a = GruArgs(ptr(x), x.stride(0), off, 2 * off, state.shape[1], ptr(state), None, ptr(slots), ptr(positions), ptr(out), out.stride(0))
    _call("b2_gru_step", a, x.shape[0], _is32(x), int(exact), int(pdl))


def ssm_conv(xz, inner, w, b, state, slots, positions, offs, u, silu=True, shift=False, pdl=False) -> None:
    """Causal convolution over time of the first ``inner`` columns, each with ``w`` [taps, inner]; ``shift``: rows of one token per slot, which enter the state."""
    a = SsmConvArgs(ptr(xz), xz.stride(0), inner, w.shape[0], ptr(w), ptr(b), ptr(state), ptr(slots), ptr(positions), ptr(offs), ptr(u), u.stride(0), int(silu), int(shift))
    _call("b2_ssm_conv", a, xz.shape[0], _is32(xz), int(pdl))


def conv_keep(xz, inner, taps, state, segs, pdl=False) -> None:
    """The last taps - 1 rows of every portion (``segs`` [n, 4] int32: first row, rows, slot, position) become its slot's convolution state."""
    if taps > 1:
        a = ConvKeepArgs(ptr(xz), xz.stride(0), inner, taps, ptr(state), ptr(segs))
        _call("b2_conv_keep", a, segs.shape[0], _is32(xz), int(pdl))


def ssm_scan(xz, off_z, u, dt, bc, off_b, dt_bias, a2, d, taps, state, conv_state, segs, out, pdl=False) -> None:
    """``segs`` [n, 4] int32: first row, rows, slot, position of the first row."""
    a = SsmScanArgs(ptr(xz), xz.stride(0), off_z, ptr(u), u.stride(0), ptr(dt), dt.stride(0), ptr(bc), bc.stride(0), off_b, ptr(dt_bias), ptr(a2), ptr(d),
                    a2.shape[0], a2.shape[1], taps, ptr(state), ptr(conv_state), ptr(segs), ptr(out), out.stride(0))
    _call("b2_ssm_scan", a, segs.shape[0], _is32(u), int(pdl))


def ssm_step(xz, off_z, conv, p, off_b, w_dt, dt, dt_bias, a2, d, state, slots, positions, out, nb, exact=False, u=None, pdl=False) -> None:
    """One token per sequence.  ``dt``: projected step sizes, or None: projected inside from the first columns of ``p``.
    ``exact``: ``a2`` holds A instead of log2(e) A (32-bit models).  ``u``: convolved inputs, or None: formed inside."""
    a = SsmStepArgs(ptr(xz), xz.stride(0), off_z, 1 - _is32(xz), ptr(conv[0]), ptr(conv[1]), ptr(conv[2]), conv[0].shape[0], a2.shape[0], a2.shape[1],
                    ptr(p), p.stride(0), off_b, ptr(w_dt), w_dt.shape[1], _is32(w_dt), ptr(dt), dt.stride(0) if dt is not None else 0, ptr(dt_bias), ptr(a2),
                    ptr(d), ptr(state), ptr(slots), ptr(positions), ptr(out), out.stride(0), 1 - _is32(out), int(exact), ptr(u), u.stride(0) if u is not None else 0)
    _call("b2_ssm_step", a, nb, int(pdl))
