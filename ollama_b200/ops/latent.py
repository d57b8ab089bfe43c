"""Bindings of latent attention and of expert feed-forwards (kernels/latent.cu, attn_latent.cu, attn_prefill_tc.cu, moe.cu, moe_rows.cu)."""
from __future__ import annotations

import ctypes as C

import torch

from .cuda import ExpertGroups, MoeRouteArgs, _check, lib, ptr, stream
from .rows import ACT, GLU_BASE, F, I, P, _call, _is32, _st

LatentStepArgs = _st("LatentStepArgs", [("q", P), ("c", P), ("ldq", I), ("ldc", I), ("n_heads", I), ("dim", I), ("rot", I), ("rank", I), ("norm", P), ("eps", F), ("freqs", P),
                                        ("interleaved", I), ("rows", P), ("positions", P), ("slots", P), ("page_table", P), ("max_pages", I), ("cache", P),
                                        ("cp", I), ("w", I), ("cache32", I), ("append", I), ("uk", P), ("w32", I), ("q_out", P), ("dp", I), ("rp", I),
                                        ("mscale", F)])
LatentMergeArgs = _st("LatentMergeArgs", [("acc", P), ("ml", P), ("n_heads", I), ("splits", I), ("cp", I), ("vdim", I), ("uv", P), ("w32", I), ("rows", P),
                                          ("out", P), ("ldo", I), ("out16", I)])
LatentGatherArgs = _st("LatentGatherArgs", [("cache", P), ("cp", I), ("w", I), ("rot", I), ("seqs", P), ("page_table", P), ("max_pages", I), ("c", P), ("r", P),
                                            ("rp", I)])
LatentAttnArgs = _st("LatentAttnArgs", [("q", P), ("cache", P), ("rows", P), ("positions", P), ("slots", P), ("page_table", P), ("max_pages", I), ("n_heads", I),
                                        ("cp", I), ("w", I), ("splits", I), ("window", I), ("scale", F), ("acc", P), ("ml", P)])
AttnPartsArgs = _st("AttnPartsArgs", [("q", P), ("kv", P), ("shared", P), ("n_rows", I), ("dp", I), ("vp", I), ("rp", I), ("tiles", P), ("H", I), ("vdim", I),
                                      ("ldo", I), ("scale", F), ("out", P), ("window", I)])
MoeUpArgs = _st("MoeUpArgs", [("z", P), ("ldz", I), ("n_experts", I), ("top", I), ("h", P), ("ldh", I), ("k", I), ("w", P), ("n", I), ("wrows", I), ("ws", P),
                              ("ns", I), ("limit", F), ("limit_s", F), ("out", P), ("ldo", I), ("ffp", I), ("ids", P), ("wts", P),
                              ("correction", P), ("real", I), ("act", I), ("groups", ExpertGroups)])
MoeDownArgs = _st("MoeDownArgs", [("a", P), ("lda", I), ("top", I), ("ffp", I), ("sfp", I), ("ids", P), ("wts", P), ("w", P), ("ws", P), ("n", I), ("wrows", I),
                                  ("x", P), ("ldx", I), ("mult", F), ("store", I), ("real", I), ("h", P), ("ldh", I), ("gate", P), ("ldg", I)])

NOT_SUPPORTED = 801                # cudaErrorNotSupported: the launch does not take the shape, nothing ran


def _taken(name: str, args, *more) -> bool:
    rc = getattr(lib(), name)(C.byref(args), *more, stream())
    if rc == NOT_SUPPORTED:
        return False
    _check(rc, name)
    return True


def latent_step(q: torch.Tensor, c: torch.Tensor, n: int, *, heads: int, dim: int, rot: int, rank: int, norm, eps: float, freqs, interleaved: bool, positions, slots, table,
                cache: torch.Tensor, cp: int, q_out: torch.Tensor, rows=None, append: bool = True, uk: torch.Tensor | None = None, dp: int = 0, rp: int = 0,
                mscale: float = 1.0, pdl: bool = False) -> None:
    """Of ``n`` rows (queries ``q``, latents with rotated key parts behind them ``c``): latent and rotated key part into the cache (``append``), and the queries taken into the latent space by ``uk`` [heads, dim, cp] ->
    ``q_out`` [n, heads, w] in the cache's type; without ``uk`` the queries as they are, rotated, each part padded: [n, heads, dp + rp] f16."""
    a = LatentStepArgs(ptr(q), ptr(c), q.stride(0), c.stride(0), heads, dim, rot, rank, ptr(norm), eps, ptr(freqs), int(interleaved), ptr(rows), ptr(positions), ptr(slots), ptr(table),
                       table.shape[1], ptr(cache), cp, cache.shape[-1], _is32(cache), int(append), ptr(uk), _is32(uk) if uk is not None else 0, ptr(q_out), dp, rp, mscale)
    _call("b2_latent_step", a, n, int(pdl))


def latent_merge(acc: torch.Tensor, ml: torch.Tensor | None, n: int, uv: torch.Tensor, out: torch.Tensor, *, heads: int, splits: int, cp: int, vdim: int, rows=None,
                 merged: torch.Tensor | None = None, pdl: bool = False) -> None:
    """Split results [n, heads, splits, cp] merged and multiplied by ``uv`` [heads * vdim, cp] into rows of ``out``.  ``merged``: bf16 scratch [n, heads, cp] for
    the two-launch form, whose product runs on the tensor cores."""
    a = LatentMergeArgs(ptr(acc), ptr(ml), heads, splits, cp, vdim, ptr(uv), _is32(uv), ptr(rows), ptr(out), out.stride(0), 1 - _is32(out))
    _call("b2_latent_merge", a, n, C.c_void_p(ptr(merged)), int(pdl))


def attn_latent(q: torch.Tensor, n: int, cache: torch.Tensor, acc, ml, *, heads: int, cp: int, scale: float, splits: int, positions, slots, table, rows=None,
                window: int = 0, pdl: bool = False) -> bool:
    """Scores and sums of absorbed queries over the cache (``window`` > 0: its last positions up to the query's own); False: shape not taken, nothing launched."""
    a = LatentAttnArgs(ptr(q), ptr(cache), ptr(rows), ptr(positions), ptr(slots), ptr(table), table.shape[1], heads, cp, cache.shape[-1], splits, window, scale, ptr(acc), ptr(ml))
    return _taken("b2_attn_latent", a, n, int(pdl))


def latent_gather(cache: torch.Tensor, cp: int, rot: int, seqs: torch.Tensor, max_len: int, table, c: torch.Tensor, r: torch.Tensor) -> None:
    """Positions of several sequences side by side: latents to bf16 rows ``c``, rotated key parts to ``r``.  ``seqs`` [n, 4] int32: row of position 0, end of the
    positions, slot, first position; ``max_len``: the most positions of one."""
    a = LatentGatherArgs(ptr(cache), cp, cache.shape[-1], rot, ptr(seqs), ptr(table), table.shape[1], ptr(c), ptr(r), r.shape[1])
    _call("b2_latent_gather", a, seqs.shape[0], max_len)


def parts_supported(dp: int, rp: int, vp: int) -> bool:
    return (vp, dp + rp) in ((64, 64), (64, 128), (64, 192), (128, 128), (128, 192))


def attn_prefill_parts(q: torch.Tensor, kv: torch.Tensor, shared: torch.Tensor, tiles: torch.Tensor, out: torch.Tensor, *, heads: int, dp: int, vp: int, rp: int,
                       vdim: int, scale: float, window: int = 0) -> None:
    """tcgen05 attention of query tiles ([n, 4] int32: first row, rows, buffer row of position 0, position) over keys in two parts.  With a ``window`` the buffer
    needs the positions from the tiles' first windows on, from multiples of 128."""
    a = AttnPartsArgs(ptr(q), ptr(kv), ptr(shared) if rp else None, kv.shape[0], dp, vp, rp, ptr(tiles), heads, vdim, out.stride(0), scale, ptr(out), window)
    _call("b2_attn_prefill_parts", a, tiles.shape[0])


NO_GROUPS = ExpertGroups(0, 0, 0.0)


def moe_route(z: torch.Tensor, outputs: int, top: int, experts: int | None = None, correction: torch.Tensor | None = None, groups: ExpertGroups = NO_GROUPS) -> tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    """Router outputs [rows, top] chosen by logits ``z``, the same with -1 for those that are no experts, and their weights: the largest logits and the softmax over those,
    or with a ``correction`` the largest of softmax + correction and that softmax; with ``groups`` the largest of sigmoid + correction in the best groups and the
    normalised sigmoids, times the groups' scale."""
    n = z.shape[0]
    ids, lids = torch.empty(2, n, top, device=z.device, dtype=torch.int32)
    wts = torch.empty(n, top, device=z.device)
    a = MoeRouteArgs(ptr(z), z.stride(0), outputs, top, 3 if groups.count else 1 if correction is None else 2, 0, 0, outputs if experts is None else experts, ptr(ids), ptr(lids), ptr(wts), ptr(correction), groups)
    _call("b2_moe_route", a, n, 0)
    return ids, lids, wts


def moe_up_rows(z: torch.Tensor, h: torch.Tensor, nb: int, w: torch.Tensor, n: int, out: torch.Tensor, ids: torch.Tensor, wts: torch.Tensor, *, experts: int, top: int,
                ffp: int, limit: float, ws: torch.Tensor | None = None, ns: int = 0, limit_s: float = 0.0, act: str = "glu:swiglu_oai", outputs: int | None = None,
                correction: torch.Tensor | None = None, groups: ExpertGroups = NO_GROUPS, pdl: bool = False) -> None:
    """Hidden columns of the chosen experts (and of the shared one, ``ws``) of up to four rows; ``w`` [experts, rows, k] with gate / up interleaved.  The choice is
    that of :func:`moe_route` among ``outputs`` router outputs."""
    a = MoeUpArgs(ptr(z), z.stride(0), experts if outputs is None else outputs, top, ptr(h), h.stride(0), w.shape[2], ptr(w), n, w.shape[1], ptr(ws), ns, limit, limit_s, ptr(out),
                  out.stride(0), ffp, ptr(ids), ptr(wts), ptr(correction), experts, ACT[act] - GLU_BASE, groups)
    _call("b2_moe_up_rows", a, nb, _is32(w), int(pdl))


def moe_down_rows(a_rows: torch.Tensor, nb: int, ids, wts, w: torch.Tensor, x: torch.Tensor, *, top: int, n: int, mult: float, ws: torch.Tensor | None = None,
                  store: bool = False, h: torch.Tensor | None = None, gate: torch.Tensor | None = None, pdl: bool = False) -> None:
    """x += mult * (sum of weight * w[id] a over the chosen experts, plus the shared expert's product); ``w`` [experts, rows, ffp].  Choices beyond the experts are the
    input ``h`` itself; ``gate`` [rows, 1]: the shared expert's product is multiplied by its sigmoid; ``store``: the result replaces x."""
    a = MoeDownArgs(ptr(a_rows), a_rows.stride(0), top, w.shape[2], ws.shape[1] if ws is not None else 0, ptr(ids), ptr(wts), ptr(w), ptr(ws), n, w.shape[1], ptr(x),
                    x.stride(0), mult, int(store), w.shape[0], ptr(h), h.stride(0) if h is not None else 0, ptr(gate), gate.stride(0) if gate is not None else 0)
    _call("b2_moe_down_rows", a, nb, _is32(w), int(pdl))
