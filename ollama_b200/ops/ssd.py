"""Bindings of the state-space mixer with one decay per head (kernels/ssd.cu)."""
from __future__ import annotations

import torch

from .cuda import ptr
from .rows import F, I, P, _call, _is32, _st

MAX_STATE = 256
SsdArgs = _st("SsdArgs", [("u", P), ("ldu", I), ("off_b", I), ("off_c", I), ("z", P), ("ldz", I), ("dt", P), ("lddt", I), ("dt_bias", P), ("a", P), ("d", P), ("heads", I),
                          ("groups", I), ("vdim", I), ("n_state", I), ("state", P), ("seg", P), ("slots", P), ("positions", P), ("out", P), ("ldo", I)])
GroupNormArgs = _st("GroupNormArgs", [("x", P), ("ldx", I), ("heads", I), ("vdim", I), ("vp", I), ("groups", I), ("w", P), ("eps", F)])


def _args(u, off_b, off_c, z, dt, dt_bias, a, d, groups, state, out, seg=None, slots=None, positions=None):
    _, heads, vdim, n = state.shape
    return SsdArgs(ptr(u), u.stride(0), off_b, off_c, ptr(z), z.stride(0), ptr(dt), dt.stride(0), ptr(dt_bias), ptr(a), ptr(d), heads, groups, vdim, n, ptr(state), ptr(seg),
                   ptr(slots), ptr(positions), ptr(out), out.stride(0))


def ssd_scan(u, off_b: int, off_c: int, z, dt, dt_bias, a, d, groups: int, state, segs, out, pdl: bool = False) -> None:
    """Prompt portions ``segs`` ([n, 4] int32: first row, rows, slot, position).  ``state`` [slots, heads, vdim, n_state]; ``out`` = (scan + D x) silu(z)."""
    _call("b2_ssd_scan", _args(u, off_b, off_c, z, dt, dt_bias, a, d, groups, state, out, seg=segs), segs.shape[0], _is32(u), int(pdl))


def ssd_step(u, off_b: int, off_c: int, z, dt, dt_bias, a, d, groups: int, state, slots, positions, out, pdl: bool = False) -> None:
    """One token per sequence."""
    _call("b2_ssd_step", _args(u, off_b, off_c, z, dt, dt_bias, a, d, groups, state, out, slots=slots, positions=positions), u.shape[0], _is32(u), int(pdl))


def group_norm(x, heads: int, vdim: int, vp: int, groups: int, w, eps: float, pdl: bool = False) -> None:
    """Every one of ``groups`` equal parts of a row of ``heads`` times ``vdim`` values (heads ``vp`` columns apart) over its own root mean square, times ``w``; in place."""
    _call("b2_group_norm", GroupNormArgs(ptr(x), x.stride(0), heads, vdim, vp, groups, ptr(w), eps), x.shape[0], _is32(x), int(pdl))
