"""Decoder stacks whose layers differ from each other: every layer names its token mixer and its feed-forward, and a span of
layers may run several times in a row with the same weights.

The description is parsed from a checkpoint's ``config.json`` (kept as one JSON string in GGUF metadata).  Constants are fields of
the mechanisms, so that another design can combine them differently.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass
from typing import Any

# checkpoint "architecture" -> GGUF architecture of the designs described this way
STACK_ARCHS = {"Vazatar": "vazatar"}


@dataclass(frozen=True)
class Rotation:
    """Rotary embedding of the first ``dims`` dimensions in the half-split order.  ``scaling`` (factor, low, high, original): frequencies
    of wavelengths beyond original / low are divided by factor, those below original / high kept, blended in between."""
    dims: int
    base: float
    scaling: tuple[float, float, float, float] | None = None

    def freqs(self) -> list[float]:
        out = []
        for i in range(self.dims // 2):
            f = self.base ** (-2.0 * i / self.dims)
            if self.scaling is not None:
                factor, low, high, original = self.scaling
                wave = 2.0 * math.pi / f
                if wave > original / low:
                    f /= factor
                elif wave >= original / high:
                    s = (original / wave - low) / (high - low)
                    f = (1.0 - s) * f / factor + s * f
            out.append(f)
        return out


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float = 0.0
    chunk: int = 0                    # > 0: position p sees the keys from floor(p / chunk) * chunk on
    rot: Rotation | None = None


@dataclass(frozen=True)
class MambaMixer:
    inner: int
    state: int
    dt_rank: int
    conv: int                         # taps of the causal convolution


@dataclass(frozen=True)
class DenseMLP:
    ff: int
    act: str = "relu2"


@dataclass(frozen=True)
class StackLayer:
    mixer: AttentionMixer | MambaMixer
    mlp: DenseMLP | None


@dataclass(frozen=True)
class LayerRun:
    layer: int                        # whose weights
    joins: bool                       # the stream is joined with the embedding output before this run


@dataclass(frozen=True)
class Stack:
    layers: tuple[StackLayer, ...]
    loop: tuple[int, int, int] | None     # start, stop, times
    embed_scale: float
    eps: float
    width: int
    vocab: int
    logit_softcap: float = 0.0

    def runs(self) -> list[LayerRun]:
        """Layer runs in order; each has a cache or state of its own."""
        if self.loop is None:
            return [LayerRun(i, False) for i in range(len(self.layers))]
        lo, hi, times = self.loop
        return ([LayerRun(i, False) for i in range(lo)] + [LayerRun(i, i == lo) for _ in range(times) for i in range(lo, hi)]
                + [LayerRun(i, False) for i in range(hi, len(self.layers))])

    def kv_bytes_per_token(self, elem_bytes: int = 2) -> int:
        """Cache bytes of one position over all layer runs."""
        ms = [self.layers[r.layer].mixer for r in self.runs()]
        return sum(m.kv_heads * (m.dim + m.vdim) for m in ms if isinstance(m, AttentionMixer)) * elem_bytes

    def state_bytes(self) -> int:
        """Recurrent state of one sequence over all layer runs (fp32)."""
        ms = [self.layers[r.layer].mixer for r in self.runs()]
        return sum(4 * m.inner * (m.state + m.conv - 1) for m in ms if isinstance(m, MambaMixer))

    @property
    def recurrent(self) -> bool:
        return any(isinstance(L.mixer, MambaMixer) for L in self.layers)


def _rotation(r: dict[str, Any] | None, dim: int) -> Rotation | None:
    if not r or not r.get("dims"):
        return None
    dims = int(r["dims"])
    if dims % 2 or not 0 < dims <= dim:
        raise ValueError(f"rotary embedding of {dims} of {dim} dimensions")
    s = r.get("scaling")
    return Rotation(dims, float(r["base"]), tuple(float(s[k]) for k in ("factor", "low", "high", "original")) if s else None)


def _mixer(kind: str, m: dict[str, Any]) -> AttentionMixer | MambaMixer:
    if kind == "attention":
        H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
        if G < 1 or H % G:
            raise ValueError(f"{H} query heads on {G} key/value heads")
        return AttentionMixer(H, G, d, int(m.get("vdim") or d), float(m["scale"]), float(m.get("softcap") or 0.0),
                              int((m.get("mask") or {}).get("size") or 0), _rotation(m.get("rot"), d))
    if kind == "mamba1":
        return MambaMixer(int(m["inner"]), int(m["state"]), int(m["dt_rank"]), int(m["conv"]))
    raise NotImplementedError(f"unknown mixer {kind!r}")


def _mlp(m: dict[str, Any] | None) -> DenseMLP | None:
    if m is None:
        return None
    if m.get("kind", "dense") != "dense":
        raise NotImplementedError(f"unknown feed-forward {m.get('kind')!r}")
    return DenseMLP(int(m["ff"]))


def parse_stack(cfg: dict[str, Any] | str) -> Stack:
    """``config.json`` of a stack checkpoint (a dictionary, or its JSON text) -> :class:`Stack`."""
    if isinstance(cfg, str):
        cfg = json.loads(cfg)
    layers = tuple(StackLayer(_mixer(L["type"], L["mixer"]), _mlp(L.get("mlp"))) for L in cfg["layers"])
    loop = cfg.get("loop")
    if loop:
        loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
            raise ValueError(f"loop {loop} over {len(layers)} layers")
    return Stack(layers, loop or None, float((cfg.get("embedding") or {}).get("scale") or 1.0), float(cfg["norm"]["eps"]), int(cfg["width"]),
                 int(cfg["vocab"]), float(cfg.get("logit_softcap") or 0.0))
