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
STACK_ARCHS = {"Vazatar": "vazatar", "Kavenex": "kavenex"}


@dataclass(frozen=True)
class Design:
    """What a design fixes for all its models."""
    parallel: bool                    # mixer and feed-forward read the same stream (two norms of one input) / one after the other
    norm: str                         # "rms_one_plus": RMS norm with weights stored as an offset from 1; "layer": layer norm with bias
    loop_join: str                    # "product": a pass begins with a matrix over [stream | embedding output]; "add": with sums of vectors
    ff_act: str                       # activation of dense feed-forwards
    interleaved: bool                 # rotary pairs are (2i, 2i + 1), otherwise (i, i + dims / 2)


DESIGNS = {"Vazatar": Design(True, "rms_one_plus", "product", "relu2", False),
           "Kavenex": Design(False, "layer", "add", "gelu_tanh", True)}
GATED_ACTS = ("gelu_tanh", "swiglu_oai")
SWIGLU_ALPHA = 1.702                  # sigmoid slope of the clamped gated unit


@dataclass(frozen=True)
class Rotation:
    """Rotary embedding of the first ``dims`` dimensions, in the half-split order or interleaved.  ``scaling`` (factor, low, high, original): frequencies
    of wavelengths beyond original / low are divided by factor, those below original / high kept, blended in between."""
    dims: int
    base: float
    scaling: tuple[float, float, float, float] | None = None
    interleaved: bool = False

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
class LatentMixer:
    """Attention whose keys and values are products of one latent vector per position: the cache holds the latent and a rotated key part
    that all heads share."""
    heads: int
    dim: int                          # unrotated query / key dimensions of a head
    rot_dim: int                      # rotated ones
    vdim: int
    kv_rank: int                      # size of the latent
    scale: float
    rot: Rotation | None


@dataclass(frozen=True)
class MambaMixer:
    inner: int
    state: int
    dt_rank: int
    conv: int                         # taps of the causal convolution


Mixer = AttentionMixer | LatentMixer | MambaMixer


@dataclass(frozen=True)
class DenseMLP:
    ff: int
    act: str = "relu2"

    @property
    def gated(self) -> bool:
        return self.act in GATED_ACTS


@dataclass(frozen=True)
class Expert:
    """Gated feed-forward min(g, limit) sigmoid(1.702 min(g, limit)) (clamp(u, -limit, limit) + 1)."""
    ff: int
    limit: float = math.inf


@dataclass(frozen=True)
class ExpertMLP:
    """``top`` of ``experts`` feed-forwards per token, weighted by the softmax over the chosen router logits; ``shared`` runs for every token."""
    experts: int
    top: int
    expert: Expert
    shared: Expert | None = None


@dataclass(frozen=True)
class StackLayer:
    mixer: Mixer
    mlp: DenseMLP | ExpertMLP | None


@dataclass(frozen=True)
class LayerRun:
    layer: int                        # whose weights
    joins: bool                       # this run begins a pass of the loop: the stream is joined with the embedding output (or a step vector) first
    turn: int = 0                     # number of the pass


@dataclass(frozen=True)
class Stack:
    layers: tuple[StackLayer, ...]
    loop: tuple[int, int, int] | None     # start, stop, times
    embed_scale: float
    eps: float
    width: int
    vocab: int
    logit_softcap: float = 0.0
    design: Design = DESIGNS["Vazatar"]
    residual_mult: float = 1.0
    side_dim: int = 0                 # > 0: every layer adds an input of its own per token, a vector of this size

    def runs(self) -> list[LayerRun]:
        """Layer runs in order; each has a cache or state of its own."""
        if self.loop is None:
            return [LayerRun(i, False) for i in range(len(self.layers))]
        lo, hi, times = self.loop
        return ([LayerRun(i, False) for i in range(lo)] + [LayerRun(i, i == lo, t) for t in range(times) for i in range(lo, hi)]
                + [LayerRun(i, False) for i in range(hi, len(self.layers))])

    def kv_bytes_per_token(self, elem_bytes: int = 2) -> int:
        """Cache bytes of one position over all layer runs."""
        ms = [self.layers[r.layer].mixer for r in self.runs()]
        return (sum(m.kv_heads * (m.dim + m.vdim) for m in ms if isinstance(m, AttentionMixer))
                + sum(m.kv_rank + m.rot_dim for m in ms if isinstance(m, LatentMixer))) * elem_bytes

    def state_bytes(self) -> int:
        """Recurrent state of one sequence over all layer runs (fp32)."""
        ms = [self.layers[r.layer].mixer for r in self.runs()]
        return sum(4 * m.inner * (m.state + m.conv - 1) for m in ms if isinstance(m, MambaMixer))

    @property
    def recurrent(self) -> bool:
        return any(isinstance(L.mixer, MambaMixer) for L in self.layers)


def _rotation(r: dict[str, Any] | None, dim: int, interleaved: bool = False) -> Rotation | None:
    if not r or not r.get("dims"):
        return None
    dims = int(r["dims"])
    if dims % 2 or not 0 < dims <= dim:
        raise ValueError(f"rotary embedding of {dims} of {dim} dimensions")
    s = r.get("scaling")
    return Rotation(dims, float(r["base"]), tuple(float(s[k]) for k in ("factor", "low", "high", "original")) if s else None, interleaved)


def _mixer(kind: str, m: dict[str, Any], design: Design) -> Mixer:
    if kind == "attention":
        H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
        if G < 1 or H % G:
            raise ValueError(f"{H} query heads on {G} key/value heads")
        return AttentionMixer(H, G, d, int(m.get("vdim") or d), float(m["scale"]), float(m.get("softcap") or 0.0),
                              int((m.get("mask") or {}).get("size") or 0), _rotation(m.get("rot"), d, design.interleaved))
    if kind == "latent_attention":
        r = int(m.get("rot_dim") or 0)
        rot = _rotation({**(m.get("rot") or {}), "dims": r}, r, design.interleaved) if r else None
        return LatentMixer(int(m["heads"]), int(m["dim"]), r, int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]), rot)
    if kind == "mamba1":
        return MambaMixer(int(m["inner"]), int(m["state"]), int(m["dt_rank"]), int(m["conv"]))
    raise NotImplementedError(f"unknown mixer {kind!r}")


def _expert(m: dict[str, Any]) -> Expert:
    limit = m.get("limit")
    return Expert(int(m["ff"]), math.inf if limit is None else float(limit))


def _mlp(m: dict[str, Any] | None, design: Design) -> DenseMLP | ExpertMLP | None:
    if m is None:
        return None
    kind = m.get("kind", "dense")
    if kind == "dense":
        return DenseMLP(int(m["ff"]), design.ff_act)
    if kind == "moe":
        n, top = int(m["router"]["experts"]), int(m["router"]["top"])
        if not 0 < top <= n:
            raise ValueError(f"{top} of {n} experts")
        return ExpertMLP(n, top, _expert(m["expert"]), _expert(m["shared"]) if m.get("shared") else None)
    raise NotImplementedError(f"unknown feed-forward {kind!r}")


def parse_stack(cfg: dict[str, Any] | str) -> Stack:
    """``config.json`` of a stack checkpoint (a dictionary, or its JSON text) -> :class:`Stack`."""
    if isinstance(cfg, str):
        cfg = json.loads(cfg)
    design = DESIGNS[cfg["architecture"]]
    layers = tuple(StackLayer(_mixer(L["type"], L["mixer"], design), _mlp(L.get("mlp"), design)) for L in cfg["layers"])
    loop = cfg.get("loop")
    if loop:
        loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
            raise ValueError(f"loop {loop} over {len(layers)} layers")
    scale, mult = (cfg.get("embedding") or {}).get("scale"), cfg.get("residual_mult")
    return Stack(layers, loop or None, 1.0 if scale is None else float(scale), float(cfg["norm"]["eps"]), int(cfg["width"]), int(cfg["vocab"]),
                 float(cfg.get("logit_softcap") or 0.0), design, 1.0 if mult is None else float(mult), int((cfg.get("token_side") or {}).get("dim") or 0))
