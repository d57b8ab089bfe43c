"""Decoder stacks whose layers differ from each other: every layer names its token mixer and its feed-forward, and a span of
layers may run several times in a row with the same weights.

The description is parsed from a checkpoint's ``config.json`` (kept as one JSON string in GGUF metadata).  Constants are fields of
the mechanisms, so that another design can combine them differently.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field
from typing import Any

# checkpoint "architecture" -> GGUF architecture of the designs described this way
STACK_ARCHS = {"Vazatar": "vazatar", "Kavenex": "kavenex", "Tirudra": "tirudra", "Rinirax": "rinirax"}


@dataclass(frozen=True)
class Design:
    """What a design fixes for all its models."""
    parallel: bool                    # mixer and feed-forward read the same stream (two norms of one input, or one) / one after the other
    norm: str                         # "rms_one_plus": RMS norm with weights stored as an offset from 1; "layer": layer norm with bias
    loop_join: str                    # "product": a pass begins with a matrix over [stream | embedding output]; "add": with sums of vectors
    ff_act: str                       # activation of dense feed-forwards
    interleaved: bool                 # rotary pairs are (2i, 2i + 1), otherwise (i, i + dims / 2)
    post_norm: bool = False           # the result of a mixer or feed-forward is normalised before it is added to the stream
    mixers: dict[str, dict] = field(default_factory=dict)     # mixer name -> fields of its class that its configuration does not give
    experts: dict[str, Any] = field(default_factory=dict)     # the same of ExpertMLP
    shared_norm: bool = False         # parallel parts read one norm
    depth_average: bool = False       # what goes on to the next layer is a weighted sum of the embedding output and all layers' results so far

    @property
    def paired(self) -> bool:
        """Parallel parts behind two norms of their own."""
        return self.parallel and not self.shared_norm


DESIGNS = {"Vazatar": Design(True, "rms_one_plus", "product", "relu2", False, mixers={"attention": {"qk_norm": "row", "mask": "chunk"}}),
           "Kavenex": Design(False, "layer", "add", "gelu_tanh", True, experts={"act": "swiglu_oai", "scoring": "chosen"}),
           "Tirudra": Design(False, "rms_one_plus", "", "", False, post_norm=True,
                             mixers={"attention": {"qk_norm": "head", "mask": "window", "gate": "element"},
                                     "attention_2": {"qk_norm": "head", "mask": "window", "gate": "head", "bias": "qk", "keys_as_values": True}},
                             experts={"act": "silu", "scoring": "all", "router_bias": False, "correction": True, "shared_gate": True}),
           "Rinirax": Design(True, "layer", "", "xielu", False, shared_norm=True, depth_average=True,
                             mixers={"attention": {"qk_norm": "", "maps": 2, "bias": "qkv", "interleaved": True}},
                             experts={"act": "silu", "scoring": "sigmoid", "router_bias": False, "correction": True})}
GATED_ACTS = ("gelu_tanh", "swiglu_oai")
SWIGLU_ALPHA = 1.702                  # sigmoid slope of the clamped gated unit


@dataclass(frozen=True)
class Rotation:
    """Rotary embedding of the first ``dims`` dimensions, in the half-split order or interleaved.  ``scaling`` (factor, low, high, original): frequencies
    of wavelengths beyond original / low are divided by factor, those below original / high kept, blended in between.  ``yarn`` (factor, original, fast,
    slow): pairs that turn at least ``fast`` times within ``original`` positions keep their frequency, those that turn at most ``slow`` times have it divided by
    factor, with a ramp over the pair's index in between, and the rotated vectors grow by ``magnitude``."""
    dims: int
    base: float
    scaling: tuple[float, float, float, float] | None = None
    interleaved: bool = False
    yarn: tuple[float, float, float, float] | None = None

    @property
    def magnitude(self) -> float:
        return 1.0 if self.yarn is None else 0.1 * math.log(self.yarn[0]) + 1.0

    def _ramp(self) -> tuple[float, float]:
        """First and last pair index of the ramp."""
        _, original, fast, slow = self.yarn

        def index(turns: float) -> float:
            return self.dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))
        return max(math.floor(index(fast)), 0), min(math.ceil(index(slow)), self.dims - 1)

    def freqs(self) -> list[float]:
        out = []
        lo, hi = self._ramp() if self.yarn is not None else (0, 0)
        for i in range(self.dims // 2):
            f = self.base ** (-2.0 * i / self.dims)
            if self.yarn is not None:
                r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
                f = f / self.yarn[0] * r + f * (1.0 - r)
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
    qk_norm: str = "row"              # RMS norm of queries and keys: "row" over the whole projection, "head" over each head with one weight vector for all, "" none
    window: int = 0                   # > 0: position p sees the keys from p - window + 1 on,
    keep: int = 0                     # and the first ``keep`` keys of the sequence
    conv: int = 0                     # > 0: taps of a causal convolution over time on every channel of q, k and v
    gate: str = ""                    # sigmoid gate of the heads' results: "element", "head" (one number each) or none
    bias: str = ""                    # projections that have one: letters of q, k, v
    keys_as_values: bool = False      # the values are the projected keys, before norm and rotation
    maps: int = 1                     # 2: differential attention.  A head has two queries and keys of ``dim``, one after the other, each with a softmax of its own over the
    diff: float = 0.0                 # same values; the result is their difference under an RMS norm, times 1 - ``diff``
    kv_from: int | None = None        # the layer whose cached keys and values are used instead of own ones

    @property
    def n_q(self) -> int:
        return self.heads * self.maps * self.dim

    @property
    def n_k(self) -> int:
        """Columns of this layer's own key projection."""
        return 0 if self.kv_from is not None else self.kv_heads * self.maps * self.dim

    @property
    def n_v(self) -> int:
        return 0 if self.keys_as_values or self.kv_from is not None else self.kv_heads * self.vdim

    @property
    def n_gate(self) -> int:
        return {"element": self.heads * self.vdim, "head": self.heads, "": 0}[self.gate]


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
    q_rank: int = 0                   # > 0: queries are products of a latent of this size too
    window: int = 0                   # > 0: position p sees the keys from p - window + 1 on


@dataclass(frozen=True)
class GruMixer:
    """Gated recurrence of ``width`` channels whose gates read the current token only: S <- (1 - z) S + z c."""
    width: int


@dataclass(frozen=True)
class MambaMixer:
    inner: int
    state: int
    dt_rank: int
    conv: int                         # taps of the causal convolution


@dataclass(frozen=True)
class Mamba2Mixer:
    """State-space mixer with one decay per head: a state of [vdim, state] per head, B and C shared by the heads of a group; the gated result is
    normalised in ``norm_groups`` equal parts."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Of the convolution."""
        return self.inner + 2 * self.groups * self.state


Mixer = AttentionMixer | LatentMixer | GruMixer | MambaMixer | Mamba2Mixer


@dataclass(frozen=True)
class DenseMLP:
    ff: int
    act: str = "relu2"

    @property
    def gated(self) -> bool:
        return self.act in GATED_ACTS


@dataclass(frozen=True)
class Expert:
    """One expert's hidden size, and the limit of gate and up where its activation has one."""
    ff: int
    limit: float = math.inf


@dataclass(frozen=True)
class ExpertMLP:
    """``top`` of ``experts`` feed-forwards per token; ``shared`` runs for every token.  Activations: "swiglu_oai" is min(g, limit) sigmoid(1.702 min(g, limit))
    (clamp(u, -limit, limit) + 1), "silu" g sigmoid(g) u.  Scoring "chosen": the largest router logits, weighted by the softmax over those alone; "all": the largest of
    softmax plus ``correction``, weighted by the softmax over all outputs as it is; "sigmoid": the largest of sigmoid plus ``correction`` among the ``keep`` best of
    ``groups`` equal groups of neighbours (a group is worth its two best), weighted by the chosen sigmoids over their sum, times ``scale``."""
    experts: int
    top: int
    expert: Expert
    shared: Expert | None = None
    act: str = "swiglu_oai"
    scoring: str = "chosen"
    router_bias: bool = True
    correction: bool = False          # a vector that is added for the choice only
    shared_gate: bool = False         # the shared expert is multiplied by the sigmoid of a number per token
    identity: int = 0                 # router outputs behind the experts' that stand for the input itself
    groups: int = 1
    keep: int = 1
    scale: float = 1.0

    @property
    def outputs(self) -> int:
        """Of the router."""
        return self.experts + self.identity


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
    logit_scale: float = 1.0

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
        return (sum(m.kv_heads * (m.maps * m.dim + m.vdim) for m in ms if isinstance(m, AttentionMixer) and m.kv_from is None)
                + sum(m.kv_rank + m.rot_dim for m in ms if isinstance(m, LatentMixer))) * elem_bytes

    def state_bytes(self) -> int:
        """Recurrent state of one sequence over all layer runs (fp32)."""
        ms = [self.layers[r.layer].mixer for r in self.runs()]
        return 4 * (sum(m.inner * (m.state + m.conv - 1) for m in ms if isinstance(m, MambaMixer)) + sum(m.width for m in ms if isinstance(m, GruMixer))
                    + sum(m.inner * m.state + m.channels * (m.conv - 1) for m in ms if isinstance(m, Mamba2Mixer))
                    + sum((m.n_q + m.n_k + m.n_v) * (m.conv - 1) for m in ms if isinstance(m, AttentionMixer) and m.conv))

    @property
    def recurrent(self) -> bool:
        """Whether a sequence has state besides its cached keys and values: a prefix of it cannot be taken up again in the middle."""
        return any(isinstance(L.mixer, (GruMixer, MambaMixer, Mamba2Mixer)) or (isinstance(L.mixer, AttentionMixer) and L.mixer.conv > 1) for L in self.layers)


def _rotation(r: dict[str, Any] | None, dim: int, interleaved: bool = False) -> Rotation | None:
    if not r or not r.get("dims"):
        return None
    dims = int(r["dims"])
    if dims % 2 or not 0 < dims <= dim:
        raise ValueError(f"rotary embedding of {dims} of {dim} dimensions")
    s = r.get("scaling")
    if s and "fast" in s:
        return Rotation(dims, float(r["base"]), None, interleaved, tuple(float(s[k]) for k in ("factor", "original", "fast", "slow")))
    return Rotation(dims, float(r["base"]), tuple(float(s[k]) for k in ("factor", "low", "high", "original")) if s else None, interleaved)


def _mixer(kind: str, m: dict[str, Any], design: Design) -> Mixer:
    if kind in design.mixers and kind.startswith("attention"):
        H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
        if G < 1 or H % G:
            raise ValueError(f"{H} query heads on {G} key/value heads")
        fixed = dict(design.mixers[kind])
        mask, keys, pairs = m.get("mask") or {}, fixed.get("keys_as_values", False), fixed.pop("interleaved", design.interleaved)
        vdim, span = int(m.get("vdim") or d), {fixed.pop("mask"): int(mask.get("size") or 0)} if "mask" in fixed else {}
        if fixed.get("maps", 1) > 1:
            fixed["diff"] = float(m["diff"])
        if m.get("kv_from") is not None:
            fixed["kv_from"] = int(m["kv_from"])
        if keys and vdim != d:
            raise ValueError(f"values of {vdim} dimensions that are keys of {d}")
        return AttentionMixer(H, G, d, vdim, float(m["scale"]), float(m.get("softcap") or 0.0), rot=_rotation(m.get("rot"), d, pairs),
                              keep=int(mask.get("keep_first") or 0), conv=int(m.get("conv") or 0), **span, **fixed)
    if kind == "latent_attention":
        r = int(m.get("rot_dim") or 0)
        rot = _rotation({**(m.get("rot") or {}), "dims": r}, r, design.interleaved) if r else None
        return LatentMixer(int(m["heads"]), int(m["dim"]), r, int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]), rot, int(m.get("q_rank") or 0),
                           int((m.get("mask") or {}).get("size") or 0))
    if kind == "mingru":
        return GruMixer(int(m["width"]))
    if kind == "mamba1":
        return MambaMixer(int(m["inner"]), int(m["state"]), int(m["dt_rank"]), int(m["conv"]))
    if kind == "mamba2":
        mix = Mamba2Mixer(int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["conv"]), int(m.get("norm_groups") or 1))
        if mix.heads % mix.groups or mix.inner % mix.norm_groups:
            raise ValueError(f"{mix.heads} heads in {mix.groups} groups, {mix.inner} channels in {mix.norm_groups} norm groups")
        return mix
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
        n, top, same = int(m["router"]["experts"]), int(m["router"]["top"]), int(m["router"].get("identity") or 0)
        if not 0 < top <= n + same:
            raise ValueError(f"{top} of {n + same} experts")
        fixed = dict(design.experts)
        if fixed.get("scoring") == "sigmoid":
            groups, scale = m["router"].get("groups") or {}, m["router"].get("scale")
            count = int(groups.get("count") or 1)
            keep = int(groups.get("keep") or count)
            if n % count or not 0 < keep <= count or top > keep * (n // count):
                raise ValueError(f"{top} of {n} experts in the best {keep} of {count} groups")
            fixed.update(groups=count, keep=keep, scale=1.0 if scale is None else float(scale))
        return ExpertMLP(n, top, _expert(m["expert"]), _expert(m["shared"]) if m.get("shared") else None, identity=same, **fixed)
    raise NotImplementedError(f"unknown feed-forward {kind!r}")


def parse_stack(cfg: dict[str, Any] | str) -> Stack:
    """``config.json`` of a stack checkpoint (a dictionary, or its JSON text) -> :class:`Stack`."""
    if isinstance(cfg, str):
        cfg = json.loads(cfg)
    design = DESIGNS[cfg["architecture"]]
    layers = tuple(StackLayer(_mixer(L["type"], L["mixer"], design), _mlp(L.get("mlp"), design)) for L in cfg["layers"])
    for i, L in enumerate(layers):
        j = getattr(L.mixer, "kv_from", None)
        if j is not None:
            src = layers[j].mixer if 0 <= j < i else None
            if not isinstance(src, AttentionMixer) or src.kv_from is not None or \
                    (src.kv_heads, src.maps, src.dim, src.vdim, src.rot) != (L.mixer.kv_heads, L.mixer.maps, L.mixer.dim, L.mixer.vdim, L.mixer.rot):
                raise ValueError(f"layer {i} cannot use the keys and values of layer {j}")
    loop = cfg.get("loop")
    if loop:
        loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
            raise ValueError(f"loop {loop} over {len(layers)} layers")
    scale, mult, out = (cfg.get("embedding") or {}).get("scale"), cfg.get("residual_mult"), cfg.get("logit_scale")
    return Stack(layers, loop or None, 1.0 if scale is None else float(scale), float(cfg["norm"]["eps"]), int(cfg["width"]), int(cfg["vocab"]),
                 float(cfg.get("logit_softcap") or 0.0), design, 1.0 if mult is None else float(mult), int((cfg.get("token_side") or {}).get("dim") or 0),
                 1.0 if out is None else float(out))
