"""Stack checkpoints (config.json with a ``layers`` list + safetensors, see models/stack.py) -> GGUF metadata and tensors.

Names follow the GGUF conventions for the same mechanisms (``blk.N.attn_q.weight``, ``blk.N.ssm_in.weight``, ...).  The norm vectors that
hold an offset from 1 are written as 1 + w and the decay matrix as A = -exp(A_log), both in fp32, as the other converters do.
"""
from __future__ import annotations

import json
import re
from typing import Any, Callable, Iterator

import torch

from ..gguf import quants
from ..gguf.types import GGMLType
from ..gguf.writer import WriteTensor
from ..models.stack import STACK_ARCHS, AttentionMixer, parse_stack

_TOP = {"embed": "token_embd.weight", "head": "output.weight", "final.norm": "output_norm.weight", "loop.in": "loop_in.weight"}
_LAYER = {
    "norm1": "attn_norm.weight", "norm2": "ffn_norm.weight", "mlp.up": "ffn_up.weight", "mlp.down": "ffn_down.weight",
    "mix.q": "attn_q.weight", "mix.k": "attn_k.weight", "mix.v": "attn_v.weight", "mix.q.norm": "attn_q_norm.weight", "mix.k.norm": "attn_k_norm.weight",
    "mix.in": "ssm_in.weight", "mix.conv": "ssm_conv1d.weight", "mix.conv.b": "ssm_conv1d.bias", "mix.x": "ssm_x.weight", "mix.dt": "ssm_dt.weight",
    "mix.dt.b": "ssm_dt.bias", "mix.A_log": "ssm_a", "mix.D": "ssm_d",
}
_ONE_PLUS = ("attn_norm.weight", "ffn_norm.weight", "output_norm.weight")
_F32 = ("ssm_a", "ssm_d", "ssm_conv1d.weight", "ssm_conv1d.bias", "ssm_dt.bias")


def is_stack_config(cfg: dict[str, Any]) -> bool:
    return cfg.get("architecture") in STACK_ARCHS


def stack_kv(cfg: dict[str, Any], name: str) -> dict[str, Any]:
    arch = STACK_ARCHS[cfg["architecture"]]
    st = parse_stack(cfg)
    kv: dict[str, Any] = {
        "general.architecture": arch, "general.name": name, "general.file_type": 32, f"{arch}.block_count": len(st.layers),
        f"{arch}.embedding_length": st.width, f"{arch}.vocab_size": st.vocab, f"{arch}.attention.layer_norm_rms_epsilon": st.eps,
        f"{arch}.stack": json.dumps(cfg, sort_keys=True),
    }
    ffs = [L.mlp.ff for L in st.layers if L.mlp is not None]
    if ffs:
        kv[f"{arch}.feed_forward_length"] = max(ffs)
    att = [L.mixer for L in st.layers if isinstance(L.mixer, AttentionMixer)]
    if att:
        kv.update({f"{arch}.attention.head_count": max(a.heads for a in att), f"{arch}.attention.head_count_kv": max(a.kv_heads for a in att),
                   f"{arch}.attention.key_length": max(a.dim for a in att), f"{arch}.attention.value_length": max(a.vdim for a in att)})
    if isinstance(cfg.get("context_length"), int):
        kv[f"{arch}.context_length"] = cfg["context_length"]
    return kv


def map_stack_name(name: str, cfg: dict[str, Any]) -> str | None:
    if name in _TOP:
        return _TOP[name]
    m = re.fullmatch(r"l(\d+)\.(.+)", name)
    if not m or int(m.group(1)) >= len(cfg["layers"]):
        return None
    rest = m.group(2)
    if rest == "mix.o":
        return f"blk.{m.group(1)}.{'ssm_out' if cfg['layers'][int(m.group(1))]['type'] == 'mamba1' else 'attn_output'}.weight"
    return f"blk.{m.group(1)}.{_LAYER[rest]}" if rest in _LAYER else None


def stack_tensors(src, cfg: dict[str, Any], outtype: str = "auto", progress: Callable[[str], None] | None = None) -> Iterator[WriteTensor]:
    """``src``: name -> tensor mapping with ``keys()`` and ``tensor(name)`` (convert/safetensors.py ModelDir)."""
    want = {"f32": GGMLType.F32, "f16": GGMLType.F16, "bf16": GGMLType.BF16}.get(outtype)
    for name in src.keys():
        out = map_stack_name(name, cfg)
        if out is None:
            raise ValueError(f"tensor {name} has no counterpart in a {cfg['architecture']} model")
        if progress:
            progress(out)
        t = src.tensor(name)
        if out.endswith(_ONE_PLUS):
            t = t.float() + 1.0
        elif out.endswith("ssm_a"):
            t = -torch.exp(t.double()).float()
        if t.dim() < 2 or out.endswith(_F32):
            dt = GGMLType.F32
        else:
            dt = want or {torch.bfloat16: GGMLType.BF16, torch.float16: GGMLType.F16}.get(t.dtype, GGMLType.F32)
        if dt == GGMLType.BF16 and t.dtype == torch.bfloat16:
            raw = t.contiguous().view(-1).view(torch.uint8)      # the stored bits as they are
        else:
            raw = quants.quantize(t.float(), dt)
        yield WriteTensor(out, tuple(reversed(t.shape)), dt, raw.cpu().numpy())
