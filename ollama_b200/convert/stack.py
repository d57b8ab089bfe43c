"""Stack checkpoints (config.json with a ``layers`` list + safetensors, see models/stack.py) -> GGUF metadata and tensors.

Names follow the GGUF conventions for the same mechanisms (``blk.N.attn_q.weight``, ``blk.N.ssm_in.weight``, ...).  Norm vectors that
hold an offset from 1 are written as 1 + w and the decay matrix as A = -exp(A_log), both in fp32; the experts of a layer are stacked into one
tensor per matrix.  All as the other converters do.
"""
from __future__ import annotations

import json
import re
from typing import Any, Callable, Iterator

import torch

from ..gguf import quants
from ..gguf.types import GGMLType
from ..gguf.writer import WriteTensor
from ..models.stack import DESIGNS, STACK_ARCHS, AttentionMixer, ExpertMLP, LatentMixer, parse_stack

_TOP = {"embed": "token_embd.weight", "head": "output.weight", "final.norm": "output_norm.weight", "final.norm.b": "output_norm.bias",
        "loop.in": "loop_in.weight", "loop.step": "loop_step.weight", "side.embed": "per_layer_token_embd.weight"}
_LAYER = {
    "norm1": "attn_norm.weight", "norm2": "ffn_norm.weight", "mlp.up": "ffn_up.weight", "mlp.down": "ffn_down.weight",
    "mix.q": "attn_q.weight", "mix.k": "attn_k.weight", "mix.v": "attn_v.weight", "mix.q.norm": "attn_q_norm.weight", "mix.k.norm": "attn_k_norm.weight",
    "mix.in": "ssm_in.weight", "mix.conv": "ssm_conv1d.weight", "mix.conv.b": "ssm_conv1d.bias", "mix.x": "ssm_x.weight", "mix.dt": "ssm_dt.weight",
    "mix.dt.b": "ssm_dt.bias", "mix.A_log": "ssm_a", "mix.D": "ssm_d",
    "norm1.b": "attn_norm.bias", "norm2.b": "ffn_norm.bias", "mlp.gate": "ffn_gate.weight",
    "mix.dkv": "attn_kv_a_mqa.weight", "mix.dkv.norm": "attn_kv_a_norm.weight", "mix.uk": "attn_k_b.weight", "mix.uv": "attn_v_b.weight",
    "mlp.router": "ffn_gate_inp.weight", "mlp.router.b": "ffn_gate_inp.bias",
    "mlp.shared.gate": "ffn_gate_shexp.weight", "mlp.shared.up": "ffn_up_shexp.weight", "mlp.shared.down": "ffn_down_shexp.weight",
    "side.gate": "inp_gate.weight", "side.proj": "proj.weight", "side.norm": "post_norm.weight",
    "norm1b": "post_attention_norm.weight", "norm2b": "post_ffw_norm.weight", "mix.g": "attn_gate.weight", "mix.q.b": "attn_q.bias", "mix.k.b": "attn_k.bias",
    "mix.q.conv": "attn_q_conv1d.weight", "mix.k.conv": "attn_k_conv1d.weight", "mix.v.conv": "attn_v_conv1d.weight",
    "mix.v.b": "attn_v.bias", "mix.lq1": "attn_lambda_q1.weight", "mix.lk1": "attn_lambda_k1.weight", "mix.lq2": "attn_lambda_q2.weight", "mix.lk2": "attn_lambda_k2.weight",
    "mix.dq": "attn_q_a.weight", "mix.dq.norm": "attn_q_a_norm.weight", "mix.uq": "attn_q_b.weight", "mlp.act": "ffn_act.weight", "dwa": "depth_average.weight",
    "mix.dt_bias": "ssm_dt.bias", "mix.norm": "ssm_norm.weight", "mlp.correction": "exp_probs_b.bias", "mlp.shared.sg": "ffn_gate_inp_shexp.weight",
}
_GRU = {"mix.z": "gru_z.weight", "mix.z.b": "gru_z.bias", "mix.x": "gru_x.weight", "mix.x.b": "gru_x.bias", "mix.g": "gru_gate.weight", "mix.o": "gru_out.weight"}
_EXPERT = re.compile(r"l(\d+)\.mlp\.e(\d+)\.(gate|up|down)")
_ONE_PLUS = ("attn_norm.weight", "ffn_norm.weight", "output_norm.weight", "post_attention_norm.weight", "post_ffw_norm.weight")
_F32 = ("ssm_a", "ssm_d", "conv1d.weight", "ssm_conv1d.bias", "ssm_dt.bias")


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
    moe = [L.mlp for L in st.layers if isinstance(L.mlp, ExpertMLP)]
    ffs = [L.mlp.ff for L in st.layers if L.mlp is not None and not isinstance(L.mlp, ExpertMLP)]
    if ffs:
        kv[f"{arch}.feed_forward_length"] = max(ffs)
    if moe:
        kv.update({f"{arch}.expert_count": max(m.experts for m in moe), f"{arch}.expert_used_count": max(m.top for m in moe),
                   f"{arch}.expert_feed_forward_length": max(m.expert.ff for m in moe)})
    lat = [L.mixer for L in st.layers if isinstance(L.mixer, LatentMixer)]
    if lat:
        kv.update({f"{arch}.attention.head_count": max(a.heads for a in lat), f"{arch}.attention.head_count_kv": 1,
                   f"{arch}.attention.key_length": max(a.dim + a.rot_dim for a in lat), f"{arch}.attention.value_length": max(a.vdim for a in lat),
                   f"{arch}.attention.kv_lora_rank": max(a.kv_rank for a in lat), f"{arch}.rope.dimension_count": max(a.rot_dim for a in lat)})
    att = [L.mixer for L in st.layers if isinstance(L.mixer, AttentionMixer)]
    if att:
        kv.update({f"{arch}.attention.head_count": max(a.heads for a in att), f"{arch}.attention.head_count_kv": max(a.kv_heads for a in att),
                   f"{arch}.attention.key_length": max(a.dim for a in att), f"{arch}.attention.value_length": max(a.vdim for a in att)})
    if isinstance(cfg.get("context_length"), int):
        kv[f"{arch}.context_length"] = cfg["context_length"]
    return kv


def map_stack_name(name: str, cfg: dict[str, Any]) -> str | None:
    """GGUF name of a checkpoint tensor; an expert's matrix gets the name of the stack it is part of."""
    if name in _TOP:
        return _TOP[name]
    m = re.fullmatch(r"l(\d+)\.(.+)", name)
    if not m or int(m.group(1)) >= len(cfg["layers"]):
        return None
    rest, kind = m.group(2), cfg["layers"][int(m.group(1))]["type"]
    if kind == "mingru" and rest in _GRU:
        return f"blk.{m.group(1)}.{_GRU[rest]}"
    if rest == "mix.o":
        return f"blk.{m.group(1)}.{'ssm_out' if kind.startswith('mamba') else 'attn_output'}.weight"
    e = _EXPERT.fullmatch(name)
    if e:
        router = (cfg["layers"][int(e.group(1))].get("mlp") or {}).get("router") or {}
        return f"blk.{e.group(1)}.ffn_{e.group(3)}_exps.weight" if int(e.group(2)) < int(router.get("experts") or 0) else None
    return f"blk.{m.group(1)}.{_LAYER[rest]}" if rest in _LAYER else None


def stack_tensors(src, cfg: dict[str, Any], outtype: str = "auto", progress: Callable[[str], None] | None = None) -> Iterator[WriteTensor]:
    """``src``: name -> tensor mapping with ``keys()`` and ``tensor(name)`` (convert/safetensors.py ModelDir)."""
    want = {"f32": GGMLType.F32, "f16": GGMLType.F16, "bf16": GGMLType.BF16}.get(outtype)
    one_plus = DESIGNS[cfg["architecture"]].norm == "rms_one_plus"
    experts: dict[str, dict[int, str]] = {}          # stacked tensor -> the checkpoint tensors it is made of

    def encode(out: str, t: torch.Tensor) -> WriteTensor:
        if one_plus and out.endswith(_ONE_PLUS):
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
        return WriteTensor(out, tuple(reversed(t.shape)), dt, raw.cpu().numpy())

    for name in src.keys():
        out = map_stack_name(name, cfg)
        if out is None:
            raise ValueError(f"tensor {name} has no counterpart in a {cfg['architecture']} model")
        e = _EXPERT.fullmatch(name)
        if e:
            experts.setdefault(out, {})[int(e.group(2))] = name
            continue
        if progress:
            progress(out)
        yield encode(out, src.tensor(name))
    for out, parts in experts.items():
        n = int(cfg["layers"][int(out.split(".")[1])]["mlp"]["router"]["experts"])
        if len(parts) != n:
            raise ValueError(f"{out}: {len(parts)} of {n} experts")
        if progress:
            progress(out)
        yield encode(out, torch.stack([src.tensor(parts[i]) for i in range(n)]))
