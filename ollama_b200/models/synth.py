"""Random-init checkpoints of the benchmark architectures.

Nothing can be downloaded where the benchmarks run, so weights are drawn from N(0, 0.02) with a
fixed seed and encoded with this package's own quantisers.  The per-tensor type mixture of a
``Q4_K_M`` file follows the rule the upstream quantiser applies (Q6_K for ``output.weight`` and for
``attn_v`` / ``ffn_down`` on the "more bits" layers, Q4_K elsewhere, F32 for 1-D tensors and the MoE
router), which is what ``general.file_type = 15`` means in practice (fs/ggml/type.go:28,70-71).
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Callable, Iterator

import torch

from ..gguf import quants
from ..gguf.types import FileType, GGMLType
from ..gguf.writer import WriteTensor, write_gguf


@dataclass
class ArchSpec:
    arch: str
    n_layers: int
    d_model: int
    n_heads: int
    n_kv_heads: int
    head_dim: int
    d_ff: int
    vocab: int
    rope_base: float = 10000.0
    eps: float = 1e-5
    ctx_train: int = 131072
    tied: bool = False
    n_experts: int = 0
    n_experts_used: int = 0
    d_ff_expert: int = 0
    sliding_window: int = 0
    extra_kv: dict = field(default_factory=dict)


SPECS: dict[str, ArchSpec] = {
    "tiny-llama": ArchSpec("llama", 2, 256, 4, 2, 64, 688, 32000, 10000.0, 1e-5, 2048),
    "llama-3.1-8b": ArchSpec("llama", 32, 4096, 32, 8, 128, 14336, 128256, 500000.0),
    "llama-3.1-70b": ArchSpec("llama", 80, 8192, 64, 8, 128, 28672, 128256, 500000.0),
    "qwen3-235b-a22b": ArchSpec("qwen3moe", 94, 4096, 64, 4, 128, 12288, 151936, 1e6, 1e-6, 40960,
                                n_experts=128, n_experts_used=8, d_ff_expert=1536),
    "gpt-oss-120b": ArchSpec("gpt-oss", 36, 2880, 64, 8, 64, 2880, 201088, 150000.0, 1e-5, 131072,
                             n_experts=128, n_experts_used=4, d_ff_expert=2880, sliding_window=128,
                             extra_kv={"rope.scaling.type": "yarn", "rope.scaling.factor": 32.0,
                                       "rope.scaling.original_context_length": 4096,
                                       "rope.scaling.yarn_beta_fast": 32.0, "rope.scaling.yarn_beta_slow": 1.0}),
    # dense models of the size of the stack models below, layer run by layer run (a gated FFN has three matrices for their two)
    "dense-1b": ArchSpec("llama", 20, 2048, 16, 4, 128, 5504, 32768, 500000.0),
    "dense-8b": ArchSpec("llama", 32, 4096, 32, 8, 128, 11008, 128256, 500000.0),
    # mixture-of-experts models of the size of kavenex-moe and tirudra-2k / 4k (whose shared expert counts as one more chosen expert)
    "experts-2k": ArchSpec("qwen3moe", 20, 2048, 16, 4, 128, 5504, 32768, 500000.0, 1e-6, n_experts=64, n_experts_used=5, d_ff_expert=1408),
    "experts-4k": ArchSpec("qwen3moe", 12, 4096, 32, 8, 128, 8192, 65536, 500000.0, 1e-6, n_experts=32, n_experts_used=5, d_ff_expert=2048),
    # small stand-ins of every family for tests
    "tiny-tp": ArchSpec("llama", 2, 1024, 16, 8, 64, 4096, 4096, 500000.0, 1e-5, 4096),      # divides 2, 4 and 8 ways
    "tiny-qwen3": ArchSpec("qwen3", 2, 256, 4, 2, 64, 768, 4096, 1e6, 1e-6, 4096),
    "tiny-qwen2": ArchSpec("qwen2", 2, 256, 4, 2, 64, 768, 4096, 1e6, 1e-6, 4096),
    "tiny-qwen3moe": ArchSpec("qwen3moe", 2, 256, 4, 2, 64, 768, 4096, 1e6, 1e-6, 4096, n_experts=8, n_experts_used=2, d_ff_expert=256),
    "tiny-gemma3": ArchSpec("gemma3", 6, 256, 4, 2, 64, 768, 4096, 1e6, 1e-6, 4096, tied=True, sliding_window=16),
    "tiny-gemma2": ArchSpec("gemma2", 2, 256, 4, 2, 64, 768, 4096, 10000.0, 1e-6, 4096, tied=True, sliding_window=16),
    "tiny-gpt-oss": ArchSpec("gpt-oss", 2, 256, 8, 2, 32, 256, 4096, 150000.0, 1e-5, 4096, n_experts=8, n_experts_used=2,
                             d_ff_expert=256, sliding_window=8,
                             extra_kv={"rope.scaling.type": "yarn", "rope.scaling.factor": 4.0,
                                       "rope.scaling.original_context_length": 64}),
    "tiny-mixtral": ArchSpec("llama", 2, 256, 4, 2, 64, 512, 4096, 10000.0, 1e-5, 4096, n_experts=4, n_experts_used=2, d_ff_expert=512),
}


def use_more_bits(i: int, n: int) -> bool:
    return i < n // 8 or i >= 7 * n // 8 or (i - n // 8) % 3 == 2


def tensor_type(name: str, shape: tuple[int, ...], file_type: int, layer: int, n_layers: int, spec: ArchSpec) -> GGMLType:
    """Encoding of one tensor inside a file of ``file_type``."""
    ft = FileType(file_type)
    if len(shape) == 1 or name.endswith(".bias") or "ffn_gate_inp" in name or name.endswith("_norm.weight") or "attn_sinks" in name:
        return GGMLType.F32
    if ft == FileType.F32:
        return GGMLType.F32
    if ft == FileType.F16:
        return GGMLType.F16
    if ft == FileType.BF16:
        return GGMLType.BF16
    base = {FileType.Q8_0: GGMLType.Q8_0, FileType.Q4_0: GGMLType.Q4_0, FileType.Q4_K_M: GGMLType.Q4_K,
            FileType.Q4_K_S: GGMLType.Q4_K, FileType.Q6_K: GGMLType.Q6_K, FileType.Q5_K_M: GGMLType.Q5_K,
            FileType.MXFP4_MOE: GGMLType.MXFP4}[ft]
    if ft == FileType.MXFP4_MOE:
        # gpt-oss layout: MXFP4 experts, bf16 attention / embeddings / output
        return GGMLType.MXFP4 if "_exps" in name else GGMLType.BF16
    k = shape[-1]
    t = base
    if ft in (FileType.Q4_K_M, FileType.Q4_K_S, FileType.Q5_K_M):
        if name == "output.weight" or (name == "token_embd.weight" and spec.tied):
            t = GGMLType.Q6_K
        elif ft != FileType.Q4_K_S and ("attn_v.weight" in name or "ffn_down" in name) and use_more_bits(layer, n_layers):
            t = GGMLType.Q6_K
        elif "attn_v.weight" in name and spec.n_layers == 80 and t == GGMLType.Q4_K:
            t = GGMLType.Q5_K     # the 70B rule: eight query heads share each V head, so it gets 5 bits
    if k % quants.block_size(t):
        t = GGMLType.Q8_0 if k % 32 == 0 else GGMLType.F16   # rows that do not fit a 256-block fall back
    return t


def tensor_table(spec: ArchSpec) -> list[tuple[str, tuple[int, ...], int]]:
    """(name, row-major shape, layer index or -1) for every tensor of the architecture."""
    s = spec
    q_dim, kv_dim = s.n_heads * s.head_dim, s.n_kv_heads * s.head_dim
    out: list[tuple[str, tuple[int, ...], int]] = [("token_embd.weight", (s.vocab, s.d_model), -1)]
    for i in range(s.n_layers):
        p = f"blk.{i}."
        out += [(p + "attn_norm.weight", (s.d_model,), i), (p + "attn_q.weight", (q_dim, s.d_model), i),
                (p + "attn_k.weight", (kv_dim, s.d_model), i), (p + "attn_v.weight", (kv_dim, s.d_model), i),
                (p + "attn_output.weight", (s.d_model, q_dim), i)]
        if s.arch in ("qwen2", "gpt-oss"):
            out += [(p + "attn_q.bias", (q_dim,), i), (p + "attn_k.bias", (kv_dim,), i), (p + "attn_v.bias", (kv_dim,), i)]
        if s.arch == "gpt-oss":
            out += [(p + "attn_output.bias", (s.d_model,), i), (p + "attn_sinks.weight", (s.n_heads,), i),
                    (p + "post_attention_norm.weight", (s.d_model,), i)]
        else:
            out += [(p + "ffn_norm.weight", (s.d_model,), i)]
        if s.arch in ("qwen3", "qwen3moe", "gemma3"):
            out += [(p + "attn_q_norm.weight", (s.head_dim,), i), (p + "attn_k_norm.weight", (s.head_dim,), i)]
        if s.arch in ("gemma2", "gemma3"):
            out += [(p + "post_attention_norm.weight", (s.d_model,), i), (p + "post_ffw_norm.weight", (s.d_model,), i)]
        if s.n_experts:
            fe = s.d_ff_expert
            out += [(p + "ffn_gate_inp.weight", (s.n_experts, s.d_model), i),
                    (p + "ffn_gate_exps.weight", (s.n_experts, fe, s.d_model), i),
                    (p + "ffn_up_exps.weight", (s.n_experts, fe, s.d_model), i),
                    (p + "ffn_down_exps.weight", (s.n_experts, s.d_model, fe), i)]
            if s.arch == "gpt-oss":
                out += [(p + "ffn_gate_inp.bias", (s.n_experts,), i), (p + "ffn_gate_exps.bias", (s.n_experts, fe), i),
                        (p + "ffn_up_exps.bias", (s.n_experts, fe), i), (p + "ffn_down_exps.bias", (s.n_experts, s.d_model), i)]
        else:
            out += [(p + "ffn_gate.weight", (s.d_ff, s.d_model), i), (p + "ffn_up.weight", (s.d_ff, s.d_model), i),
                    (p + "ffn_down.weight", (s.d_model, s.d_ff), i)]
    out.append(("output_norm.weight", (s.d_model,), -1))
    if not s.tied:
        out.append(("output.weight", (s.vocab, s.d_model), -1))
    return out


def metadata(spec: ArchSpec, file_type: int, name: str = "", with_tokenizer: bool = True) -> dict:
    s = spec
    kv: dict = {
        "general.architecture": s.arch, "general.name": name or s.arch, "general.file_type": int(file_type),
        "block_count": s.n_layers, "context_length": s.ctx_train, "embedding_length": s.d_model,
        "feed_forward_length": s.d_ff, "attention.head_count": s.n_heads, "attention.head_count_kv": s.n_kv_heads,
        "attention.key_length": s.head_dim, "attention.value_length": s.head_dim,
        "attention.layer_norm_rms_epsilon": float(s.eps), "rope.freq_base": float(s.rope_base),
        "rope.dimension_count": s.head_dim, "vocab_size": s.vocab,
    }
    if s.n_experts:
        kv.update({"expert_count": s.n_experts, "expert_used_count": s.n_experts_used, "expert_feed_forward_length": s.d_ff_expert})
    if s.sliding_window:
        kv["attention.sliding_window"] = s.sliding_window
    if s.arch == "gemma3":
        kv["rope.local.freq_base"] = 10000.0
    kv.update(s.extra_kv)
    if with_tokenizer:
        kv.update(synthetic_tokenizer_kv(s.vocab))
    return kv


def synthetic_tokenizer_kv(vocab: int) -> dict:
    """A vocabulary in which every id has a unique surface form ``<t{id}>`` that tokenises back to itself.

    Ids 0..2 are <unk>, <s>, </s>; ids 3..258 are the byte-fallback tokens ``<0xHH>`` so arbitrary text is
    representable; the rest are user-defined tokens (matched verbatim before the piece tokeniser runs).
    """
    toks, types, scores = [], [], []
    for i in range(vocab):
        if i == 0:
            toks.append("<unk>"); types.append(2)
        elif i == 1:
            toks.append("<s>"); types.append(3)
        elif i == 2:
            toks.append("</s>"); types.append(3)
        elif i < 259:
            toks.append(f"<0x{i - 3:02X}>"); types.append(6)
        else:
            toks.append(f"<t{i}>"); types.append(4)
        scores.append(0.0)
    return {
        "tokenizer.ggml.model": "llama", "tokenizer.ggml.tokens": toks, "tokenizer.ggml.token_type": types,
        "tokenizer.ggml.scores": scores, "tokenizer.ggml.bos_token_id": 1, "tokenizer.ggml.eos_token_id": 2,
        "tokenizer.ggml.unknown_token_id": 0, "tokenizer.ggml.add_bos_token": False, "tokenizer.ggml.add_eos_token": False,
        "tokenizer.ggml.add_space_prefix": False,
    }


def random_tensor(name: str, shape: tuple[int, ...], seed: int, device="cpu", std: float = 0.02) -> torch.Tensor:
    """Deterministic N(0, std) values for ``name`` (norm weights are 1 + noise, sinks/biases small)."""
    h = 0
    for ch in name:
        h = (h * 131 + ord(ch)) & 0x7FFFFFFF
    gen = torch.Generator(device=device)
    gen.manual_seed((seed * 1000003 + h) & 0x7FFFFFFFFFFF)
    n = math.prod(shape)
    x = torch.randn(n, generator=gen, device=device, dtype=torch.float32).mul_(std).view(*shape)
    if name.endswith("_norm.weight"):
        x = x + 1.0
    return x


def iter_tensors(spec: ArchSpec, file_type: int, seed: int = 0, device="cpu",
                 select: Callable[[str], bool] | None = None) -> Iterator[tuple[str, tuple[int, ...], GGMLType, torch.Tensor]]:
    """Yield (name, shape, type, encoded bytes) one tensor at a time."""
    for name, shape, layer in tensor_table(spec):
        if select is not None and not select(name):
            continue
        t = tensor_type(name, shape, file_type, max(layer, 0), spec.n_layers, spec)
        x = random_tensor(name, shape, seed, device)
        yield name, shape, t, quants.quantize(x, t)


def write_synthetic_gguf(path: str, spec_name: str, file_type: str | int = "F32", seed: int = 0, device="cpu",
                         template: str | None = None) -> None:
    spec = SPECS[spec_name]
    ft = file_type if isinstance(file_type, int) else int(getattr(FileType, file_type if file_type != "MXFP4" else "MXFP4_MOE"))
    kv = metadata(spec, ft, spec_name)
    if template:
        kv["tokenizer.chat_template"] = template
    tensors = []
    for name, shape, t, raw in iter_tensors(spec, ft, seed, device):
        tensors.append(WriteTensor(name, tuple(reversed(shape)), t, raw.cpu().numpy()))
    write_gguf(path, kv, tensors)


class SyntheticTensors:
    """Mapping-like source of :class:`QWeight` that draws and encodes each tensor when it is asked for.

    ``rows`` optionally restricts a tensor to a row range (tensor-parallel shards are generated
    directly, the full matrix is never materialised on one device).
    """

    def __init__(self, spec_name: str, file_type: str | int = "Q4_K_M", seed: int = 0, device="cpu"):
        from .weights import QWeight
        self._QWeight = QWeight
        self.spec = SPECS[spec_name]
        self.ft = file_type if isinstance(file_type, int) else int(getattr(FileType, file_type if file_type != "MXFP4" else "MXFP4_MOE"))
        self.seed, self.device = seed, device
        self.table = {n: (shape, layer) for n, shape, layer in tensor_table(self.spec)}

    def __contains__(self, name: str) -> bool:
        return name in self.table

    def keys(self):
        return self.table.keys()

    def type_of(self, name: str) -> GGMLType:
        shape, layer = self.table[name]
        return tensor_type(name, shape, self.ft, max(layer, 0), self.spec.n_layers, self.spec)

    def __getitem__(self, name: str):
        shape, layer = self.table[name]
        t = self.type_of(name)
        x = random_tensor(name, shape, self.seed, self.device)
        return self._QWeight(name, t, tuple(shape), quants.quantize(x, t))


def synthetic_header(spec_name: str, file_type: str | int = "Q4_K_M", with_tokenizer: bool = False):
    """A data-less :class:`GGUFFile` carrying the metadata of a synthetic checkpoint (for config parsing)."""
    from ..gguf.reader import GGUFFile, TensorInfo
    spec = SPECS[spec_name]
    ft = file_type if isinstance(file_type, int) else int(getattr(FileType, file_type if file_type != "MXFP4" else "MXFP4_MOE"))
    raw = metadata(spec, ft, spec_name, with_tokenizer=with_tokenizer)
    kv = {}
    for k, v in raw.items():
        kv[k if k.startswith(("general.", "tokenizer.")) else f"{spec.arch}.{k}"] = v
    tensors = {n: TensorInfo(n, tuple(reversed(shape)), tensor_type(n, shape, ft, max(layer, 0), spec.n_layers, spec), 0, 0)
               for n, shape, layer in tensor_table(spec)}
    return GGUFFile("", 3, "<", kv, {}, tensors, 0, 32)


# ---------------------------------------------------------------------------------------------------
# stack models (models/stack.py)
# ---------------------------------------------------------------------------------------------------
def stack_config(width: int, heads: int, kv_heads: int, dim: int, ff: int, inner: int, state: int, dt_rank: int, vocab: int, layers: str,
                 loop: tuple[int, int, int] | None, chunk: int) -> dict:
    """``config.json`` of a Vazatar model; ``layers``: one letter per layer, A (attention) or M (Mamba)."""
    att = {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": chunk}, "scale": dim ** -0.5, "softcap": 50.0,
                                          "rot": {"base": 500000.0, "dims": dim, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}}
    mam = {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": 4}}
    return {"architecture": "Vazatar", "embedding": {"scale": math.sqrt(width)}, "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None,
            "layers": [{**(att if c == "A" else mam), "mlp": {"kind": "dense", "ff": ff}} for c in layers]}


def latent_config(width: int, heads: int, dim: int, rot: int, vdim: int, rank: int, ff: int, vocab: int, layers: str, loop: tuple[int, int, int] | None, side: int,
                  experts: int = 0, top: int = 0, ff_expert: int = 0, ff_shared: int = 0) -> dict:
    """``config.json`` of a Kavenex model; ``layers``: one letter per layer, D (dense feed-forward), E (experts) or N (none)."""
    mix = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": (dim + rot) ** -0.5, "rot": {"base": 500000.0, "dims": rot}}
    moe = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff_expert, "limit": 7.0}}
    if ff_shared:
        moe["shared"] = {"ff": ff_shared, "limit": 7.0}
    mlp = {"D": {"kind": "dense", "ff": ff}, "E": moe, "N": None}
    return {"architecture": "Kavenex", "embedding": {"scale": math.sqrt(width)}, "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "residual_mult": 0.5,
            "token_side": {"dim": side} if side else None, "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None,
            "layers": [{"type": "latent_attention", "mixer": mix, "mlp": mlp[c]} for c in layers]}


def heads_config(width: int, heads: int, kv_heads: int, dim: int, window: int, full_kv: int, ssm_heads: int, ssm_dim: int, state: int, groups: int, vocab: int, layers: str,
                 experts: int, top: int, identity: int, ff_expert: int, ff_shared: int) -> dict:
    """``config.json`` of a Tirudra model; ``layers``: one letter per layer, W (windowed attention), F (full attention), M (Mamba-2), in lower case without a feed-forward."""
    mix = {"W": {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": 4, "mask": {"size": window, "keep_first": 4}, "scale": dim ** -0.5,
                                               "rot": {"base": 10000.0, "dims": dim, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}},
           "F": {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": full_kv, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
                                                 "rot": {"base": 500000.0, "dims": dim, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}},
           "M": {"type": "mamba2", "mixer": {"heads": ssm_heads, "vdim": ssm_dim, "state": state, "groups": groups, "conv": 4, "norm_groups": groups}}}
    moe = {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}, "expert": {"ff": ff_expert}, "shared": {"ff": ff_shared}}
    return {"architecture": "Tirudra", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "logit_scale": 0.5,
            "layers": [{**mix[c.upper()], "mlp": moe if c.isupper() else None} for c in layers]}


def shared_norm_config(width: int, heads: int, kv_heads: int, dim: int, gru: int, rank: int, q_rank: int, window: int, ff: int, vocab: int, layers: str, experts: int = 0, top: int = 0,
                       ff_expert: int = 0, groups: int = 1, keep: int = 1) -> dict:
    """``config.json`` of a Rinirax model; ``layers``: one letter per layer, A (differential attention), S (the same on the keys and values of the last A), G (gated recurrence), L (latent
    attention), followed by d for a dense feed-forward, e for experts or - for none."""
    att = {"heads": heads, "kv_heads": kv_heads, "dim": dim // 2, "vdim": dim, "conv": 4, "diff": 0.5, "scale": (dim // 2) ** -0.5, "rot": {"base": 500000.0, "dims": dim // 2}}
    lat = {"heads": heads, "dim": dim, "rot_dim": 64, "vdim": dim, "kv_rank": rank, "q_rank": q_rank, "mask": {"size": window}, "scale": (dim + 64) ** -0.5,
           "rot": {"base": 500000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    mix = {"A": ("attention", att), "G": ("mingru", {"width": gru}), "L": ("latent_attention", lat)}
    mlp = {"d": {"kind": "dense", "ff": ff}, "-": None,
           "e": {"kind": "moe", "expert": {"ff": ff_expert}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}, "scale": 2.0}}}
    out: list[dict] = []
    for i in range(0, len(layers), 2):
        c, f = layers[i:i + 2]
        source = layers[:i:2].rfind("A")
        kind, m = ("attention", {**att, "kv_from": source}) if c == "S" else mix[c]
        out.append({"type": kind, "mixer": m, "mlp": mlp[f]})
    return {"architecture": "Rinirax", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "layers": out}


STACK_SPECS: dict[str, dict] = {
    "tiny-rinirax": shared_norm_config(192, 6, 2, 64, 136, 80, 64, 40, 384, 4096, "AdGeLeSe", 6, 2, 96, 3, 2),
    "rinirax-1b": shared_norm_config(2048, 16, 4, 128, 2048, 512, 768, 1024, 8192, 32768, "AdGdLdSd" * 4),
    "rinirax-8b": shared_norm_config(4096, 32, 8, 128, 4096, 512, 1536, 1024, 16384, 128256, "AdGdLdSd" * 8),
    "rinirax-2k": shared_norm_config(2048, 16, 4, 128, 2048, 512, 768, 1024, 8192, 32768, "AeGeLeSe" * 5, 64, 4, 1408, 8, 4),
    "tiny-tirudra": heads_config(192, 6, 2, 48, 40, 3, 12, 16, 40, 3, 4096, "MWFm", 6, 3, 1, 96, 80),
    "tirudra-2k": heads_config(2048, 16, 4, 128, 1024, 4, 64, 64, 128, 2, 32768, "MWMF" * 5, 64, 4, 4, 1408, 1408),
    "tirudra-4k": heads_config(4096, 32, 8, 128, 1024, 8, 128, 64, 128, 8, 65536, "MWMF" * 3, 32, 4, 2, 2048, 2048),
    "tiny-kavenex": latent_config(192, 6, 40, 24, 48, 80, 384, 4096, "DED", (1, 3, 2), 24, 6, 2, 96, 64),
    "kavenex-1b": latent_config(2048, 16, 128, 64, 128, 512, 5504, 32768, "D" * 16, (0, 4, 2), 256),
    "kavenex-8b": latent_config(4096, 32, 128, 64, 128, 512, 11008, 128256, "D" * 28, (0, 4, 2), 256),
    "kavenex-moe": latent_config(2048, 16, 128, 64, 128, 512, 0, 32768, "E" * 16, (0, 4, 2), 256, 64, 4, 1408, 1408),
    "tiny-vazatar": stack_config(256, 4, 2, 64, 512, 512, 16, 16, 4096, "AMA", (0, 2, 2), 128),
    "vazatar-1b": stack_config(2048, 16, 4, 128, 8192, 4096, 16, 128, 32768, "AAMA" * 4, (0, 4, 2), 2048),
    "vazatar-8b": stack_config(4096, 32, 8, 128, 16384, 8192, 16, 256, 128256, "AAMA" * 7, (0, 4, 2), 8192),
}


class SyntheticStackTensors:
    """Mapping-like source of random :class:`QWeight` tensors of a stack model, under their GGUF names."""

    def __init__(self, cfg: dict, seed: int = 0, device="cpu"):
        from ..convert.stack import map_stack_name
        self.seed, self.device, w = seed, device, cfg["width"]
        shared = cfg["architecture"] == "Rinirax"    # one norm per layer, averages over depth
        names: dict[str, tuple[int, ...]] = {"embed": (cfg["vocab"], w), "head": (cfg["vocab"], w), "final.norm": (w,)}
        seq = cfg["architecture"] == "Kavenex"       # layer norms, gated feed-forwards, a loop that begins with sums
        post = cfg["architecture"] == "Tirudra"      # norms behind every part, a correction of the router and a gate of the shared expert instead of a bias
        if cfg.get("loop"):
            names.update({"loop.step": (cfg["loop"]["times"], w)} if seq else {"loop.in": (w, 2 * w)})
        side = (cfg.get("token_side") or {}).get("dim")
        if side:
            names["side.embed"] = (cfg["vocab"], len(cfg["layers"]) * side)
        stacked: dict[str, tuple[int, ...]] = {}
        for i, L in enumerate(cfg["layers"]):
            m, p = L["mixer"], f"l{i}."
            names.update({p + "norm1": (w,), **({p + "norm1b": (w,)} if post else {})})
            if L["type"] == "latent_attention":
                H, d, r, dv, k, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m.get("q_rank")
                names.update({p + "mix.dq": (rank, w), p + "mix.dq.norm": (rank,), p + "mix.uq": (H * (d + r), rank)} if rank else {p + "mix.q": (H * (d + r), w)})
                names.update({p + "mix.dkv": (k + r, w), p + "mix.dkv.norm": (k,), p + "mix.uk": (H * d, k), p + "mix.uv": (H * dv, k),
                              p + "mix.o": (w, H * dv)})
            elif L["type"] == "mamba2":
                H, c, bc = m["heads"], m["heads"] * m["vdim"], 2 * m["groups"] * m["state"]
                names.update({p + "mix.in": (2 * c + bc + H, w), p + "mix.conv": (c + bc, m["conv"]), p + "mix.conv.b": (c + bc,), p + "mix.dt_bias": (H,), p + "mix.A_log": (H,),
                              p + "mix.D": (H,), p + "mix.norm": (c,), p + "mix.o": (w, c)})
            elif L["type"] == "mingru":
                n = m["width"]
                names.update({p + "mix.z": (n, w), p + "mix.z.b": (n,), p + "mix.x": (n, w), p + "mix.x.b": (n,), p + "mix.g": (n, w), p + "mix.o": (w, n)})
            elif shared:
                n = {"q": 2 * m["heads"] * m["dim"], "k": 2 * m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
                for x in "q" if "kv_from" in m else "qkv":
                    names.update({p + "mix." + x: (n[x], w), f"{p}mix.{x}.b": (n[x],), f"{p}mix.{x}.conv": (n[x], m["conv"])})
                names.update({p + "mix.o": (w, m["heads"] * m["vdim"]), **{p + "mix." + x: (m["dim"],) for x in ("lq1", "lk1", "lq2", "lk2")}})
            elif post:
                H, nq, nk, nv = m["heads"], m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
                names.update({p + "mix.q": (nq, w), p + "mix.k": (nk, w), p + "mix.q.norm": (m["dim"],), p + "mix.k.norm": (m["dim"],), p + "mix.o": (w, H * m["vdim"])})
                if L["type"] == "attention":
                    names.update({p + "mix.v": (nv, w), p + "mix.g": (H * m["vdim"], w), **{p + f"mix.{n}.conv": (k, m["conv"]) for n, k in (("q", nq), ("k", nk), ("v", nv))}})
                else:
                    names.update({p + "mix.q.b": (nq,), p + "mix.k.b": (nk,), p + "mix.g": (H, w)})
            elif L["type"] == "attention":
                nq, nk, nv, no = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
                names.update({p + "mix.q": (nq, w), p + "mix.k": (nk, w), p + "mix.v": (nv, w), p + "mix.q.norm": (nq,), p + "mix.k.norm": (nk,), p + "mix.o": (w, no)})
            else:
                c, n, r = m["inner"], m["state"], m["dt_rank"]
                names.update({p + "mix.in": (2 * c, w), p + "mix.conv": (c, m["conv"]), p + "mix.conv.b": (c,), p + "mix.x": (r + 2 * n, c), p + "mix.dt": (c, r),
                              p + "mix.dt.b": (c,), p + "mix.A_log": (c, n), p + "mix.D": (c,), p + "mix.o": (w, c)})
            f = L.get("mlp")
            if shared:
                names[p + "dwa"] = (i + 2,)
            if f and not shared:
                names.update({p + "norm2": (w,), **({p + "norm2b": (w,)} if post else {})})
            if f and f["kind"] == "dense":
                names.update({p + "mlp.up": (f["ff"], w), p + "mlp.down": (w, f["ff"]), **({p + "mlp.gate": (f["ff"], w)} if seq else {p + "mlp.act": (2,)} if shared else {})})
            elif f:
                E, fe, fs = f["router"]["experts"], f["expert"]["ff"], (f.get("shared") or {}).get("ff")
                n = E + f["router"].get("identity", 0)
                names.update({p + "mlp.router": (n, w), **({p + "mlp.correction": (n,)} if post or shared else {p + "mlp.router.b": (n,)}), **({p + "mlp.shared.sg": (1, w)} if post else {})})
                for pre, fx in ((f"blk.{i}.ffn_%s_exps.weight", (E, fe)), (f"blk.{i}.ffn_%s_shexp.weight", (fs,))):
                    if fx[-1]:
                        stacked.update({pre % "gate": (*fx, w), pre % "up": (*fx, w), pre % "down": (*fx[:-1], w, fx[-1])})
            if side:
                names.update({p + "side.gate": (side, w), p + "side.proj": (w, side), p + "side.norm": (w,)})
        if seq or shared:
            names.update({n + ".b": s for n, s in names.items() if n.endswith(("norm1", "norm2", "final.norm"))})
        self.table = {**{map_stack_name(n, cfg): s for n, s in names.items()}, **stacked}

    def __contains__(self, name: str) -> bool:
        return name in self.table

    def keys(self):
        return self.table.keys()

    def __getitem__(self, name: str):
        from .weights import QWeight
        s = self.table[name]
        x = random_tensor(name, s, self.seed, self.device)
        if name.endswith("ssm_a"):
            x = -(1.0 + torch.arange(s[-1], device=x.device, dtype=torch.float32)).expand(s).contiguous()
        if name.endswith("depth_average.weight"):
            x = 0.1 * torch.sin(torch.arange(s[0], device=x.device, dtype=torch.float32))
            x[-1] = 1.0
        f32 = len(s) < 2 or name.endswith(("ssm_a", "conv1d.weight"))
        raw = (x if f32 else x.to(torch.bfloat16)).contiguous().view(-1).view(torch.uint8)
        return QWeight(name, GGMLType.F32 if f32 else GGMLType.BF16, tuple(s), raw)


def stack_model_config(cfg: dict):
    """:class:`ModelConfig` of a stack configuration, as a file with that metadata would give it."""
    from ..convert.stack import stack_kv
    from ..gguf.reader import GGUFFile
    from .config import config_from_gguf
    return config_from_gguf(GGUFFile("", 3, "<", stack_kv(cfg, ""), {}, {}, 0, 32))
