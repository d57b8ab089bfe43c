"""Throughput of stack models beside a model of equal size, both in bf16 with random weights on one GPU.

    python bench.py --stack [--model NAME|all] [--steps K] [--warmup W]

For each size: prompt evaluation of a 2048-token prompt, and decode steps of 1, 4 and 16 sequences at 1024 tokens of context.  Besides
tokens per second every figure carries its fraction of the roofline: the matrix products' FLOPs over the bf16 GEMM peak for prompts, the
weight and cache bytes of a step over the copy bandwidth for decoding (of experts, the ones that a step of so many tokens picks on average).
Weights of a step exceed the L2, so that nothing has to be flushed.
"""
from __future__ import annotations

import json
import os
import statistics

import torch

PAIRS = {"vazatar-1b": "dense-1b", "vazatar-8b": "dense-8b", "kavenex-1b": "dense-1b", "kavenex-8b": "dense-8b", "kavenex-moe": "experts-2k", "tirudra-2k": "experts-2k",
         "tirudra-4k": "experts-4k", "rinirax-1b": "dense-1b", "rinirax-8b": "dense-8b", "rinirax-2k": "experts-2k"}
PROMPT, CONTEXT, BATCHES, LOOP = 2048, 1024, (1, 4, 16), 32


def peaks() -> tuple[float, float]:
    """(bytes/s, bf16 FLOP/s) measured on the machine class, or the stated fallback."""
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        with open(path, encoding="utf-8") as f:
            p = json.load(f)
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12
    except (OSError, KeyError, ValueError):
        return 6.65e12, 1.59e15


def load(name: str, dev: str):
    """(backend, matrix weights that a token is multiplied with, weights of the experts of one such pass, share of the experts a token picks)."""
    from ..models import synth
    if name in synth.STACK_SPECS:
        from ..engine.stack import StackBackend
        cfg = synth.stack_model_config(synth.STACK_SPECS[name])
        be = StackBackend(None, device=dev, cfg=cfg, tensors=synth.SyntheticStackTensors(synth.STACK_SPECS[name], device=dev))
        dense, routed, share = be.product_weights()
        return be, dense, routed, share
    from ..engine.b200 import B200Backend
    from ..models.config import config_from_gguf
    cfg = config_from_gguf(synth.synthetic_header(name, "BF16"))
    be = B200Backend(None, device=dev, cfg=cfg, tensors=synth.SyntheticTensors(name, "BF16", seed=0, device=dev), kv_type="f16")
    n = cfg.n_layers * cfg.d_model * (2 * cfg.q_dim + 2 * cfg.kv_dim) + cfg.vocab_size * cfg.d_model
    if cfg.is_moe:
        return be, n + cfg.n_layers * cfg.d_model * cfg.n_experts, cfg.n_layers * cfg.n_experts * 3 * cfg.d_model * cfg.d_ff_expert, cfg.n_experts_used / cfg.n_experts
    return be, n + cfg.n_layers * 3 * cfg.d_model * cfg.d_ff, 0, 0.0


def timed(fn, warmup: int, steps: int) -> float:
    """Median device time of ``fn`` in seconds."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    ms = []
    for _ in range(steps):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ms.append(a.elapsed_time(b))
    return statistics.median(ms) / 1e3


def measure(name: str, steps: int, warmup: int, dev: str = "cuda:0") -> dict:
    be, dense, routed, share = load(name, dev)
    n = int(dense + routed * share)
    cfg = be.cfg
    hbm, flops = peaks()
    be.alloc(max(BATCHES), PROMPT + 64)
    gen = torch.Generator().manual_seed(1)
    toks = torch.randint(0, cfg.vocab_size, (PROMPT,), generator=gen).tolist()
    head = cfg.vocab_size * cfg.d_model
    t = timed(lambda: be.prefill(0, toks, 0), warmup, steps)
    out = {"model": name, "weights_per_pass": n, "prompt": {"tokens": PROMPT, "tok_s": round(PROMPT / t, 1), "roofline": round(2 * (n - head) * PROMPT / t / flops, 3)}}
    for nb in BATCHES:
        slots = list(range(nb))
        for s in slots:               # sequences of their own, which choose experts of their own
            be.prefill(s, torch.randint(0, cfg.vocab_size, (CONTEXT,), generator=gen).tolist(), 0, need_logits=False)
        first = torch.randint(0, cfg.vocab_size, (nb,), generator=gen).tolist()
        t = timed(lambda: be.decode_loop(slots, first, [CONTEXT] * nb, LOOP), warmup, steps) / LOOP
        byts = 2 * (dense + routed * (1.0 - (1.0 - share) ** nb)) + nb * cfg.kv_bytes_per_token() * CONTEXT
        out[f"decode_{nb}"] = {"tok_s": round(nb / t, 1), "step_us": round(t * 1e6, 1), "roofline": round(byts / t / hbm, 3), "launches": be.launches_per_step}
    from ..ops import cuda as K
    out["status"] = K.gemm_status()
    be.close()
    del be
    torch.cuda.empty_cache()
    return out


def run(model: str, steps: int, warmup: int) -> dict:
    names = list(PAIRS) if model in ("auto", "all") else [model]
    rows = [measure(m, steps, max(warmup, 3)) for m in dict.fromkeys(m for name in names for m in (name, PAIRS[name]))]
    return {"metric": "stack_models", "unit": "tok/s", "dtype": "bf16", "data": "synthetic", "config": {"prompt": PROMPT, "context": CONTEXT, "batches": list(BATCHES),
            "l2": "weights of a step are larger than L2"}, "results": rows}
