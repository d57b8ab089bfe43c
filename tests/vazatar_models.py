"""Small Vazatar configurations with random weights for the tests."""
import json
import math
import os

import torch

from ollama_b200.convert.safetensors import save_file


def attention(heads=3, kv_heads=1, dim=40, vdim=24, size=20, rot=None, softcap=12.0, scale=0.2, ff=72):
    rot = rot if rot is not None else {"base": 700.0, "dims": 16, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 60}}
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "rot": rot,
                                           "scale": scale, "softcap": softcap}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mamba(inner=56, state=10, dt_rank=5, conv=4, ff=60):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=52, vocab=173, loop=(1, 3, 2), scale=3.5, eps=1e-5, cap=9.0):
    return {"architecture": "Vazatar", "embedding": {"scale": scale}, "layers": layers, "logit_softcap": cap,
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def shapes(cfg):
    """Tensor names and shapes of a configuration."""
    w, out = cfg["width"], {}
    out["embed"] = (cfg["vocab"], w)
    if cfg.get("loop"):
        out["loop.in"] = (w, 2 * w)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        out[p + "norm1"] = (w,)
        if L["type"] == "attention":
            nq, nk, nv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            out.update({p + "mix.q": (nq, w), p + "mix.k": (nk, w), p + "mix.v": (nv, w), p + "mix.q.norm": (nq,), p + "mix.k.norm": (nk,),
                        p + "mix.o": (w, m["heads"] * m["vdim"])})
        else:
            c, n, r = m["inner"], m["state"], m["dt_rank"]
            out.update({p + "mix.in": (2 * c, w), p + "mix.conv": (c, m["conv"]), p + "mix.conv.b": (c,), p + "mix.x": (r + 2 * n, c), p + "mix.dt": (c, r),
                        p + "mix.dt.b": (c,), p + "mix.A_log": (c, n), p + "mix.D": (c,), p + "mix.o": (w, c)})
        if L["mlp"]:
            out.update({p + "norm2": (w,), p + "mlp.up": (L["mlp"]["ff"], w), p + "mlp.down": (w, L["mlp"]["ff"])})
    out.update({"final.norm": (w,), "head": (cfg["vocab"], w)})
    return out


def weights(cfg, seed=0, sharp=1.8):
    """Random bf16 weights.  ``sharp`` widens q and k, so that single keys stand out of a softmax; step sizes and decays span fast and
    slow channels, so that a state from far back still counts."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        t = torch.randn(s, generator=g)
        if name.endswith(("norm1", "norm2", "final.norm")):
            t = 0.3 * t
        elif name.endswith((".q.norm", ".k.norm")):
            t = sharp * (1.0 + 0.3 * t)
        elif name.endswith("A_log"):
            t = torch.log(0.05 + 4.0 * torch.rand(s, generator=g) ** 3)
        elif name.endswith(".dt.b"):
            t = -4.0 + 1.5 * t
        elif name.endswith((".conv.b", ".D")):
            t = 0.5 + 0.3 * t
        elif name.endswith(".conv"):
            t = t / math.sqrt(s[1])
        elif name == "embed":
            t = 0.3 * t
        else:
            t = t / math.sqrt(s[1])
        out[name] = t.to(torch.bfloat16)
    return out


def write(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(w, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def small():
    """Two kinds of attention (one with vdim > dim, one key/value head per query head) around a Mamba layer in a loop that starts late."""
    return config([attention(), mamba(), attention(heads=2, kv_heads=2, dim=12, vdim=32, size=33, softcap=8.0, scale=0.35, ff=None, rot={"base": 50.0, "dims": 8}), mamba(inner=40, state=17, dt_rank=1, conv=2, ff=None),
                   attention(heads=4, kv_heads=2, dim=24, vdim=24, size=64, rot={"base": 90.0, "dims": 24, "scaling": None})])
