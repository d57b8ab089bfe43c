"""Small Rinirax configurations with random weights for the tests."""
import math

import torch

from vazatar_models import tokens, write  # noqa: F401  (re-exported for the tests)

YARN = {"factor": 3.0, "original": 90, "fast": 9.0, "slow": 0.7}


def dense(ff=44):
    return {"kind": "dense", "ff": ff}


def moe(experts=12, top=2, ff=20, groups=3, keep=2, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale}}


def diff(mlp=None, heads=4, kv_heads=2, dim=20, vdim=36, conv=4, offset=0.45, rot=None, scale=0.3, kv_from=None):
    rot = rot if rot is not None else {"base": 700.0, "dims": 12}
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "diff": offset, "rot": rot, "scale": scale}
    return {"type": "attention", "mlp": mlp, "mixer": {**m, **({} if kv_from is None else {"kv_from": kv_from})}}


def gru(mlp=None, width=70):
    return {"type": "mingru", "mlp": mlp, "mixer": {"width": width}}


def latent(mlp=None, heads=5, dim=24, rot_dim=12, vdim=28, kv_rank=36, q_rank=44, size=37, rot=None, scale=0.25):
    rot = rot if rot is not None else {"base": 900.0, "dims": rot_dim, "scaling": YARN}
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                                              "mask": {"size": size}, "rot": rot, "scale": scale}}


def config(layers, width=60, vocab=173, eps=1e-5):
    return {"architecture": "Rinirax", "layers": layers, "norm": {"eps": eps}, "width": width, "vocab": vocab}


def shapes(cfg):
    """Tensor names and shapes of a configuration."""
    w = cfg["width"]
    out = {"embed": (cfg["vocab"], w), "final.norm": (w,), "final.norm.b": (w,), "head": (cfg["vocab"], w)}
    for i, L in enumerate(cfg["layers"]):
        m, p, f = L["mixer"], f"l{i}.", L["mlp"]
        out.update({p + "norm1": (w,), p + "norm1.b": (w,), p + "dwa": (i + 2,)})
        if L["type"] == "mingru":
            n = m["width"]
            out.update({p + "mix.z": (n, w), p + "mix.z.b": (n,), p + "mix.x": (n, w), p + "mix.x.b": (n,), p + "mix.g": (n, w), p + "mix.o": (w, n)})
        elif L["type"] == "latent_attention":
            H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            out.update({p + "mix.dq": (m["q_rank"], w), p + "mix.dq.norm": (m["q_rank"],), p + "mix.uq": (H * (d + r), m["q_rank"]), p + "mix.dkv": (rank + r, w),
                        p + "mix.dkv.norm": (rank,), p + "mix.uk": (H * d, rank), p + "mix.uv": (H * dv, rank), p + "mix.o": (w, H * dv)})
        else:
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, k in (("q", 2 * H * d), ("k", 2 * G * d), ("v", G * dv)):
                if n == "q" or m.get("kv_from") is None:
                    out.update({p + "mix." + n: (k, w), f"{p}mix.{n}.b": (k,), f"{p}mix.{n}.conv": (k, m["conv"])})
            out.update({p + "mix." + n: (d,) for n in ("lq1", "lk1", "lq2", "lk2")})
            out[p + "mix.o"] = (w, H * dv)
        if f and f["kind"] == "dense":
            out.update({p + "mlp.up": (f["ff"], w), p + "mlp.down": (w, f["ff"]), p + "mlp.act": (2,)})
        elif f:
            for e in range(f["router"]["experts"]):
                out.update({f"{p}mlp.e{e}.gate": (f["expert"]["ff"], w), f"{p}mlp.e{e}.up": (f["expert"]["ff"], w), f"{p}mlp.e{e}.down": (w, f["expert"]["ff"])})
            out.update({p + "mlp.router": (f["router"]["experts"], w), p + "mlp.correction": (f["router"]["experts"],)})
    return out


def weights(cfg, seed=0, sharp=1.8):
    """Random bf16 weights.  ``sharp`` widens queries and keys, so that single keys stand out of a softmax; update gates span channels that forget at once and channels that
    remember; the correction is large enough to change choices, and negative for some groups as a whole."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        t = torch.randn(s, generator=g)
        if name.endswith(("norm1", "final.norm", ".dq.norm", ".dkv.norm")):
            t = 1.0 + 0.3 * t
        elif name.endswith("z.b"):
            t = -2.0 + 2.5 * t
        elif name.endswith("dwa"):
            t = 0.3 * t / math.sqrt(s[0])
            t[-1] += 0.8
        elif name.endswith((".b", ".act")):
            t = 0.5 * t
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = 0.6 * t / math.sqrt(s[0])
        elif name.endswith("correction"):
            t = 0.3 * t - 0.4
        elif name.endswith("router"):
            t = 2.0 * t / math.sqrt(s[1])
        elif name.endswith(("mix.q", "mix.k", "mix.uq", "mix.uk")):
            t = sharp * t / math.sqrt(s[1])
        elif name != "embed":
            t = t / math.sqrt(s[1])
        out[name] = t.to(torch.bfloat16)
    return out


def small():
    """Every mixer with every kind of feed-forward or none, keys and values shared across other layers."""
    return config([diff(moe()), gru(dense()), diff(dense(20), conv=2, kv_from=0), latent(moe(8, 3, 12, 4, 3, 0.6)), gru(moe(9, 4, 28, 3, 2), width=33), diff(None, conv=3, kv_from=0, offset=0.1),
                   latent(None, size=64, q_rank=17, rot={"base": 50.0, "dims": 12}), diff(None, heads=3, kv_heads=3, dim=16, vdim=16, conv=1, rot={"base": 90.0, "dims": 16}), gru(None)])
