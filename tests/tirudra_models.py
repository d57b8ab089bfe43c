"""Small Tirudra configurations with random weights for the tests."""
import math

import torch

from vazatar_models import tokens, write  # noqa: F401  (re-exported for the tests)

YARN = {"factor": 3.0, "original": 90, "fast": 9.0, "slow": 0.7}
LOW_HIGH = {"factor": 5.0, "low": 1.0, "high": 3.5, "original": 70}


def moe(experts=6, top=3, ff=28, identity=2, shared=20):
    return {"kind": "moe", "router": {"experts": experts, "top": top, **({"identity": identity} if identity else {})}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def windowed(mlp=None, heads=4, kv_heads=2, dim=20, vdim=28, size=37, keep=3, conv=4, rot=None, scale=0.3):
    rot = rot if rot is not None else {"base": 800.0, "dims": 12, "scaling": YARN}
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": size, "keep_first": keep},
                                                      "rot": rot, "scale": scale}}


def full(mlp=None, heads=6, kv_heads=3, dim=24, rot=None, scale=0.25):
    rot = rot if rot is not None else {"base": 600.0, "dims": 24, "scaling": LOW_HIGH}
    return {"type": "attention_2", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": rot, "scale": scale}}


def mamba(mlp=None, heads=6, vdim=12, state=20, groups=3, conv=3, norm_groups=2):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def config(layers, width=52, vocab=173, eps=1e-5, logit_scale=0.37):
    return {"architecture": "Tirudra", "layers": layers, "norm": {"eps": eps}, "width": width, "vocab": vocab, "logit_scale": logit_scale}


def shapes(cfg):
    """Tensor names and shapes of a configuration."""
    w = cfg["width"]
    out = {"embed": (cfg["vocab"], w), "final.norm": (w,), "head": (cfg["vocab"], w)}
    for i, L in enumerate(cfg["layers"]):
        m, p, f = L["mixer"], f"l{i}.", L["mlp"]
        out.update({p + "norm1": (w,), p + "norm1b": (w,)})
        H = m["heads"]
        if L["type"] == "mamba2":
            inner, bc = H * m["vdim"], m["groups"] * m["state"]
            out.update({p + "mix.in": (2 * inner + 2 * bc + H, w), p + "mix.conv": (inner + 2 * bc, m["conv"]), p + "mix.conv.b": (inner + 2 * bc,), p + "mix.dt_bias": (H,),
                        p + "mix.A_log": (H,), p + "mix.D": (H,), p + "mix.norm": (inner,), p + "mix.o": (w, inner)})
        else:
            nq, nk, nv = H * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            out.update({p + "mix.q": (nq, w), p + "mix.k": (nk, w), p + "mix.q.norm": (m["dim"],), p + "mix.k.norm": (m["dim"],), p + "mix.o": (w, H * m["vdim"])})
            if L["type"] == "attention":
                out.update({p + "mix.v": (nv, w), p + "mix.g": (H * m["vdim"], w)})
                out.update({p + f"mix.{n}.conv": (k, m["conv"]) for n, k in (("q", nq), ("k", nk), ("v", nv))})
            else:
                out.update({p + "mix.q.b": (nq,), p + "mix.k.b": (nk,), p + "mix.g": (H, w)})
        if not f:
            continue

        def gated(pre, ff):
            out.update({pre + "gate": (ff, w), pre + "up": (ff, w), pre + "down": (w, ff)})

        out.update({p + "norm2": (w,), p + "norm2b": (w,)})
        r = f["router"]
        for e in range(r["experts"]):
            gated(p + f"mlp.e{e}.", f["expert"]["ff"])
        n = r["experts"] + r.get("identity", 0)
        out.update({p + "mlp.router": (n, w), p + "mlp.correction": (n,)})
        if f.get("shared"):
            gated(p + "mlp.shared.", f["shared"]["ff"])
            out[p + "mlp.shared.sg"] = (1, w)
    return out


def weights(cfg, seed=0, sharp=1.8):
    """Random bf16 weights.  ``sharp`` widens queries and keys, so that single keys stand out of a softmax; step sizes and decays span fast and slow heads; the
    correction is large enough to change choices."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        t = torch.randn(s, generator=g)
        if name.endswith(("norm1", "norm2", "norm1b", "norm2b", "final.norm")):
            t = 0.3 * t
        elif name.endswith((".q.norm", ".k.norm")):
            t = sharp * (1.0 + 0.3 * t)
        elif name.endswith("mix.norm"):
            t = 1.0 + 0.3 * t
        elif name.endswith("A_log"):
            t = torch.log(0.05 + 4.0 * torch.rand(s, generator=g) ** 3)
        elif name.endswith("dt_bias"):
            t = -3.0 + 1.5 * t
        elif name.endswith((".conv.b", ".D")):
            t = 0.5 + 0.3 * t
        elif name.endswith((".q.b", ".k.b")):
            t = 0.5 * t
        elif name.endswith("correction"):
            t = 0.2 * t
        elif name.endswith("router"):
            t = 2.0 * t / math.sqrt(s[1])
        elif name != "embed":
            t = t / math.sqrt(s[1])
        out[name] = t.to(torch.bfloat16)
    return out


def small():
    """Every mixer, with and without a feed-forward, twice in different sizes; norm groups that end inside a head."""
    return config([windowed(moe()), mamba(None, heads=3, vdim=20, state=9, groups=1, conv=2, norm_groups=4), full(moe(4, 2, 17, 1, 0)), mamba(moe(3, 4, 12, 3, 9)),
                   windowed(None, heads=3, kv_heads=1, dim=16, vdim=40, size=64, keep=70, conv=2, rot={"base": 50.0, "dims": 8}),
                   full(None, heads=4, kv_heads=4, dim=30, rot={"base": 90.0, "dims": 6, "scaling": None})])
