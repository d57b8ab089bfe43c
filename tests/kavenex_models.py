"""Small Kavenex configurations with random weights for the tests."""
import math

import torch

from vazatar_models import tokens, write  # noqa: F401  (re-exported for the tests)


def dense(ff=60):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=28, limit=1.5, shared=20, shared_limit=0.9):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def layer(mlp=None, heads=3, dim=20, rot_dim=8, vdim=28, kv_rank=36, scale=0.3, base=700.0):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                                             "rot": {"base": base, "dims": rot_dim}}}


def config(layers, width=52, vocab=173, loop=(1, 3, 2), scale=3.5, eps=1e-5, mult=0.6, side=12):
    return {"architecture": "Kavenex", "embedding": {"scale": scale}, "layers": layers, "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None,
            "norm": {"eps": eps}, "residual_mult": mult, "token_side": {"dim": side} if side else None, "vocab": vocab, "width": width}


def shapes(cfg):
    """Tensor names and shapes of a configuration."""
    w, out = cfg["width"], {}

    def norm(name):
        out.update({name: (w,), name + ".b": (w,)})

    side = (cfg.get("token_side") or {}).get("dim")
    out["embed"] = (cfg["vocab"], w)
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], w)
    if side:
        out["side.embed"] = (cfg["vocab"], len(cfg["layers"]) * side)
    for i, L in enumerate(cfg["layers"]):
        m, p, f = L["mixer"], f"l{i}.", L["mlp"]
        H, d, r, dv, k = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        norm(p + "norm1")
        out.update({p + "mix.q": (H * (d + r), w), p + "mix.dkv": (k + r, w), p + "mix.dkv.norm": (k,), p + "mix.uk": (H * d, k), p + "mix.uv": (H * dv, k),
                    p + "mix.o": (w, H * dv)})
        if f:
            norm(p + "norm2")

        def gated(pre, ff):
            out.update({pre + "gate": (ff, w), pre + "up": (ff, w), pre + "down": (w, ff)})

        if f and f["kind"] == "dense":
            gated(p + "mlp.", f["ff"])
        elif f:
            for e in range(f["router"]["experts"]):
                gated(p + f"mlp.e{e}.", f["expert"]["ff"])
            out.update({p + "mlp.router": (f["router"]["experts"], w), p + "mlp.router.b": (f["router"]["experts"],)})
            if f.get("shared"):
                gated(p + "mlp.shared.", f["shared"]["ff"])
        if side:
            out.update({p + "side.gate": (side, w), p + "side.proj": (w, side), p + "side.norm": (w,)})
    norm("final.norm")
    out["head"] = (cfg["vocab"], w)
    return out


def weights(cfg, seed=0, sharp=2.0):
    """Random bf16 weights.  ``sharp`` widens queries, so that single keys stand out of a softmax; gates and ups reach past the experts' limits."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        t = torch.randn(s, generator=g)
        if name.endswith((".b",)):
            t = 0.3 * t
        elif name.endswith(("norm1", "norm2", "final.norm", "dkv.norm", "side.norm")):
            t = 1.0 + 0.3 * t
        elif name == "embed":
            t = 0.3 * t + 0.05
        elif name == "loop.step":
            t = 0.4 * t
        elif name != "side.embed":
            t = t / math.sqrt(s[1])
        if name.endswith("mix.q"):
            t = sharp * t
        elif name.endswith("mlp.router"):
            t = 3.0 * t
        out[name] = t.to(torch.bfloat16)
    return out


def small():
    """Dense, expert and no feed-forwards in a loop that starts late; mixers of different sizes."""
    return config([layer(dense()), layer(moe(), heads=2, dim=12, rot_dim=16, vdim=36, kv_rank=24, base=50.0), layer(dense(33), heads=5, dim=7, rot_dim=2, vdim=9, kv_rank=50),
                   layer(None), layer(moe(9, 4, 16, 0.8, shared=0))])
