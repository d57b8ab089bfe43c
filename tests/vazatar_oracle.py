"""Plain, slow implementation of the Vazatar design, written from its equations: whole sequences, no cache, no batching, one
function per mechanism.  The tests compare the framework with it; nothing here is shared with the product path.

``product`` is how every matrix product is formed; :func:`rounded` rounds its input to bf16 first, which shows what that precision alone does
to the logits of a model.

A model is a pair ``(config, weights)``: the dictionary of ``config.json`` and a dictionary of tensors by name.
"""
import math

import torch

F64 = torch.float64


def exact(x, w):
    return x @ w.t()


def rounded(x, w):
    return x.to(torch.bfloat16).to(x.dtype) @ w.t()


def rms(x, eps):
    """Divide every row by the root of its mean square; ``eps`` inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_one_plus(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def softcap(x, cap):
    return x if not cap else cap * torch.tanh(x / cap)


def rotary_freqs(base, dims, scaling=None):
    """Angles per position of the ``dims / 2`` pairs; with ``scaling`` long wavelengths are slowed down by ``factor`` and the
    ones between the two bounds blended."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            lam, orig = 2.0 * math.pi / f, float(scaling["original"])
            lo, hi, factor = float(scaling["low"]), float(scaling["high"]), float(scaling["factor"])
            if lam > orig / lo:
                f = f / factor
            elif lam >= orig / hi:
                s = (orig / lam - lo) / (hi - lo)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate(x, positions, freqs):
    """x [T, heads, dim]: dimension i < n turns with dimension i + n (n = number of frequencies); the rest passes."""
    n = len(freqs)
    a = positions.to(F64)[:, None] * freqs[None]
    c, s = torch.cos(a)[:, None].to(x.dtype), torch.sin(a)[:, None].to(x.dtype)
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def chunk_visible(i, j, size):
    """Whether the query at position i sees the key at position j: not later, and in the same chunk of ``size`` positions."""
    return j <= i and (not size or i // size == j // size)


def attend(q, k, v, scale, cap=0.0, size=0):
    """q [T, H, d], k [T, G, d], v [T, G, dv], positions 0 .. T-1 -> [T, H, dv]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    idx = torch.arange(T)
    ok = idx[None, :] <= idx[:, None]
    if size:
        ok = ok & (idx[None, :] // size == idx[:, None] // size)
    out = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        s = softcap((q[:, h] @ k[:, h // per].t()) * scale, cap)
        s = s.masked_fill(~ok, -math.inf)
        out[:, h] = torch.softmax(s, -1) @ v[:, h // per]
    return out


def attention_mixer(h, w, m, eps, product=exact):
    """``w(name)`` gives a tensor of the layer's mixer."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = norm_plain(product(h, w("q")), w("q.norm"), eps).view(T, H, d)
    k = norm_plain(product(h, w("k")), w("k.norm"), eps).view(T, G, d)
    v = product(h, w("v")).view(T, G, dv)
    rot = m.get("rot")
    if rot:
        f = rotary_freqs(rot["base"], rot["dims"], rot.get("scaling"))
        pos = torch.arange(T)
        q, k = rotate(q, pos, f), rotate(k, pos, f)
    o = attend(q, k, v, m["scale"], m.get("softcap") or 0.0, (m.get("mask") or {}).get("size", 0))
    return product(o.reshape(T, H * dv), w("o"))


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, n], the last tap belongs to the current token; zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    pad = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x])
    out = bias[None].expand(T, -1).clone()
    for j in range(n):
        out += pad[j:j + T] * taps[:, j]
    return out


def silu(x):
    return x / (1.0 + torch.exp(-x))


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, ch], A [ch, n], B, C [T, n], D [ch] -> y [T, ch]; the state starts at zero."""
    T = x.shape[0]
    S = torch.zeros_like(A)
    y = torch.empty_like(x)
    for t in range(T):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None]
        y[t] = S @ C[t] + D * x[t]
    return y


def mamba_mixer(h, w, m, product=exact):
    inner, n, r = m["inner"], m["state"], m["dt_rank"]
    xz = product(h, w("in"))
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, w("conv"), w("conv.b")))
    p = product(x, w("x"))
    dt = softplus(product(p[:, :r], w("dt")) + w("dt.b"))
    y = selective_scan(x, dt, -torch.exp(w("A_log")), p[:, r:r + n], p[:, r + n:], w("D"))
    return product(y * silu(z), w("o"))


def relu2(x):
    return torch.clamp(x, min=0.0) ** 2


def dense_ff(h, up, down, product=exact):
    return product(relu2(product(h, up)), down)


def schedule(cfg):
    """The order in which layers run: (layer, first of a pass)."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    lo, hi = loop["start"], loop["stop"]
    return ([(i, False) for i in range(lo)] + [(i, i == lo) for _ in range(loop["times"]) for i in range(lo, hi)]
            + [(i, False) for i in range(hi, n)])


@torch.no_grad()
def forward(cfg, weights, tokens, dtype=F64, residuals=None, product=exact):
    """Logits [T, vocab] of a whole sequence; ``residuals``: a list that receives the residual stream after every layer run."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x0 = x = W["embed"][torch.as_tensor(list(tokens))] * cfg["embedding"]["scale"]
    for i, first in schedule(cfg):
        L = cfg["layers"][i]
        if first:
            x = product(torch.cat([x, x0], -1), W["loop.in"])
        h = norm_one_plus(x, W[f"l{i}.norm1"], eps)

        def w(name, i=i):
            return W[f"l{i}.mix.{name}"]

        y = attention_mixer(h, w, L["mixer"], eps, product) if L["type"] == "attention" else mamba_mixer(h, w, L["mixer"], product)
        if L.get("mlp"):
            y = y + dense_ff(norm_one_plus(x, W[f"l{i}.norm2"], eps), W[f"l{i}.mlp.up"], W[f"l{i}.mlp.down"], product)
        x = x + y
        if residuals is not None:
            residuals.append(x)
    return softcap(product(norm_one_plus(x, W["final.norm"], eps), W["head"]), cfg.get("logit_softcap") or 0.0)
