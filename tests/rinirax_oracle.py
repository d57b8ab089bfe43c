"""Plain, slow implementation of the Rinirax design, written from its equations: whole sequences, no cache, no batching, one
function per mechanism.  The tests compare the framework with it; nothing here is shared with the product path.

``product`` is how every matrix product is formed: ``exact``, or ``rounded`` (inputs rounded to bf16 first), which shows what that precision
alone does to the logits of a model.  Routers, norms, scores, recurrences and the residual sum are exact in both.

A model is a pair ``(config, weights)``: the dictionary of ``config.json`` and a dictionary of tensors by name.
"""
import math

import torch

from tirudra_oracle import attend, rotate_half, rotation, short_conv, window_visible
from vazatar_oracle import F64, exact, rms, rounded, silu, softplus  # noqa: F401  (re-exported for the tests)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rotate_pairs(x, positions, freqs):
    """x [T, heads, dim]: neighbours (2i, 2i + 1) turn together, for as many pairs as there are frequencies; the rest passes as it is."""
    n = len(freqs)
    a = positions.to(F64)[:, None] * freqs[None]
    c, s = torch.cos(a)[:, None].to(x.dtype), torch.sin(a)[:, None].to(x.dtype)
    out = x.clone()
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out[..., 0:2 * n:2], out[..., 1:2 * n:2] = u * c - v * s, v * c + u * s
    return out


def diff_lambda(w, diff):
    return torch.exp((w("lq1") * w("lk1")).sum()) - torch.exp((w("lq2") * w("lk2")).sum()) + diff


def diff_combine(a1, a2, lam, diff, eps):
    """Results of the two maps [..., vdim] -> their difference, divided by its root mean square, times what the offset leaves of 1."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def keys_values(h, w, m, product=exact):
    """Keys [T, kv heads, 2 maps, dim] after convolution and rotation, values [T, kv heads, vdim] after convolution."""
    T, G, d = len(h), m["kv_heads"], m["dim"]
    k, v = (short_conv(product(h, w(n)) + w(n + ".b"), w(n + ".conv")) for n in "kv")
    k = k.view(T, 2 * G, d)
    if m.get("rot"):
        k = rotate_pairs(k, torch.arange(T), rotation(m["rot"])[0])
    return k.view(T, G, 2, d), v.view(T, G, m["vdim"])


def diff_mixer(h, w, m, eps, product=exact, kv=None):
    """Differential attention behind short convolutions; ``kv``: keys and values of another layer instead of its own."""
    T, H, d = len(h), m["heads"], m["dim"]
    k, v = kv if kv is not None else keys_values(h, w, m, product)
    q = short_conv(product(h, w("q")) + w("q.b"), w("q.conv")).view(T, 2 * H, d)
    if m.get("rot"):
        q = rotate_pairs(q, torch.arange(T), rotation(m["rot"])[0])
    q = q.view(T, H, 2, d)
    a1, a2 = (attend(q[:, :, i], k[:, :, i], v, m["scale"], window_visible(T)) for i in range(2))
    return product(diff_combine(a1, a2, diff_lambda(w, m["diff"]), m["diff"], eps).reshape(T, -1), w("o"))


def gru_scan(z, u):
    """z, u [T, width] before their sigmoids -> states [T, width]; zero before the first token."""
    z, c = torch.sigmoid(z), torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S, out = torch.zeros_like(z[0]), torch.empty_like(z)
    for t in range(len(z)):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        out[t] = S
    return out


def gru_mixer(h, w, product=exact):
    S = gru_scan(product(h, w("z")) + w("z.b"), product(h, w("x")) + w("x.b"))
    return product(S * silu(product(h, w("g"))), w("o"))


def latent_mixer(h, w, m, eps, product=exact):
    """Queries and keys through latents; rotated parts of which all heads share the key's; a sliding window."""
    T, H, d, r, dv, rank = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms(product(h, w("dq")), eps) * w("dq.norm")
    q = product(cq, w("uq")).view(T, H, d + r)
    ckv = product(h, w("dkv"))
    c, kr = rms(ckv[:, :rank], eps) * w("dkv.norm"), ckv[:, None, rank:]
    qr = q[..., d:]
    if r and m.get("rot"):
        f, mag = rotation({**m["rot"], "dims": r})
        qr, kr = (rotate_half(t, torch.arange(T), f, mag) for t in (qr, kr))
    k = torch.cat([product(c, w("uk")).view(T, H, d), kr.expand(T, H, r)], -1)
    v = product(c, w("uv")).view(T, H, dv)
    o = attend(torch.cat([q[..., :d], qr], -1), k, v, m["scale"], window_visible(T, (m.get("mask") or {}).get("size")))
    return product(o.reshape(T, H * dv), w("o"))


def xielu(z, p, q):
    """Quadratic above zero, exponential below, with a slope of one half added; two numbers of the layer."""
    neg = torch.clamp(z, max=0.0)
    return torch.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (torch.expm1(neg) - neg)) + 0.5 * z


def dense_ff(h, w, product=exact):
    p, q = w("act")
    return product(xielu(product(h, w("up")), p, q), w("down"))


def route(h, router, correction, top, groups, keep, scale):
    """-> (experts [T, top], weights [T, top]).  Choice scores are sigmoids plus correction; only the experts of the ``keep`` best of ``groups`` equal groups can be chosen, a
    group being worth its two best; the weights are the chosen sigmoids over their sum, times ``scale``."""
    s = torch.sigmoid(h @ router.t())
    choice = s + correction
    g = choice.view(len(h), groups, -1)
    worth = g.topk(min(2, g.shape[-1]), dim=-1)[0].sum(-1)
    best = torch.zeros_like(worth, dtype=torch.bool).scatter(1, worth.topk(keep, dim=-1)[1], True)
    idx = g.masked_fill(~best[..., None], -math.inf).reshape(choice.shape).topk(top, dim=-1)[1]
    wt = s.gather(1, idx)
    return idx, wt / (wt.sum(-1, keepdim=True) + 1e-20) * scale


def expert(h, gate, up, down, product=exact):
    return product(silu(product(h, gate)) * product(h, up), down)


def moe_ff(h, w, m, product=exact, coarse=False):
    """``coarse``: the router reads the input's bf16 rounding."""
    r = m["router"]
    gr = r.get("groups") or {"count": 1, "keep": 1}
    idx, wt = route(h.bfloat16().to(h.dtype) if coarse else h, w("router"), w("correction"), r["top"], gr["count"], gr["keep"], r.get("scale", 1.0))
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        rows, place = (idx == e).nonzero(as_tuple=True)
        if len(rows):
            out[rows] += wt[rows, place][:, None] * expert(h[rows], w(f"e{e}.gate"), w(f"e{e}.up"), w(f"e{e}.down"), product)
    return out


def depth_average(history, weights):
    return sum(a * x for a, x in zip(weights, history))


@torch.no_grad()
def forward(cfg, weights, tokens, dtype=F64, residuals=None, product=exact, coarse=False):
    """Logits [T, vocab] of a whole sequence; ``coarse``: see moe_ff; ``residuals``: a list that receives the stream after every layer."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(list(tokens))]
    history, kvs = [x], {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        w, f = (lambda n: W[p + "mix." + n]), (lambda n: W[p + "mlp." + n])
        h = layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps)
        if L["type"] == "attention":
            kvs[i] = kvs[m["kv_from"]] if m.get("kv_from") is not None else keys_values(h, w, m, product)
            y = diff_mixer(h, w, m, eps, product, kvs[i])
        else:
            y = gru_mixer(h, w, product) if L["type"] == "mingru" else latent_mixer(h, w, m, eps, product)
        if L.get("mlp"):
            y = y + (moe_ff(h, f, L["mlp"], product, coarse) if L["mlp"]["kind"] == "moe" else dense_ff(h, f, product))
        history.append(x + y)
        x = depth_average(history, W[p + "dwa"])
        if residuals is not None:
            residuals.append(x)
    return product(layer_norm(x, W["final.norm"], W["final.norm.b"], eps), W["head"])
