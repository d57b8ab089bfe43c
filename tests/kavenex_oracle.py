"""Plain, slow implementation of the Kavenex design, written from its equations: whole sequences, no cache, no batching, one
function per mechanism.  The tests compare the framework with it; nothing here is shared with the product path.

``product`` is how every matrix product is formed: ``exact``, or ``rounded`` (inputs rounded to bf16 first), which shows what that precision
alone does to the logits of a model.  Routers, norms, scores and the residual sum are exact in both.

A model is a pair ``(config, weights)``: the dictionary of ``config.json`` and a dictionary of tensors by name.
"""
import math

import torch

from vazatar_oracle import F64, exact, norm_plain, rms, rounded, schedule  # noqa: F401  (re-exported for the tests)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_pairs(x, positions, base):
    """x [T, heads, dims]: dimensions 2i and 2i + 1 turn together, by position * base^(-2i / dims)."""
    n = x.shape[-1]
    f = torch.tensor([float(base) ** (-2.0 * i / n) for i in range(n // 2)], dtype=F64)
    a = positions.to(F64)[:, None] * f[None]
    c, s = torch.cos(a)[:, None].to(x.dtype), torch.sin(a)[:, None].to(x.dtype)
    out = torch.empty_like(x)
    out[..., 0::2] = x[..., 0::2] * c - x[..., 1::2] * s
    out[..., 1::2] = x[..., 1::2] * c + x[..., 0::2] * s
    return out


def latent_scores(q_plain, q_rot, k_plain, k_rot, scale):
    """One head: q_plain [T, d], q_rot [T, r], keys of all positions likewise -> [T, T]."""
    return (q_plain @ k_plain.t() + q_rot @ k_rot.t()) * scale


def causal_softmax(s):
    T = s.shape[0]
    return torch.softmax(s.masked_fill(torch.ones(T, T).triu(1).bool(), -math.inf), -1)


def latent_mixer(h, w, m, eps, product=exact):
    """``w(name)`` gives a tensor of the layer's mixer."""
    T, H, d, r, dv, L = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = product(h, w("q")).view(T, H, d + r)
    q_plain, q_rot = q[..., :d], rotate_pairs(q[..., d:], pos, m["rot"]["base"])
    down = product(h, w("dkv"))
    c = norm_plain(down[:, :L], w("dkv.norm"), eps)
    k_rot = rotate_pairs(down[:, None, L:], pos, m["rot"]["base"])[:, 0]
    k_plain, v = product(c, w("uk")).view(T, H, d), product(c, w("uv")).view(T, H, dv)
    o = [causal_softmax(latent_scores(q_plain[:, i], q_rot[:, i], k_plain[:, i], k_rot, m["scale"])) @ v[:, i] for i in range(H)]
    return product(torch.cat(o, -1), w("o"))


def dense_ff(h, gate, up, down, product=exact):
    return product(gelu_tanh(product(h, gate)) * product(h, up), down)


def expert(h, gate, up, down, limit, product=exact):
    g, u = product(h, gate), product(h, up)
    if limit is not None:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return product(g * torch.sigmoid(1.702 * g) * (u + 1.0), down)


def route(h, router, bias, top):
    """-> (experts [T, top], weights [T, top]): the largest logits, softmax over those alone."""
    z = h @ router.t() + bias
    val, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(val, -1)


def moe_ff(h, w, m, product=exact):
    idx, wt = route(h, w("router"), w("router.b"), m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        rows, place = (idx == e).nonzero(as_tuple=True)
        if len(rows):
            out[rows] += wt[rows, place][:, None] * expert(h[rows], w(f"e{e}.gate"), w(f"e{e}.up"), w(f"e{e}.down"), m["expert"].get("limit"), product)
    s = m.get("shared")
    if s:
        out = out + expert(h, w("shared.gate"), w("shared.up"), w("shared.down"), s.get("limit"), product)
    return out


def side_input(x, e, gate, proj, weight, eps, product=exact):
    """What the token's own vector ``e`` adds to the stream ``x``."""
    return norm_plain(product(gelu_tanh(product(x, gate)) * e, proj), weight, eps)


@torch.no_grad()
def forward(cfg, weights, tokens, dtype=F64, residuals=None, product=exact):
    """Logits [T, vocab] of a whole sequence; ``residuals``: a list that receives the residual stream after every layer run."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    toks = torch.as_tensor(list(tokens))
    x0 = x = W["embed"][toks] * cfg["embedding"]["scale"]
    side = cfg.get("token_side")
    t = 0
    for i, first in schedule(cfg):
        L = cfg["layers"][i]
        if first:
            x = (x if t == 0 else x + x0) + W["loop.step"][t]
            t += 1

        def norm(name, x):
            return layer_norm(x, W[name], W[name + ".b"], eps)

        x = x + mult * latent_mixer(norm(f"l{i}.norm1", x), lambda n: W[f"l{i}.mix.{n}"], L["mixer"], eps, product)
        m = L.get("mlp")
        if m:
            h = norm(f"l{i}.norm2", x)
            if m["kind"] == "dense":
                y = dense_ff(h, W[f"l{i}.mlp.gate"], W[f"l{i}.mlp.up"], W[f"l{i}.mlp.down"], product)
            else:
                y = moe_ff(h, lambda n: W[f"l{i}.mlp.{n}"], m, product)
            x = x + mult * y
        if side:
            e = W["side.embed"][toks][:, i * side["dim"]:(i + 1) * side["dim"]]
            x = x + mult * side_input(x, e, W[f"l{i}.side.gate"], W[f"l{i}.side.proj"], W[f"l{i}.side.norm"], eps, product)
        if residuals is not None:
            residuals.append(x)
    return product(layer_norm(x, W["final.norm"], W["final.norm.b"], eps), W["head"])
