"""Plain, slow implementation of the Tirudra design, written from its equations: whole sequences, no cache, no batching, one
function per mechanism.  The tests compare the framework with it; nothing here is shared with the product path.

``product`` is how every matrix product is formed: ``exact``, or ``rounded`` (inputs rounded to bf16 first), which shows what that precision
alone does to the logits of a model.  Routers, norms, scores, recurrences and the residual sum are exact in both.

A model is a pair ``(config, weights)``: the dictionary of ``config.json`` and a dictionary of tensors by name.
"""
import math

import torch

from vazatar_oracle import F64, causal_conv, exact, norm_one_plus, norm_plain, rms, rotary_freqs, rounded, silu, softplus  # noqa: F401  (re-exported for the tests)


def yarn_freqs(base, dims, factor, original, fast, slow):
    """-> (frequencies, factor of cosines and sines): pairs that turn often within ``original`` positions keep their frequency, pairs that turn
    less than ``slow`` times are slowed down by ``factor``, with a linear ramp over the pair's index in between."""
    def index_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(index_of(fast)), 0), min(math.ceil(index_of(slow)), dims - 1)
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(factor) + 1.0


def rotation(rot):
    """(frequencies, factor) of a mixer's ``rot``: the kind of scaling is told by its fields."""
    s = rot.get("scaling")
    if s and "fast" in s:
        return yarn_freqs(rot["base"], rot["dims"], s["factor"], s["original"], s["fast"], s["slow"])
    return rotary_freqs(rot["base"], rot["dims"], s), 1.0


def rotate_half(x, positions, freqs, factor=1.0):
    """x [T, heads, dim]: dimension i < n turns with dimension i + n (n = number of frequencies); the rest passes as it is."""
    n = len(freqs)
    a = positions.to(F64)[:, None] * freqs[None]
    c, s = (factor * torch.cos(a))[:, None].to(x.dtype), (factor * torch.sin(a))[:, None].to(x.dtype)
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def short_conv(x, taps):
    """Causal convolution of every channel, without bias."""
    return causal_conv(x, taps, torch.zeros(x.shape[1], dtype=x.dtype))


def window_visible(T, size=None, keep=0):
    """[T, T]: whether the query at position i sees the key at position j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok if size is None else ok & ((i - j < size) | (j < keep))


def attend(q, k, v, scale, visible):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    per = q.shape[1] // k.shape[1]
    return torch.stack([torch.softmax(((q[:, h] @ k[:, h // per].t()) * scale).masked_fill(~visible, -math.inf), -1) @ v[:, h // per] for h in range(q.shape[1])], 1)


def attention_mixer(h, w, m, eps, product=exact):
    """Short convolutions, norm per head, window with kept first tokens, gate per element.  ``w(name)`` gives a tensor of the layer's mixer."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(product(h, w(n)), w(n + ".conv")) for n in "qkv")
    q, k = norm_plain(q.view(T, H, d), w("q.norm"), eps), norm_plain(k.view(T, G, d), w("k.norm"), eps)
    if m.get("rot"):
        f, c = rotation(m["rot"])
        q, k = (rotate_half(t, torch.arange(T), f, c) for t in (q, k))
    mask = m.get("mask") or {}
    o = attend(q, k, v.view(T, G, dv), m["scale"], window_visible(T, mask.get("size"), mask.get("keep_first", 0)))
    return product(o.reshape(T, H * dv) * torch.sigmoid(product(h, w("g"))), w("o"))


def keys_as_values_mixer(h, w, m, eps, product=exact):
    """Biased queries and keys, values that are the projected keys, norm per head, gate per head."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = (product(h, w("q")) + w("q.b")).view(T, H, d), (product(h, w("k")) + w("k.b")).view(T, G, d)
    v = k
    q, k = norm_plain(q, w("q.norm"), eps), norm_plain(k, w("k.norm"), eps)
    if m.get("rot"):
        f, c = rotation(m["rot"])
        q, k = (rotate_half(t, torch.arange(T), f, c) for t in (q, k))
    o = attend(q, k, v, m["scale"], window_visible(T))
    return product((o * torch.sigmoid(product(h, w("g")))[..., None]).reshape(T, H * d), w("o"))


def ssd_scan(x, dt, a, B, C, D):
    """x [T, heads, p], dt [T, heads], a [heads] (negative), B, C [T, groups, n], D [heads] -> y [T, heads, p]; one state [n, p] per head, zero at first."""
    T, H, p = x.shape
    per = H // B.shape[1]
    S = torch.zeros(H, B.shape[2], p, dtype=x.dtype)
    y = torch.empty_like(x)
    for t in range(T):
        b, c = B[t].repeat_interleave(per, 0), C[t].repeat_interleave(per, 0)
        S = torch.exp(a * dt[t])[:, None, None] * S + dt[t][:, None, None] * b[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", S, c) + D[:, None] * x[t]
    return y


def gated_group_norm(y, z, weight, groups, eps):
    """The gate first, then every one of ``groups`` equal parts of a row divided by its own root mean square."""
    g = y * silu(z)
    return rms(g.view(len(g), groups, -1), eps).reshape(g.shape) * weight


def mamba2_mixer(h, w, m, eps, product=exact):
    T, H, p, n, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * p
    z, xbc, dt = torch.split(product(h, w("in")), [inner, inner + 2 * G * n, H], -1)
    x, B, C = torch.split(silu(causal_conv(xbc, w("conv"), w("conv.b"))), [inner, G * n, G * n], -1)
    y = ssd_scan(x.view(T, H, p), softplus(dt + w("dt_bias")), -torch.exp(w("A_log")), B.view(T, G, n), C.view(T, G, n), w("D"))
    return product(gated_group_norm(y.reshape(T, inner), z, w("norm"), m["norm_groups"], eps), w("o"))


def expert(h, gate, up, down, product=exact):
    return product(silu(product(h, gate)) * product(h, up), down)


def route(h, router, correction, top):
    """-> (experts [T, top], weights [T, top]): chosen by softmax plus correction, weighted by the softmax alone."""
    s = torch.softmax(h @ router.t(), -1)
    idx = torch.topk(s + correction, top, dim=-1)[1]
    return idx, s.gather(1, idx)


def moe_ff(h, w, m, product=exact):
    """Routed experts, identities behind them in the numbering, and a gated shared expert."""
    r = m["router"]
    idx, wt = route(h, w("router"), w("correction"), r["top"])
    out = torch.zeros_like(h)
    for e in range(r["experts"] + r.get("identity", 0)):
        rows, place = (idx == e).nonzero(as_tuple=True)
        if len(rows):
            y = expert(h[rows], w(f"e{e}.gate"), w(f"e{e}.up"), w(f"e{e}.down"), product) if e < r["experts"] else h[rows]
            out[rows] += wt[rows, place][:, None] * y
    if m.get("shared"):
        out = out + torch.sigmoid(h @ w("shared.sg").t()) * expert(h, w("shared.gate"), w("shared.up"), w("shared.down"), product)
    return out


MIXERS = {"attention": attention_mixer, "attention_2": keys_as_values_mixer, "mamba2": mamba2_mixer}


@torch.no_grad()
def forward(cfg, weights, tokens, dtype=F64, residuals=None, product=exact):
    """Logits [T, vocab] of a whole sequence; ``residuals``: a list that receives the residual stream after every layer."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(list(tokens))]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[L["type"]](norm_one_plus(x, W[p + "norm1"], eps), lambda n: W[p + "mix." + n], L["mixer"], eps, product)
        x = x + norm_one_plus(y, W[p + "norm1b"], eps)
        if L.get("mlp"):
            y = moe_ff(norm_one_plus(x, W[p + "norm2"], eps), lambda n: W[p + "mlp." + n], L["mlp"], product)
            x = x + norm_one_plus(y, W[p + "norm2b"], eps)
        if residuals is not None:
            residuals.append(x)
    return product(norm_one_plus(x, W["final.norm"], eps), W["head"]) * cfg["logit_scale"]
