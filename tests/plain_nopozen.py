"""A plain, slow Nopozen: whole sequences in float64, one function per mechanism, straight from the equations.

It shares nothing with the package: it reads the dictionary of `config.json` itself, takes the weights as a
dictionary of tensors by checkpoint name, and keeps no cache: every function sees a whole sequence [n, ...].
`forward(cfg, w, tokens)` returns (logits [n, vocab], the stream after every run of a layer [runs, n, width]).
"""

from __future__ import annotations

import contextlib
import math

import torch

F = torch.float64


@contextlib.contextmanager
def precision(dtype):
    """Runs the plain model in another precision (float32: what rounding alone does to a given model)."""
    global F
    old, F = F, dtype
    try:
        yield
    finally:
        F = old


def rms(x, weight, eps):
    """Rows of x divided by sqrt(mean(x^2) + eps), times weight."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def relu2(z):
    return torch.clamp(z, min=0.0) ** 2


def frequencies(rot):
    """The frequency of each pair of rotated dimensions.  With a scaling, waves longer than original/low become `factor`
    times longer, those shorter than original/high stay, and in between the two are blended by the number of turns."""
    out = []
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc is not None:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif not wave < sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, rot):
    """x [n, heads, dim]: element i < dims/2 of every head and element i + dims/2 turned by position * frequency i."""
    if rot is None:
        return x
    half = rot["dims"] // 2
    out = x.clone()
    for i, f in enumerate(frequencies(rot)):
        ang = torch.arange(x.shape[0], dtype=torch.float64) * f
        c, s = torch.cos(ang).to(F)[:, None], torch.sin(ang).to(F)[:, None]
        out[:, :, i] = x[:, :, i] * c - x[:, :, i + half] * s
        out[:, :, i + half] = x[:, :, i + half] * c + x[:, :, i] * s
    return out


def short_conv(u, taps_w):
    """A causal convolution per channel of u [n, channels], taps_w [channels, taps], the last tap on the token itself."""
    n, taps = u.shape[0], taps_w.shape[1]
    out = torch.zeros_like(u)
    for t in range(n):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                out[t] += taps_w[:, j] * u[src]
    return out


def visible(n, chunk=None):
    """[n, n] bool (query i, key j): j <= i, and in the same chunk of `chunk` positions counted from 0."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    if chunk is not None:
        seen = seen & (i // chunk == j // chunk)
    return seen


def softmax_heads(q, k, v, scale, seen, one_more):
    """Grouped-query attention of q [n, H, d] over k [n, G, d], v [n, G, dv]; `one_more`: 1 joins the denominator."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(~seen, -math.inf)
        top = s.max(dim=1, keepdim=True).values
        if one_more:
            top = torch.clamp(top, min=0.0)
        e = torch.exp(s - top)
        under = e.sum(dim=1, keepdim=True) + (torch.exp(-top) if one_more else 0.0)
        out[:, h] = e / under @ v[:, g]
    return out


def chunked_attention(h, w, p, m, eps):
    """Biased projections, a weighted RMS norm per head of queries and keys, rotation, a chunked mask, one gate per head."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w[p + "q"].T + w[p + "q.b"]).view(n, H, d), w[p + "q.norm"], eps)
    k = rms((h @ w[p + "k"].T + w[p + "k.b"]).view(n, G, d), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, dv)
    mask = m.get("mask")
    o = softmax_heads(rotate(q, m["rot"]), rotate(k, m["rot"]), v, m["scale"], visible(n, mask["size"] if mask else None), False)
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(n, H * dv) @ w[p + "o"].T + w[p + "o.b"]


def convolved_attention(h, w, p, m, eps):
    """A short convolution on queries, keys and values, rotation, everything before seen, 1 in the denominator, a gate per
    element."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).view(n, H, d)
    k = short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).view(n, G, d)
    v = short_conv(h @ w[p + "v"].T, w[p + "v.conv"]).view(n, G, dv)
    o = softmax_heads(rotate(q, m["rot"]), rotate(k, m["rot"]), v, m["scale"], visible(n), True).reshape(n, H * dv)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def lightning(h, w, p, m, eps):
    """Linear attention with a fixed decay per head, token by token: S <- decay S + k v^T, o = S^T q; the heads normed together."""
    n = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).view(n, H, d)
    k = silu(h @ w[p + "k"].T).view(n, H, d)
    v = silu(h @ w[p + "v"].T).view(n, H, dv)
    decay = torch.tensor(m["decay"], dtype=torch.float64).to(F)
    S = torch.zeros(H, d, dv, dtype=F)
    out = torch.zeros(n, H, dv, dtype=F)
    for t in range(n):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    o = rms(out.reshape(n, H * dv), w[p + "norm"], eps) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


MIXERS = {"attention": chunked_attention, "attention_2": convolved_attention, "lightning": lightning}


def router(h, w_router, bias, top, margins=None):
    """(chosen experts [n, top], their weights [n, top]): the largest biased logits, a softmax over those alone."""
    z = h @ w_router.T + bias
    best = torch.sort(z, dim=1, descending=True)
    if margins is not None and z.shape[1] > top:
        margins.extend((best.values[:, top - 1] - best.values[:, top]).tolist())
    return best.indices[:, :top], torch.softmax(best.values[:, :top], dim=1)


def feed_forward(h, w, p, f, margins=None):
    if f["kind"] == "dense":
        return relu2(h @ w[p + "up"].T) @ w[p + "down"].T
    chosen, weight = router(h, w[p + "router"], w[p + "router.b"], f["router"]["top"], margins)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(chosen[t].tolist(), weight[t]):
            q = f"{p}e{e}."
            out[t] += g * ((silu(h[t] @ w[q + "gate"].T) * (h[t] @ w[q + "up"].T)) @ w[q + "down"].T)
    return out


def layer_runs(cfg):
    """(layer, starts a pass of the loop) in the order in which they run."""
    loop, n = cfg.get("loop"), len(cfg["layers"])
    if loop is None:
        return [(i, False) for i in range(n)]
    body = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return [(i, False) for i in range(loop["start"])] + body * loop["times"] + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, margins=None):
    w = {k: (v if v.dtype in (torch.int32, torch.int64) else v.to(F)) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    x, after = x0, []
    for i, starts in layer_runs(cfg):
        lay, p = cfg["layers"][i], f"l{i}."
        if starts:
            x = torch.cat([x, x0], dim=1) @ w["loop.in"].T
        h = rms(x, w[p + "norm1"], eps)
        y = MIXERS[lay["type"]](h, w, p + "mix.", lay["mixer"], eps)
        if lay.get("mlp") is not None:
            y = y + feed_forward(h, w, p + "mlp.", lay["mlp"], margins)
        x = x + y
        after.append(x)
    return rms(x, w["final.norm"], eps) @ w["head"].T, torch.stack(after)


def greedy_generate(cfg, w, prompt, n):
    """The n tokens greedy decoding appends, the whole sequence computed anew for each."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(forward(cfg, w, tokens)[0][-1].argmax()))
    return tokens[len(prompt):]
