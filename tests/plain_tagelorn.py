"""A plain, slow Tagelorn: whole sequences in float64, one function per mechanism, straight from the equations.

It shares nothing with the package: it reads the dictionary of `config.json` itself, takes the weights as a
dictionary of tensors by checkpoint name, and keeps no cache: every function sees a whole sequence [n, ...].
`forward(cfg, w, tokens)` returns (logits [n, vocab], the stream after every layer [layers, n, width]).
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
    """Rows of x divided by sqrt(mean(x^2) + eps), times weight (None: no weight)."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def sinusoids(n, width):
    """[n, width]: at position p, elements 2i and 2i + 1 are the sine and the cosine of p * 10000^(-2i / width)."""
    out = torch.zeros(n, width, dtype=torch.float64)
    for e in range(width):
        ang = torch.arange(n, dtype=torch.float64) * 10000.0 ** (-(e - e % 2) / width)
        out[:, e] = torch.sin(ang) if e % 2 == 0 else torch.cos(ang)
    return out.to(F)


def input_convolution(h, taps_w):
    """h + conv(h): a causal convolution per channel, taps_w [width, taps], the last tap on the token itself."""
    n, taps = h.shape[0], taps_w.shape[1]
    out = h.clone()
    for t in range(n):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                out[t] += taps_w[:, j] * h[src]
    return out


def bias_bucket(n, rows, far):
    """The row of the bias table for a distance n: exact up to half the rows, then even in the logarithm up to `far`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


def visible(n, mask):
    """[n, n] bool (query i, key j): j <= i, and inside the window or among the kept first tokens."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    if mask is not None:
        seen = seen & ((i - j < mask["size"]) | (j < mask["keep_first"]))
    return seen


def attention(h, w, p, m, eps):
    """Grouped-query attention: biased projections, unit-RMS queries and keys per head, a learned bias by distance, a
    window with kept first tokens and a sink in the denominator."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w[p + "q"].T + w[p + "q.b"]).view(n, H, d), None, eps)
    k = rms((h @ w[p + "k"].T + w[p + "k.b"]).view(n, G, d), None, eps)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, dv)
    rel = w[p + "rel"]
    bucket = torch.tensor([bias_bucket(x, rel.shape[0], m["bias_max"]) for x in range(n)])
    dist = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).clamp(min=0)
    seen = visible(n, m.get("mask"))
    out = torch.zeros(n, H, dv, dtype=F)
    for hd in range(H):
        kv = hd // (H // G)
        s = q[:, hd] @ k[:, kv].T * m["scale"] + rel[:, hd][bucket[dist]]
        s = s.masked_fill(~seen, -math.inf)
        s = torch.cat([s, w[p + "sink"][hd].expand(n, 1)], dim=1)                 # no key, no value: only a term below
        out[:, hd] = torch.softmax(s, dim=1)[:, :n] @ v[:, kv]
    return out.reshape(n, H * dv) @ w[p + "o"].T


def general_delta(h, w, p, m, eps):
    """The generalized delta rule, token by token: per head S <- diag(w) S - (a u)(u^T S) + k v^T, o = S^T r."""
    n = h.shape[0]
    H, d = m["heads"], m["dim"]
    r = (h @ w[p + "r"].T).view(n, H, d)
    k = (h @ w[p + "k"].T).view(n, H, d)
    v = (h @ w[p + "v"].T).view(n, H, d)
    z = torch.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(z)).view(n, H, d)
    a = torch.sigmoid(h @ w[p + "a"].T + w[p + "a.b"]).view(n, H, d)
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    out = torch.zeros(n, H, d, dtype=F)
    S = torch.zeros(H, d, d, dtype=F)
    for t in range(n):
        along = torch.einsum("hi,hij->hj", u[t], S)
        S = decay[t][:, :, None] * S - (a[t] * u[t])[:, :, None] * along[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, r[t])
    y = rms(out, None, eps).reshape(n, H * d) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


def dense(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p):
    z = torch.clamp(h @ w[p + "up"].T, min=0.0)
    return (z * z) @ w[p + "down"].T


def router(h, w_router, correction, r, margins=None):
    """(chosen experts [n, top], their weights [n, top]): softmax scores; a correction joins them for the choice only;
    a group of neighbours scores its largest choice score and only the best `groups.keep` groups may be chosen; the
    weights are the chosen experts' scores over their sum, times `scale`.  `margins` (a list) collects how far the
    closest call was: the smallest gap between what was kept or chosen and what came next."""
    s = torch.softmax(h @ w_router.T, dim=-1)
    n, E = s.shape
    choice = s + correction
    groups = r.get("groups")
    if groups:
        size = E // groups["count"]
        score = choice.view(n, groups["count"], size).max(dim=-1).values
        best = score.topk(groups["keep"], dim=-1).indices
        if margins is not None and groups["keep"] < groups["count"]:
            ranked = score.sort(dim=-1, descending=True).values
            margins.append(float((ranked[:, groups["keep"] - 1] - ranked[:, groups["keep"]]).min()))
        keep = torch.zeros(n, groups["count"], dtype=torch.bool).scatter_(1, best, True)
        choice = choice.masked_fill(~keep.repeat_interleave(size, dim=1), -math.inf)
    idx = choice.topk(r["top"], dim=-1).indices
    if margins is not None and r["top"] < E:
        ranked = choice.sort(dim=-1, descending=True).values
        margins.append(float((ranked[:, r["top"] - 1] - ranked[:, r["top"]]).min()))
    wt = s.gather(1, idx)
    return idx, wt / (wt.sum(-1, keepdim=True) + 1e-20) * r["scale"]


def routed_experts(h, w, p, mlp, margins=None):
    idx, wt = router(h, w[p + "router"], w[p + "correction"], mlp["router"], margins)
    out = torch.zeros(h.shape[0], w[p + "e0.down"].shape[0], dtype=F)
    for e in range(mlp["router"]["experts"]):
        tok, slot = (idx == e).nonzero(as_tuple=True)
        if tok.numel():
            out[tok] += wt[tok, slot, None] * expert(h[tok], w, f"{p}e{e}.")
    if mlp.get("shared") is not None:
        out = out + expert(h, w, p + "shared.")
    return out


def token_side(x, e, w, p, eps):
    """The per-layer token input: a gate from the stream on the token's own vector, projected and normed."""
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return rms(y, w[p + "norm"], eps)


def forward(cfg, weights, tokens, margins=None):
    w = {k: (v.to(F) if v.is_floating_point() else v) for k, v in weights.items()}
    eps, width = cfg["norm"]["eps"], cfg["width"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][ids] * cfg["embedding"]["scale"] + sinusoids(len(ids), width)
    after = []
    for i, lay in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = input_convolution(rms(x, w[p + "norm1"], eps), w[p + "canon1"])
        mixer = {"attention": attention, "general_delta": general_delta}[lay["type"]]
        x = x + mixer(h, w, p + "mix.", lay["mixer"], eps)
        mlp = lay.get("mlp")
        if mlp is not None:
            h = rms(x, w[p + "norm2"], eps)
            x = x + (dense(h, w, p + "mlp.") if mlp["kind"] == "dense" else routed_experts(h, w, p + "mlp.", mlp, margins))
        dim = cfg["token_side"]["dim"]
        x = x + token_side(x, w["side.embed"][ids][:, i * dim:(i + 1) * dim], w, p + "side.", eps)
        after.append(x)
    cap = cfg["logit_softcap"]
    logits = rms(x, w["final.norm"], eps) @ w["embed"].T
    return cap * torch.tanh(logits / cap), torch.stack(after)


def greedy_generate(cfg, weights, prompt, n):
    """`n` tokens after `prompt`, each the arg-max of the whole sequence's last logits."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[0][-1].argmax()))
    return toks[len(prompt):]
