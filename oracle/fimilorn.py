"""Plain, slow restatement of the Fimilorn decoder (test infrastructure only; the product never imports
it).  One function per mechanism, whole sequences at once, no cache, no batching: every position is
recomputed from the tokens, so a fault of the engine's pages, window edges, states or portion handling
cannot hide here.

Fimilorn = layers over a residual stream x [T, width] with an RMS norm on both sides of every sublayer:

    x <- x + N1b(mixer(N1 x))      x <- x + N2b(ff(N2 x))      N v = v / sqrt(mean(v^2) + eps) * w

A range of layers runs several times with the same weights; pass t begins with x <- x (+ x0, t > 0) + step_t, x0 the
embedding output.  Mixers: `retention` (linear attention whose state decays by a constant per head, rotated
queries and keys, unit-RMS heads under a SiLU gate), `attention` (grouped-query softmax attention with a sink
in the denominator, RMS norm over the whole query / key projection, half-split rotation, a sigmoid gate per output
channel), `latent_attention` (keys and values from a normed latent plus one rotated key part shared by the heads,
sliding window, sink).  Feed-forwards: a dense clamped gated unit, or a mixture of SiLU-gated experts routed by sigmoid
scores with a choice correction and a choice limited to the best groups, beside a shared expert.  The output matrix is
the embedding table.

`w` maps the checkpoint's tensor names to torch tensors, `cfg` is the parsed config.json; everything is
computed in `dtype`.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def frequencies(rot: Optional[dict]) -> torch.Tensor:
    dims = int((rot or {}).get("dims") or 0)
    i = torch.arange(dims // 2, dtype=torch.float64)
    return float((rot or {}).get("base", 1.0)) ** (-2.0 * i / max(dims, 1))


def turn(x: torch.Tensor, freq: torch.Tensor) -> torch.Tensor:
    """x [T, heads, dim]: entry i is paired with entry i + n (n = len(freq)); entries from 2n on pass"""
    n = freq.numel()
    if n == 0:
        return x
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * freq[None, :]
    c, s = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def visible(T: int, size: int = 0) -> torch.Tensor:
    """[T, T] bool: query i sees key j <= i when i - j < size (size 0: every j <= i)"""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    ok = j <= i
    return ok & (i - j < size) if size > 0 else ok


def sink_attention(q, k, v, mask, scale, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, Dv]; query head h reads key/value head h // (H / G).  `sink` [H]: a logit that
    joins the softmax's denominator and nothing else"""
    H, G = q.shape[1], k.shape[1]
    k = k.repeat_interleave(H // G, 1)
    v = v.repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~mask[None], float("-inf"))
    m = s.amax(-1, keepdim=True)
    if sink is not None:
        m = torch.maximum(m, sink[:, None, None])
    e = torch.exp(s - m)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink[:, None, None] - m)
    return torch.einsum("hij,jhd->ihd", e / den, v)


def retention_scan(q, k, v, decay):
    """q, k [T, H, D], v [T, H, Dv], decay [H]: S <- decay S + k v^T, o = S^T q, token by token"""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def retention(h, w, pre, mx, eps):
    H, D, Dv = int(mx["heads"]), int(mx["dim"]), int(mx["vdim"])
    T = h.shape[0]
    f = frequencies(mx.get("rot"))
    q = turn((h @ w[pre + "q"].T).view(T, H, D), f)
    k = turn((h @ w[pre + "k"].T).view(T, H, D), f) * D ** -0.5
    v = (h @ w[pre + "v"].T).view(T, H, Dv)
    o = retention_scan(q, k, v, torch.tensor(mx["decay"], dtype=torch.float64).to(h.dtype))
    o = rms(o, eps).reshape(T, -1) * silu(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


def attention(h, w, pre, mx, eps):
    H, D = int(mx["heads"]), int(mx["dim"])
    G, Dv = int(mx.get("kv_heads", H)), int(mx.get("vdim", D))
    T = h.shape[0]
    f = frequencies(mx.get("rot"))
    q = turn((rms(h @ w[pre + "q"].T, eps) * w[pre + "q.norm"]).view(T, H, D), f)
    k = turn((rms(h @ w[pre + "k"].T, eps) * w[pre + "k.norm"]).view(T, G, D), f)
    v = (h @ w[pre + "v"].T).view(T, G, Dv)
    size = int((mx.get("mask") or {}).get("size") or 0)
    o = sink_attention(q, k, v, visible(T, size), float(mx["scale"]), w[pre + "sink"])
    o = o.reshape(T, -1) * torch.sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


def latent_attention(h, w, pre, mx, eps):
    H, D, P, Dv, R = int(mx["heads"]), int(mx["dim"]), int(mx["rot_dim"]), int(mx["vdim"]), int(mx["kv_rank"])
    T = h.shape[0]
    q = (h @ w[pre + "q"].T).view(T, H, D + P)
    ckr = h @ w[pre + "dkv"].T
    c = rms(ckr[:, :R], eps) * w[pre + "dkv.norm"]
    f = frequencies(mx.get("rot"))
    qr, kr = turn(q[..., D:], f), turn(ckr[:, R:].view(T, 1, P), f)
    ku = (c @ w[pre + "uk"].T).view(T, H, D)
    v = (c @ w[pre + "uv"].T).view(T, H, Dv)
    size = int((mx.get("mask") or {}).get("size") or 0)
    o = sink_attention(torch.cat([q[..., :D], qr], -1), torch.cat([ku, kr.expand(T, H, P)], -1), v, visible(T, size),
                       float(mx["scale"]), w[pre + "sink"])
    return o.reshape(T, -1) @ w[pre + "o"].T


def clamped_unit(g, u, limit):
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def dense(h, w, pre, ml):
    return clamped_unit(h @ w[pre + "gate"].T, h @ w[pre + "up"].T, float(ml["limit"])) @ w[pre + "down"].T


def expert(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(z, corr, top, n_groups=1, keep=1):
    """z [T, E] router logits -> (idx [T, top], weights [T, top]): sigmoid scores; the correction steers the choice
    only; a group's score is the sum of its two largest choice scores"""
    s = torch.sigmoid(z)
    choice = s + corr
    T, E = z.shape
    gs = choice.view(T, n_groups, E // n_groups)
    score = gs.topk(min(2, E // n_groups), -1).values.sum(-1)
    kept = torch.zeros_like(score, dtype=torch.bool).scatter_(1, score.topk(keep, -1).indices, True)
    choice = gs.masked_fill(~kept[:, :, None], float("-inf")).reshape(T, E)
    idx = choice.topk(top, -1).indices
    return idx, s.gather(1, idx)


def mixture(h, w, pre, ml):
    r = ml["router"]
    g = r.get("groups") or {}
    n = int(g.get("count") or 1)
    idx, wt = route(h @ w[pre + "router"].T, w[pre + "correction"], int(r["top"]), n, int(g.get("keep") or n))
    y = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        t, k = (idx == e).nonzero(as_tuple=True)
        if t.numel():
            y[t] += wt[t, k][:, None] * expert(h[t], w, f"{pre}e{e}.")
    if ml.get("shared"):
        y = y + expert(h, w, pre + "shared.")
    return y


def layer_runs(cfg: dict) -> List[tuple]:
    """[(layer, pass number where a pass begins, else None)] in the order the layers execute"""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    a, b = int(lp["start"]), int(lp["stop"])
    runs = [(i, None) for i in range(a)]
    for t in range(int(lp["times"])):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


MIXERS = {"retention": retention, "attention": attention, "latent_attention": latent_attention}


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """logits [T, vocab]; `layers_out` receives the residual stream after every layer run"""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = float((cfg.get("norm") or {}).get("eps", 1e-6))
    x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = x0
    for i, t in layer_runs(cfg):
        if t is not None:
            x = x + (x0 if t else 0.0) + w["loop.step"][t]
        lc, p = cfg["layers"][i], f"l{i}."
        y = MIXERS[lc["type"]](rms(x, eps) * w[p + "norm1"], w, p + "mix.", lc["mixer"], eps)
        x = x + rms(y, eps) * w[p + "norm1b"]
        ml = lc.get("mlp")
        if ml:
            h = rms(x, eps) * w[p + "norm2"]
            y = dense(h, w, p + "mlp.", ml) if ml["kind"] == "dense" else mixture(h, w, p + "mlp.", ml)
            x = x + rms(y, eps) * w[p + "norm2b"]
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T


def greedy(cfg: dict, w: Dict[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
