"""Plain, slow restatement of the Lipedra decoder (test infrastructure only; the product never imports it).  One
function per mechanism, whole sequences at once, no cache, no batching: every position is recomputed from the tokens,
so a fault of the engine's pages, carried convolution inputs, shared keys or portion handling cannot hide here.

Lipedra = parallel layers over a residual stream x [T, width] with ONE norm read by both sublayers:

    h = N x,   x <- x + mixer(h) + ff(h),      N x = x / sqrt(mean(x^2) + eps) * (1 + w)

The mixer is differential attention: two softmax maps per head over the same values, subtracted with a learned factor,

    o_h = R(softmax(q1 k1) v - lambda softmax(q2 k2) v) * (1 - diff) * sigmoid(gate_h),   R without a weight,

over grouped queries; q, k and v have biases and pass a short causal convolution per channel before q and k are turned
(interleaved pairs, YaRN-scaled frequencies); a layer may read the keys and values an earlier layer made.  The
feed-forward is a clamped gated unit with biases.

`w` maps the checkpoint's tensor names to torch tensors, `cfg` is the parsed config.json; everything is computed in
`dtype`.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centered_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * (1.0 + weight)


def short_conv(u: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """u [T, C], weight [C, taps]: y[t] = sum_j weight[:, j] * u[t - taps + 1 + j], zeros before the first row"""
    T, taps = u.shape[0], weight.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += u[:T - back] * weight[:, j]
    return y


def frequencies(rot: dict):
    """angles per position of the rotated pairs, and the factor by which sine and cosine grow"""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor = float(sc["factor"])

    def at(turns):
        return dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(at(float(sc["fast"]))), 0)
    hi = min(math.ceil(at(float(sc["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def turn_pairs(x: torch.Tensor, freq: torch.Tensor, mag: float = 1.0) -> torch.Tensor:
    """x [T, ..., dim]: entry 2i turns with entry 2i + 1; entries from 2 len(freq) on pass"""
    n = freq.numel()
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * freq[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (n,)
    c, s = (torch.cos(a) * mag).to(x.dtype).view(shape), (torch.sin(a) * mag).to(x.dtype).view(shape)
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out = x.clone()
    out[..., 0:2 * n:2] = u * c - v * s
    out[..., 1:2 * n:2] = v * c + u * s
    return out


def project(h, w, name):
    """projection with bias, then the causal convolution of every channel"""
    y = h @ w[name].T + w[name + ".b"]
    return short_conv(y, w[name + ".conv"]) if name + ".conv" in w else y


def keys_and_values(h, w, pre, mx):
    """keys [T, G, 2, dim] (convolved and turned) and values [T, G, vdim] (convolved) of a layer with its own"""
    G, D, V = int(mx.get("kv_heads", mx["heads"])), int(mx["dim"]), int(mx.get("vdim", mx["dim"]))
    T = h.shape[0]
    k = project(h, w, pre + "k").view(T, G, 2, D)
    if mx.get("rot"):
        k = turn_pairs(k, *frequencies(mx["rot"]))
    return k, project(h, w, pre + "v").view(T, G, V)


def causal_map(q, k, v, scale):
    """q [T, H, D], k [T, G, D], v [T, G, V]: one ordinary softmax attention, head h reading key head h // (H / G)"""
    T, rep = q.shape[0], q.shape[1] // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, 1)) * scale
    ahead = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    return torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(ahead, float("-inf")), -1), v.repeat_interleave(rep, 1))


def map_factor(w, pre, diff: float):
    """lambda: how much of the second map is taken off the first"""
    return torch.exp((w[pre + "lq1"] * w[pre + "lk1"]).sum()) - torch.exp((w[pre + "lq2"] * w[pre + "lk2"]).sum()) + diff


def combine_maps(a1, a2, lam, diff: float, eps: float):
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, w, pre, mx, eps, kv):
    H, D = int(mx["heads"]), int(mx["dim"])
    T, diff, scale = h.shape[0], float(mx["diff"]), float(mx["scale"])
    q = project(h, w, pre + "q").view(T, H, 2, D)
    if mx.get("rot"):
        q = turn_pairs(q, *frequencies(mx["rot"]))
    k, v = kv
    a1, a2 = (causal_map(q[:, :, m], k[:, :, m], v, scale) for m in (0, 1))
    o = combine_maps(a1, a2, map_factor(w, pre, diff), diff, eps)
    o = o * torch.sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[pre + "o"].T


def clamped_unit(g, u, limit: float):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def feed_forward(h, w, pre, ml):
    if ml["kind"] != "dense":
        raise ValueError(f"unknown feed-forward kind {ml['kind']!r}")
    g, u = (h @ w[pre + n].T + w[pre + n + ".b"] for n in ("gate", "up"))
    return clamped_unit(g, u, float(ml["limit"])) @ w[pre + "down"].T + w[pre + "down.b"]


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """logits [T, vocab]; `layers_out` receives the residual stream after every layer"""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    made = {}
    for i, lc in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", lc["mixer"]
        if lc["type"] != "attention":
            raise ValueError(f"layer {i}: unknown layer type {lc['type']!r}")
        h = centered_norm(x, w[p + "norm1"], eps)
        src = mx.get("kv_from")
        if src is None:
            made[i] = keys_and_values(h, w, p + "mix.", mx)
        y = differential_attention(h, w, p + "mix.", mx, eps, made[i if src is None else int(src)])
        if lc.get("mlp"):
            y = y + feed_forward(h, w, p + "mlp.", lc["mlp"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return centered_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg: dict, w: Dict[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
