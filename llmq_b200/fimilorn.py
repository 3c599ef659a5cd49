"""Host side of the Fimilorn decoder: reading its config.json, mapping its checkpoint to the engine's
layered-model weights, and drawing random checkpoints for tests and benchmarks.

Fimilorn is a stack of layers over an fp32 residual stream with an RMS norm on BOTH sides of every sublayer,

    x <- x + N1b(mixer(N1 x))      x <- x + N2b(ff(N2 x))      N v = v / sqrt(mean(v^2) + eps) * w

A range of layers may run several times with the same weights; pass t begins with x <- x (+ x0, t > 0) + step_t (x0 =
the embedding output) and has its own caches and states.  Mixers:

  retention         linear attention with a constant decay per head, S <- decay S + k v^T, o = S^T q, over half-split
                    rotated queries and keys; every head's output by its root mean square, times silu(gate)
  attention         grouped-query attention over every earlier key; one RMS norm over the whole query (key)
                    projection, half-split rotation, a learned sink per head in the softmax's denominator, a sigmoid
                    gate per output channel
  latent_attention  full-rank queries; keys and values from a normed latent plus one rotated key part shared by the
                    heads (only those two are cached); half-split rotation, sliding window, a sink per head

Feed-forwards: a dense clamped gated unit, or a top-k mixture of SiLU-gated experts routed by sigmoid scores with a
choice correction and a choice limited to the best groups of experts, beside a shared expert.  The output matrix is the
embedding table.

The engine sees one layer per layer RUN: a repeated layer is listed once per pass, bound to the same device tensors,
with its own cache region and state.  Every size comes from config.json or a tensor's shape.
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import Dict, Iterable, List, Optional, Tuple

import torch

from . import lib as L
from .kabavik import GLU_BLOCK, _interleave, _pad_rows
from .ramopel import checkpoint_shapes, load_checkpoint, save_checkpoint  # noqa: F401  (one file format)

ARCHITECTURE = "Fimilorn"
KINDS = ("retention", "attention", "latent_attention")


@dataclass
class FimilornLayer:
    kind: str                        # one of KINDS
    heads: int = 0
    kv_heads: int = 0                # attention
    dim: int = 0                     # per-head query / key size (latent attention: the unrotated part)
    vdim: int = 0
    rot_dim: int = 0                 # latent attention: the rotated part of a head
    kv_rank: int = 0                 # latent attention: size of the cached latent
    window: int = 0                  # 0 = every earlier key
    rot_dims: int = 0                # rotated dimensions; 0 = no rotation
    rot_base: float = 10000.0
    scale: float = 1.0
    decay: Tuple[float, ...] = ()    # retention: one per head
    # feed-forward
    ff: Optional[str] = None         # None | "dense" | "moe"
    ff_dim: int = 0
    ff_limit: float = 0.0            # dense
    n_experts: int = 0
    top_k: int = 0
    n_groups: int = 1
    keep_groups: int = 1
    shared_ff: int = 0               # size of the shared expert; 0 = none
    # place in the stack
    src: int = 0                     # checkpoint layer whose tensors this run uses
    step: Optional[int] = None       # the pass that begins here (None: no pass does)

    def desc(self) -> L.LayerDesc:
        ff = {None: L.FF_NONE, "dense": L.FF_CLAMPED, "moe": L.FF_MOE_GATED}[self.ff]
        inject = L.INJECT_NONE if self.step is None else (L.INJECT_STEP_EMBED if self.step else L.INJECT_STEP)
        common = dict(heads=self.heads, dim=self.dim, vdim=self.vdim, rot_dims=self.rot_dims, rot_base=self.rot_base,
                      kv_from=-1, ff=ff, ff_dim=self.ff_dim, ff_limit=self.ff_limit, n_experts=self.n_experts,
                      top_k=self.top_k, n_groups=self.n_groups, keep_groups=self.keep_groups, shared_dim=self.shared_ff,
                      inject=inject)
        if self.kind == "retention":
            return L.LayerDesc(mixer=L.MIXER_RETENTION, **common)
        if self.kind == "latent_attention":
            return L.LayerDesc(mixer=L.MIXER_LATENT_ATTN, rot_dim=self.rot_dim, kv_rank=self.kv_rank, window=self.window,
                               attn_scale=self.scale, rot_half=1, sink=1, **common)
        return L.LayerDesc(mixer=L.MIXER_WINDOW_ATTN, kv_heads=self.kv_heads, window=self.window, attn_scale=self.scale,
                           qk_norm=1, bare=1, channel_gate=1, sink=1, **common)


def _rotation(i: int, mx: dict, limit: int) -> dict:
    rot = mx.get("rot") or {}
    dims = int(rot.get("dims") or 0)
    if dims % 2 or dims > limit:
        raise ValueError(f"layer {i}: rot.dims ({dims}) must be even and at most {limit}")
    return dict(rot_dims=dims, rot_base=float(rot.get("base", 10000.0)))


def _layer_from_config(i: int, lc: dict) -> FimilornLayer:
    mx, kind = lc["mixer"], lc["type"]
    if kind not in KINDS:
        raise ValueError(f"layer {i}: unknown layer type {kind!r}")
    heads, dim = int(mx["heads"]), int(mx["dim"])
    ly = FimilornLayer(kind=kind, heads=heads, dim=dim, vdim=int(mx.get("vdim", dim)))
    if kind == "retention":
        ly.decay = tuple(float(v) for v in mx["decay"])
        if len(ly.decay) != heads:
            raise ValueError(f"layer {i}: {len(ly.decay)} decays for {heads} heads")
        rot = _rotation(i, mx, dim)
    else:
        ly.scale, ly.window = float(mx["scale"]), int((mx.get("mask") or {}).get("size") or 0)
        if kind == "attention":
            ly.kv_heads = int(mx.get("kv_heads", heads))
            if heads % ly.kv_heads:
                raise ValueError(f"layer {i}: kv_heads ({ly.kv_heads}) must divide heads ({heads})")
            rot = _rotation(i, mx, dim)
        else:
            ly.rot_dim, ly.kv_rank = int(mx.get("rot_dim") or 0), int(mx["kv_rank"])
            rot = _rotation(i, mx, ly.rot_dim)
    ly.rot_dims, ly.rot_base = rot["rot_dims"], rot["rot_base"]
    ml = lc.get("mlp")
    if not ml:
        return ly
    if ml["kind"] == "dense":
        ly.ff, ly.ff_dim, ly.ff_limit = "dense", int(ml["ff"]), float(ml["limit"])
    elif ml["kind"] == "moe":
        r = ml["router"]
        g = r.get("groups") or {}
        ly.ff, ly.ff_dim = "moe", int(ml["expert"]["ff"])
        ly.n_experts, ly.top_k = int(r["experts"]), int(r["top"])
        ly.n_groups = int(g.get("count") or 1)
        ly.keep_groups = int(g.get("keep") or ly.n_groups)
        ly.shared_ff = int((ml.get("shared") or {}).get("ff") or 0)
        if (ly.n_experts % ly.n_groups or ly.keep_groups > ly.n_groups
                or ly.top_k > ly.keep_groups * (ly.n_experts // ly.n_groups)):
            raise ValueError(f"layer {i}: {ly.n_groups} groups must divide {ly.n_experts} experts, keep at most that many, "
                             f"and the kept groups must hold top = {ly.top_k} experts")
    else:
        raise ValueError(f"layer {i}: unknown feed-forward kind {ml['kind']!r}")
    return ly


def _layer_to_config(ly: FimilornLayer) -> dict:
    mx: dict = {"heads": ly.heads, "dim": ly.dim, "vdim": ly.vdim}
    if ly.rot_dims:
        mx["rot"] = {"dims": ly.rot_dims, "base": ly.rot_base}
    if ly.kind == "retention":
        mx["decay"] = list(ly.decay)
    else:
        mx["scale"] = ly.scale
        if ly.window:
            mx["mask"] = {"size": ly.window}
        if ly.kind == "attention":
            mx["kv_heads"] = ly.kv_heads
        else:
            mx.update(rot_dim=ly.rot_dim, kv_rank=ly.kv_rank)
    ml = None
    if ly.ff == "dense":
        ml = {"kind": "dense", "ff": ly.ff_dim, "limit": ly.ff_limit}
    elif ly.ff == "moe":
        ml = {"kind": "moe", "expert": {"ff": ly.ff_dim},
              "router": {"experts": ly.n_experts, "top": ly.top_k,
                         "groups": {"count": ly.n_groups, "keep": ly.keep_groups}}}
        if ly.shared_ff:
            ml["shared"] = {"ff": ly.shared_ff}
    return {"type": ly.kind, "mixer": mx, "mlp": ml}


@dataclass
class FimilornSpec:
    """What `NativeModel` needs to know about a Fimilorn checkpoint (the counterpart of `ModelSpec`).
    `layers` lists the layer RUNS in the order they execute; `base_layers` the checkpoint's layers."""
    width: int
    vocab: int
    base_layers: List[FimilornLayer]
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times): layers start..stop-1 run `times` times
    rms_eps: float = 1e-6
    name: str = "fimilorn"
    max_position_embeddings: int = 1 << 20   # positions are computed, not tabulated: the pool is the limit
    eos_token_id: Optional[int] = None
    eos_token_ids: Tuple[int, ...] = ()
    bos_token_id: Optional[int] = None
    arch: str = "fimilorn"
    layered: bool = field(default=True, repr=False)
    layers: List[FimilornLayer] = field(default_factory=list, repr=False)

    def __post_init__(self):
        n = len(self.base_layers)
        for i, ly in enumerate(self.base_layers):
            ly.src, ly.step = i, None
        if self.loop is None:
            self.layers = list(self.base_layers)
            return
        start, stop, times = self.loop
        if not (0 <= start < stop <= n and times >= 1):
            raise ValueError(f"loop {self.loop}: need 0 <= start < stop <= {n} layers and times >= 1")
        runs = list(self.base_layers[:start])
        for t in range(times):
            for i in range(start, stop):
                runs.append(replace(self.base_layers[i], step=t if i == start else None))
        self.layers = runs + list(self.base_layers[stop:])

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    def config_extras(self) -> dict:
        """the fields of b200q_model_config that describe this design's layer form"""
        return dict(arch=L.ARCH_FIMILORN, layer_form=L.FORM_SANDWICH, norm_kind=L.NORM_RMS, embed_scale=0.0)

    @staticmethod
    def from_config(cfg: dict, shapes: Optional[Dict[str, Tuple[int, ...]]] = None,
                    name: str = "fimilorn") -> "FimilornSpec":
        if cfg.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} config: architecture={cfg.get('architecture')!r}")
        lp = cfg.get("loop")
        loop = (int(lp["start"]), int(lp["stop"]), int(lp.get("times", 1))) if lp else None
        return FimilornSpec(width=int(cfg["width"]), vocab=int(cfg["vocab"]),
                            base_layers=[_layer_from_config(i, lc) for i, lc in enumerate(cfg["layers"])], loop=loop,
                            rms_eps=float((cfg.get("norm") or {}).get("eps", 1e-6)), name=name)

    def to_config(self) -> dict:
        cfg = {"architecture": ARCHITECTURE, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.rms_eps},
               "layers": [_layer_to_config(ly) for ly in self.base_layers]}
        if self.loop is not None:
            cfg["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return cfg

    def engine_weights(self, sd: Dict[str, torch.Tensor]) -> Iterable[Tuple[str, torch.Tensor]]:
        return engine_weights(self, sd)

    def random_checkpoint(self, seed: int = 0, device="cpu") -> Dict[str, torch.Tensor]:
        return random_checkpoint(self, seed, device)

    def weight_bytes_per_token(self, esize: int = 2, batch: int = 1) -> int:
        """matrix bytes one decode step of `batch` tokens touches (a repeated layer is read once per pass; a routed
        layer reads at most min(experts, batch * top_k) of its experts; embedding rows are read by row, the
        output matrix in full)"""
        W, n = self.width, self.vocab * self.width
        for ly in self.layers:
            hv = ly.heads * ly.vdim
            if ly.kind == "retention":
                n += W * (2 * ly.heads * ly.dim + 2 * hv) + W * hv
            elif ly.kind == "attention":
                n += W * (ly.heads * ly.dim + ly.kv_heads * (ly.dim + ly.vdim) + hv) + W * hv
            else:
                n += W * (ly.heads * (ly.dim + ly.rot_dim) + ly.kv_rank + ly.rot_dim)
                n += ly.heads * ly.kv_rank * (ly.dim + ly.vdim) + W * hv
            if ly.ff == "dense":
                n += 3 * W * ly.ff_dim
            elif ly.ff == "moe":
                n += W * ly.n_experts + 3 * W * ly.ff_dim * min(ly.n_experts, batch * ly.top_k) + 3 * W * ly.shared_ff
        return n * esize


# ---- checkpoint names -> engine names --------------------------------------------------------------
def engine_weights(spec: FimilornSpec, sd: Dict[str, torch.Tensor]) -> Iterable[Tuple[str, torch.Tensor]]:
    """Checkpoint tensors -> the layered engine's weights, one set of names per layer RUN.  2-D results are matrices
    (bound in the model's dtype); 1-D results are vectors and constants (bound as fp32 rows).  Runs of the same
    checkpoint layer yield the SAME tensor objects, which the model uploads once.  Fusions: the projections that read a
    mixer's input become one matrix with zero rows up to a multiple of 64 (retention and attention: q, k, v, gate;
    latent attention: q, the latent, the shared rotated key; the router alone); each head's key up-projection is stored transposed too (single
    tokens carry the query into the latent space); gate and up of the dense unit are stacked (interleaved in blocks of 128 rows
    when ff is a multiple of 128); the experts' matrices are stacked, a shared expert of their size as one more."""
    yield "embed", sd["embed"]
    yield "final_norm", sd["final.norm"]
    yield "lm_head", sd["embed"]
    made: Dict[int, List[Tuple[str, torch.Tensor]]] = {}
    for run, ly in enumerate(spec.layers):
        if ly.src not in made:
            made[ly.src] = list(_layer_weights(ly, sd))
        o = f"layers.{run}."
        if ly.step is not None:
            yield o + "step", sd["loop.step"][ly.step].clone()
        for name, t in made[ly.src]:
            yield o + name, t


def _layer_weights(ly: FimilornLayer, sd) -> Iterable[Tuple[str, torch.Tensor]]:
    p = f"l{ly.src}."
    m = p + "mix."
    yield "norm1", sd[p + "norm1"]
    yield "norm1b", sd[p + "norm1b"]
    if ly.kind == "latent_attention":
        yield "mix.down", _pad_rows(torch.cat([sd[m + "q"], sd[m + "dkv"]], 0))
        yield "mix.kv_norm", sd[m + "dkv.norm"]
        uk = sd[m + "uk"].reshape(ly.heads, ly.dim, ly.kv_rank)
        yield "mix.uk_t", uk.transpose(1, 2).reshape(ly.heads * ly.kv_rank, ly.dim)
        yield "mix.uk", sd[m + "uk"]     # prompts expand the latents they see instead
        yield "mix.uv", sd[m + "uv"]
        yield "mix.sink", sd[m + "sink"].reshape(-1)
    else:
        yield "mix.proj", _pad_rows(torch.cat([sd[m + n] for n in ("q", "k", "v", "g")], 0))
        if ly.kind == "retention":
            # a decay acts at every token of a sequence: rounded once, from the config's double
            yield "mix.decay", torch.tensor(ly.decay, dtype=torch.float64).to(torch.float32)
        else:
            yield "mix.q_norm", sd[m + "q.norm"]
            yield "mix.k_norm", sd[m + "k.norm"]
            yield "mix.sink", sd[m + "sink"].reshape(-1)
    yield "mix.o", sd[m + "o"]
    if ly.ff is None:
        return
    f = p + "mlp."
    yield "norm2", sd[p + "norm2"]
    yield "norm2b", sd[p + "norm2b"]
    if ly.ff == "dense":
        if ly.ff_dim % GLU_BLOCK == 0:
            yield "mlp.gate_up_il", _interleave(sd[f + "gate"], sd[f + "up"])
        else:
            yield "mlp.gate_up", torch.cat([sd[f + "gate"], sd[f + "up"]], 0)
        yield "mlp.down", sd[f + "down"]
        return
    yield "mlp.router", _pad_rows(sd[f + "router"])
    yield "mlp.router_bias", sd[f + "correction"].reshape(-1)
    stack = [f"{f}e{e}." for e in range(ly.n_experts)]
    if ly.shared_ff and ly.shared_ff == ly.ff_dim:
        stack.append(f + "shared.")
    elif ly.shared_ff:
        yield "mlp.shared_gate_up", torch.cat([sd[f + "shared.gate"], sd[f + "shared.up"]], 0)
        yield "mlp.shared_down", sd[f + "shared.down"]
    yield "mlp.experts_gate_up", torch.cat([sd[e + n] for e in stack for n in ("gate", "up")], 0)
    yield "mlp.experts_down", torch.cat([sd[e + "down"] for e in stack], 0)


def random_checkpoint(spec: FimilornSpec, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """A random checkpoint in the checkpoint's own names.  Matrices are Normal(0, 1/sqrt(fan_in)); norm weights, sinks,
    step vectors and corrections are non-trivial values so that none of them is silently ignored."""
    g = torch.Generator(device=device).manual_seed(seed)
    W = spec.width

    def mat(r, c, s=None):
        s = s if s is not None else c ** -0.5
        return (torch.randn(r, c, generator=g, device=device, dtype=torch.float32) * s).to(dtype)

    def vec(n, mean=0.0, s=0.1):
        return (mean + torch.randn(n, generator=g, device=device, dtype=torch.float32) * s).to(dtype)

    sd: Dict[str, torch.Tensor] = {"embed": mat(spec.vocab, W, 1.0), "final.norm": vec(W, W ** -0.5, 0.1 * W ** -0.5)}
    if spec.loop is not None:
        sd["loop.step"] = mat(spec.loop[2], W, 0.5)
    for i, ly in enumerate(spec.base_layers):
        p = f"l{i}."
        m = p + "mix."
        sd[p + "norm1"], sd[p + "norm1b"] = vec(W, 1.0), vec(W, 0.5)
        hd, hv = ly.heads * ly.dim, ly.heads * ly.vdim
        if ly.kind == "latent_attention":
            sd[m + "q"], sd[m + "dkv"] = mat(ly.heads * (ly.dim + ly.rot_dim), W), mat(ly.kv_rank + ly.rot_dim, W)
            sd[m + "dkv.norm"] = vec(ly.kv_rank, 1.0)
            sd[m + "uk"], sd[m + "uv"] = mat(hd, ly.kv_rank), mat(hv, ly.kv_rank)
            sd[m + "sink"] = vec(ly.heads, 1.0, 1.0)
        else:
            gd, gv = (hd, hv) if ly.kind == "retention" else (ly.kv_heads * ly.dim, ly.kv_heads * ly.vdim)
            sd[m + "q"], sd[m + "k"], sd[m + "v"], sd[m + "g"] = mat(hd, W), mat(gd, W), mat(gv, W), mat(hv, W)
            if ly.kind == "attention":
                sd[m + "q.norm"], sd[m + "k.norm"], sd[m + "sink"] = vec(hd, 1.0), vec(gd, 1.0), vec(ly.heads, 1.0, 1.0)
        sd[m + "o"] = mat(W, hv)
        if ly.ff is None:
            continue
        f = p + "mlp."
        sd[p + "norm2"], sd[p + "norm2b"] = vec(W, 1.0), vec(W, 0.5)
        if ly.ff == "dense":
            sd[f + "gate"], sd[f + "up"], sd[f + "down"] = mat(ly.ff_dim, W), mat(ly.ff_dim, W), mat(W, ly.ff_dim)
            continue
        sd[f + "router"] = mat(ly.n_experts, W, 2.0 * W ** -0.5)
        sd[f + "correction"] = vec(ly.n_experts, 0.0, 0.2)
        for e in range(ly.n_experts):
            q = f"{f}e{e}."
            sd[q + "gate"], sd[q + "up"], sd[q + "down"] = mat(ly.ff_dim, W), mat(ly.ff_dim, W), mat(W, ly.ff_dim)
        if ly.shared_ff:
            q = f + "shared."
            sd[q + "gate"], sd[q + "up"], sd[q + "down"] = mat(ly.shared_ff, W), mat(ly.shared_ff, W), mat(W, ly.shared_ff)
    return sd


def _cycle(width: int, vocab: int, n_layers: int, heads: int, kv_heads: int, experts: int, top: int, ff: int,
           name: str, loop=None) -> FimilornSpec:
    """layers in the order retention, attention, attention, latent_attention, ... with a routed feed-forward in every
    layer but the first, whose feed-forward is dense; head sizes the tensor-core kernels take"""
    rh = width // 128
    layers: List[FimilornLayer] = []
    for i in range(n_layers):
        f = dict(ff="moe", ff_dim=ff, n_experts=experts, top_k=top, n_groups=4, keep_groups=2, shared_ff=ff)
        if i == 0:
            f = dict(ff="dense", ff_dim=3 * width, ff_limit=7.0)
        if i % 4 == 0:
            decay = tuple(1.0 - 2.0 ** (-5.0 - 7.0 * h / max(rh - 1, 1)) for h in range(rh))
            layers.append(FimilornLayer(kind="retention", heads=rh, dim=64, vdim=128, rot_dims=64, rot_base=1000000.0,
                                        decay=decay, **f))
        elif i % 4 == 3:
            layers.append(FimilornLayer(kind="latent_attention", heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=512,
                                        window=4096, rot_dims=64, rot_base=20000.0, scale=192 ** -0.5, **f))
        else:
            layers.append(FimilornLayer(kind="attention", heads=heads, kv_heads=kv_heads, dim=128, vdim=128, rot_dims=128,
                                        rot_base=500000.0, scale=128 ** -0.5, **f))
    return FimilornSpec(width=width, vocab=vocab, base_layers=layers, loop=loop, rms_eps=1e-6, name=name)


# sizes that resemble a real model's layers (random weights; `random:<name>` as a model name)
BUILTIN_SPECS = {
    "fimilorn-1b": _cycle(2048, 32768, 16, 16, 4, 16, 4, 1024, "fimilorn-1b"),
    "fimilorn-3b": _cycle(3072, 32768, 24, 24, 8, 32, 6, 1536, "fimilorn-3b"),
}
