"""Host side of the Lipedra decoder: reading its config.json, mapping its checkpoint to the engine's layered-model
weights, and drawing random checkpoints for tests and benchmarks.

Lipedra is a stack of parallel layers over an fp32 residual stream with ONE norm per layer that both sublayers read,

    h = N x,   x <- x + mixer(h) + ff(h),      N x = x / sqrt(mean(x^2) + eps) * (1 + w)

  attention     differential attention: every head has two query / key maps over the same values; the second map's
                output, times lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff, is taken off the first's, the rest is
                divided by its root mean square and multiplied by 1 - diff and by the sigmoid of a gate number of the
                head.  q, k and v have biases and pass a short causal convolution per channel; neighbouring dimensions
                (2i, 2i + 1) of every map turn with YaRN-scaled frequencies; grouped key heads; a layer may read the
                keys and values an earlier layer cached
  feed-forward  down(g sigmoid(1.702 g) (u + 1)), g = min(gate h, limit), u = clamp(up h, -limit, limit), with biases

Logits = head N x.  Every size comes from config.json or a tensor's shape.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, Iterable, List, Optional, Tuple

import torch

from . import lib as L
from .kabavik import GLU_BLOCK, _interleave
from .ramopel import checkpoint_shapes, load_checkpoint, save_checkpoint  # noqa: F401  (one file format)

ARCHITECTURE = "Lipedra"
MAX_TAPS = 16


@dataclass
class LipedraLayer:
    heads: int
    kv_heads: int
    dim: int                         # query / key size of one map
    vdim: int
    scale: float
    diff: float = 0.0                # lambda's constant part; heads' outputs are multiplied by 1 - diff
    conv_taps: int = 0               # taps of the convolution on q, k and v; 0 = none
    rot_dims: int = 0                # rotated dimensions of every map; 0 = no rotation
    rot_base: float = 10000.0
    rot_factor: float = 0.0          # 0 = unscaled frequencies
    rot_original: float = 0.0        # > 0: YaRN (with rot_fast, rot_slow)
    rot_fast: float = 0.0
    rot_slow: float = 0.0
    kv_from: int = -1                # layer whose cached keys and values are read, -1 = own
    ff: Optional[str] = None         # None | "dense"
    ff_dim: int = 0
    ff_limit: float = 0.0
    kind: str = "attention"

    @property
    def channels(self) -> int:
        """columns of q | k | v (q alone when the keys and values are an earlier layer's)"""
        own = self.kv_heads * (2 * self.dim + self.vdim) if self.kv_from < 0 else 0
        return self.heads * 2 * self.dim + own

    @property
    def proj_rows(self) -> int:
        """rows of the attention's part of the fused input projection: channels, a gate number per head, zero rows"""
        n = self.channels + self.heads
        return n + -n % (256 if n >= 1024 else 64)

    def desc(self) -> L.LayerDesc:
        return L.LayerDesc(mixer=L.MIXER_DIFF_ATTN, heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim,
                           kv_from=self.kv_from, conv_taps=self.conv_taps, attn_scale=self.scale, diff=self.diff,
                           proj_bias=1, head_gate=1, rot_dims=self.rot_dims, rot_base=self.rot_base,
                           rot_factor=self.rot_factor, rot_original=self.rot_original, rot_fast=self.rot_fast,
                           rot_slow=self.rot_slow, ff=L.FF_CLAMPED if self.ff else L.FF_NONE, ff_dim=self.ff_dim,
                           ff_limit=self.ff_limit)

    def rotation(self) -> tuple:
        return (self.rot_dims, self.rot_base, self.rot_factor, self.rot_original, self.rot_fast, self.rot_slow)


def _layer_from_config(i: int, lc: dict, layers: List[LipedraLayer]) -> LipedraLayer:
    if lc["type"] != "attention":
        raise ValueError(f"layer {i}: unknown layer type {lc['type']!r}")
    mx = lc["mixer"]
    ly = LipedraLayer(heads=int(mx["heads"]), kv_heads=int(mx.get("kv_heads", mx["heads"])), dim=int(mx["dim"]),
                      vdim=int(mx.get("vdim", mx["dim"])), scale=float(mx["scale"]), diff=float(mx["diff"]),
                      conv_taps=int(mx.get("conv") or 0))
    if ly.heads % ly.kv_heads:
        raise ValueError(f"layer {i}: kv_heads ({ly.kv_heads}) must divide heads ({ly.heads})")
    if not 0 <= ly.conv_taps <= MAX_TAPS:
        raise ValueError(f"layer {i}: a convolution of {ly.conv_taps} taps (at most {MAX_TAPS})")
    rot = mx.get("rot") or {}
    ly.rot_dims, ly.rot_base = int(rot.get("dims") or 0), float(rot.get("base", 10000.0))
    if ly.rot_dims % 2 or ly.rot_dims > ly.dim:
        raise ValueError(f"layer {i}: rot.dims ({ly.rot_dims}) must be even and at most dim ({ly.dim})")
    sc = rot.get("scaling")
    if sc:
        ly.rot_factor, ly.rot_original = float(sc["factor"]), float(sc["original"])
        ly.rot_fast, ly.rot_slow = float(sc["fast"]), float(sc["slow"])
    src = mx.get("kv_from")
    if src is not None:
        src = int(src)
        o = layers[src] if 0 <= src < i else None
        if o is None or o.kv_from >= 0 or (o.heads, o.kv_heads, o.dim, o.vdim, o.rotation()) != (
                ly.heads, ly.kv_heads, ly.dim, ly.vdim, ly.rotation()):
            raise ValueError(f"layer {i}: kv_from={src} must name an earlier layer with keys and values of its own, the "
                             "same head counts and sizes and the same rotation")
        ly.kv_from = src
    ml = lc.get("mlp")
    if ml:
        if ml["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {ml['kind']!r}")
        ly.ff, ly.ff_dim, ly.ff_limit = "dense", int(ml["ff"]), float(ml["limit"])
    return ly


def _layer_to_config(ly: LipedraLayer) -> dict:
    mx: dict = {"heads": ly.heads, "kv_heads": ly.kv_heads, "dim": ly.dim, "vdim": ly.vdim, "scale": ly.scale,
                "diff": ly.diff}
    if ly.conv_taps:
        mx["conv"] = ly.conv_taps
    if ly.rot_dims:
        mx["rot"] = {"dims": ly.rot_dims, "base": ly.rot_base}
        if ly.rot_original:
            mx["rot"]["scaling"] = {"factor": ly.rot_factor, "original": ly.rot_original, "fast": ly.rot_fast,
                                    "slow": ly.rot_slow}
    if ly.kv_from >= 0:
        mx["kv_from"] = ly.kv_from
    ml = {"kind": "dense", "ff": ly.ff_dim, "limit": ly.ff_limit} if ly.ff else None
    return {"type": ly.kind, "mixer": mx, "mlp": ml}


@dataclass
class LipedraSpec:
    """What `NativeModel` needs to know about a Lipedra checkpoint (the counterpart of `ModelSpec`)."""
    width: int
    vocab: int
    layers: List[LipedraLayer]
    rms_eps: float = 1e-6
    embed_scale: float = 1.0
    name: str = "lipedra"
    max_position_embeddings: int = 1 << 20   # positions are computed, not tabulated: the pool is the limit
    eos_token_id: Optional[int] = None
    eos_token_ids: Tuple[int, ...] = ()
    bos_token_id: Optional[int] = None
    arch: str = "lipedra"
    layered: bool = field(default=True, repr=False)

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    def config_extras(self) -> dict:
        """the fields of b200q_model_config that describe this design's layer form"""
        return dict(arch=L.ARCH_LIPEDRA, layer_form=L.FORM_PARALLEL, shared_norm=1, embed_scale=self.embed_scale)

    @staticmethod
    def from_config(cfg: dict, shapes: Optional[Dict[str, Tuple[int, ...]]] = None,
                    name: str = "lipedra") -> "LipedraSpec":
        if cfg.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} config: architecture={cfg.get('architecture')!r}")
        layers: List[LipedraLayer] = []
        for i, lc in enumerate(cfg["layers"]):
            layers.append(_layer_from_config(i, lc, layers))
        return LipedraSpec(width=int(cfg["width"]), vocab=int(cfg["vocab"]), layers=layers,
                           rms_eps=float(cfg["norm"]["eps"]),
                           embed_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)), name=name)

    def to_config(self) -> dict:
        return {"architecture": ARCHITECTURE, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.rms_eps},
                "embedding": {"scale": self.embed_scale}, "layers": [_layer_to_config(ly) for ly in self.layers]}

    def engine_weights(self, sd: Dict[str, torch.Tensor]) -> Iterable[Tuple[str, torch.Tensor]]:
        return engine_weights(self, sd)

    def random_checkpoint(self, seed: int = 0, device="cpu") -> Dict[str, torch.Tensor]:
        return random_checkpoint(self, seed, device)

    def weight_bytes_per_token(self, esize: int = 2, batch: int = 1) -> int:
        """matrix bytes one decode step touches (embedding rows are read by row, the output matrix in full)"""
        W, n = self.width, self.vocab * self.width
        for ly in self.layers:
            n += W * (ly.channels + ly.heads + ly.heads * ly.vdim)
            if ly.ff:
                n += 3 * W * ly.ff_dim
        return n * esize


# ---- checkpoint names -> engine names --------------------------------------------------------------
def map_lambda(sd: Dict[str, torch.Tensor], m: str, diff: float) -> torch.Tensor:
    """the factor of the second map, one number per layer (fp64 on the host, bound as fp32)"""
    def dot(a, b):
        return (sd[m + a].double() * sd[m + b].double()).sum()
    return (torch.exp(dot("lq1", "lk1")) - torch.exp(dot("lq2", "lk2")) + diff).reshape(1)


def engine_weights(spec: LipedraSpec, sd: Dict[str, torch.Tensor]) -> Iterable[Tuple[str, torch.Tensor]]:
    """Checkpoint tensors -> the layered engine's weights.  2-D results are matrices (bound in the model's dtype); 1-D
    results are vectors and constants (bound as fp32 rows).  Fusions: everything that reads a layer's normed row is one
    matrix `in` = q | k | v (q alone when the keys and values are an earlier layer's) | gate numbers | zero rows, then
    gate | up of the feed-forward (interleaved in blocks of 128 rows when ff is a multiple of 128); what joins the
    residual is one matrix `out` = [output projection | down projection] over [heads | unit]; the taps of q, k and v are
    one table [taps][channels]."""
    yield "embed", sd["embed"]
    yield "final_norm", sd["final.norm"]
    yield "lm_head", sd["head"]
    for i, ly in enumerate(spec.layers):
        p, o = f"l{i}.", f"layers.{i}."
        m, f = p + "mix.", p + "mlp."
        parts = ("q", "k", "v") if ly.kv_from < 0 else ("q",)
        rows = [sd[m + n] for n in parts] + [sd[m + "g"]]
        bias = [sd[m + n + ".b"].float() for n in parts]
        pad = ly.proj_rows - ly.channels - ly.heads
        rows.append(rows[0].new_zeros(pad, spec.width))
        bias.append(bias[0].new_zeros(ly.heads + pad))
        il = bool(ly.ff) and ly.ff_dim % GLU_BLOCK == 0
        if il:
            rows.append(_interleave(sd[f + "gate"], sd[f + "up"]))
            bias.append(_interleave(sd[f + "gate.b"].float()[:, None], sd[f + "up.b"].float()[:, None]).reshape(-1))
        elif ly.ff:
            rows += [sd[f + "gate"], sd[f + "up"]]
            bias += [sd[f + "gate.b"].float(), sd[f + "up.b"].float()]
        yield o + "norm1", sd[p + "norm1"]
        yield o + ("in_il" if il else "in"), torch.cat(rows, 0)
        yield o + "in_b", torch.cat(bias, 0)
        if ly.conv_taps:
            yield o + "mix.conv", torch.cat([sd[m + n + ".conv"].float() for n in parts], 0).t().contiguous().reshape(-1)
        yield o + "mix.lambda", map_lambda(sd, m, ly.diff)
        if ly.ff:
            yield o + "out", torch.cat([sd[m + "o"], sd[f + "down"]], 1)
            yield o + "out_b", sd[f + "down.b"]
        else:
            yield o + "out", sd[m + "o"]


def random_checkpoint(spec: LipedraSpec, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """A random checkpoint in the checkpoint's own names.  Matrices are Normal(0, 1/sqrt(fan_in)); norm weights, biases,
    taps and the vectors of lambda are non-trivial values so that none of them is silently ignored."""
    g = torch.Generator(device=device).manual_seed(seed)
    W = spec.width

    def mat(r, c, s=None):
        s = s if s is not None else c ** -0.5
        return (torch.randn(r, c, generator=g, device=device, dtype=torch.float32) * s).to(dtype)

    def vec(n, mean=0.0, s=0.1):
        return (mean + torch.randn(n, generator=g, device=device, dtype=torch.float32) * s).to(dtype)

    def taps(channels, n):      # the newest value weighs most
        t = torch.randn(channels, n, generator=g, device=device, dtype=torch.float32) * 0.3
        t[:, -1] += 1.0
        return t.to(dtype)

    sd: Dict[str, torch.Tensor] = {"embed": mat(spec.vocab, W, 1.0 / max(spec.embed_scale, 1e-6))}
    for i, ly in enumerate(spec.layers):
        p = f"l{i}."
        m, f = p + "mix.", p + "mlp."
        sd[p + "norm1"] = vec(W)
        sizes = {"q": ly.heads * 2 * ly.dim}
        if ly.kv_from < 0:
            sizes.update(k=ly.kv_heads * 2 * ly.dim, v=ly.kv_heads * ly.vdim)
        for n, rows in sizes.items():
            sd[m + n], sd[m + n + ".b"] = mat(rows, W), vec(rows)
            if ly.conv_taps:
                sd[m + n + ".conv"] = taps(rows, ly.conv_taps)
        for n in ("lq1", "lk1", "lq2", "lk2"):
            sd[m + n] = vec(ly.dim, s=0.5 * ly.dim ** -0.25)
        sd[m + "g"], sd[m + "o"] = mat(ly.heads, W), mat(W, ly.heads * ly.vdim)
        if ly.ff:
            sd[f + "gate"], sd[f + "up"], sd[f + "down"] = mat(ly.ff_dim, W), mat(ly.ff_dim, W), mat(W, ly.ff_dim)
            sd[f + "gate.b"], sd[f + "up.b"], sd[f + "down.b"] = vec(ly.ff_dim), vec(ly.ff_dim), vec(W)
    sd["final.norm"], sd["head"] = vec(W), mat(spec.vocab, W)
    return sd


def _cycle(width: int, vocab: int, n_layers: int, heads: int, kv_heads: int, ff: int, name: str) -> LipedraSpec:
    """every fourth layer reads the keys and values of the one before it; map and value sizes the tensor-core kernels take"""
    layers = [LipedraLayer(heads=heads, kv_heads=kv_heads, dim=64, vdim=128, scale=64 ** -0.5, diff=0.2 + 0.02 * i,
                           conv_taps=4, rot_dims=32, rot_base=100000.0, rot_factor=8.0, rot_original=4096.0,
                           rot_fast=32.0, rot_slow=1.0, kv_from=i - 1 if i % 4 == 3 else -1, ff="dense", ff_dim=ff,
                           ff_limit=7.0) for i in range(n_layers)]
    return LipedraSpec(width=width, vocab=vocab, layers=layers, rms_eps=1e-6, embed_scale=float(width) ** 0.5, name=name)


# sizes that resemble a real model's layers (random weights; `random:<name>` as a model name)
BUILTIN_SPECS = {
    "lipedra-1b": _cycle(2048, 32768, 16, 16, 4, 6144, "lipedra-1b"),
    "lipedra-3b": _cycle(3072, 32768, 24, 24, 8, 8192, "lipedra-3b"),
}
