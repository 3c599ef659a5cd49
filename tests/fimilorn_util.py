"""Shared helpers of the Fimilorn tests: small configurations whose sizes differ from one another (key heads fewer than
heads or as many, values narrower and wider than keys, rotation over part of a head, all of it or none, windows that are
neither a page nor a tile, groups of one expert and of many, shared experts of the experts' size, of another, none;
layers without feed-forward; layers before, inside and behind a loop), random checkpoints, error measures."""
import numpy as np
import torch

from llmq_b200.fimilorn import FimilornLayer, FimilornSpec, random_checkpoint

DENSE = dict(ff="dense", ff_dim=72, ff_limit=0.8)
MOE = dict(ff="moe", ff_dim=40, n_experts=12, top_k=3, n_groups=4, keep_groups=2, shared_ff=40)
MOE_OTHER_SHARED = dict(ff="moe", ff_dim=24, n_experts=6, top_k=2, n_groups=2, keep_groups=1, shared_ff=56)
MOE_ALONE = dict(ff="moe", ff_dim=16, n_experts=5, top_k=4, n_groups=1, keep_groups=1, shared_ff=0)
MOE_GROUPS_OF_ONE = dict(ff="moe", ff_dim=32, n_experts=7, top_k=2, n_groups=7, keep_groups=3, shared_ff=8)
MOE_ALL = dict(ff="moe", ff_dim=16, n_experts=4, top_k=4, n_groups=2, keep_groups=2, shared_ff=16)


def retention(heads=3, dim=20, vdim=28, rot_dims=12, rot_base=300.0, decay=None, **ff):
    decay = decay or tuple(1.0 - 2.0 ** (-1.0 - 2.0 * h) for h in range(heads))
    return FimilornLayer(kind="retention", heads=heads, dim=dim, vdim=vdim, rot_dims=rot_dims,
                         rot_base=rot_base if rot_dims else 10000.0, decay=decay, **ff)


def attn(heads=6, kv_heads=2, dim=24, vdim=40, rot_dims=16, rot_base=500.0, scale=0.4, window=0, **ff):
    return FimilornLayer(kind="attention", heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot_dims=rot_dims,
                         rot_base=rot_base if rot_dims else 10000.0, scale=scale, window=window, **ff)


def latent(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, window=19, rot_base=100.0, scale=0.3, rot_dims=None, **ff):
    return FimilornLayer(kind="latent_attention", heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank,
                         window=window, rot_dims=rot_dim if rot_dims is None else rot_dims, rot_base=rot_base, scale=scale,
                         **ff)


def small_spec(width=96, vocab=211, layers=None, eps=1e-5, loop=(1, 4, 3)):
    """by default: a layer before the loop, three inside it (three passes), two behind it"""
    layers = layers or [
        retention(**DENSE),
        latent(**MOE),
        attn(**MOE_OTHER_SHARED),
        retention(heads=2, dim=12, vdim=8, rot_dims=12, rot_base=50.0, decay=(0.97, 0.35)),     # no feed-forward
        attn(heads=3, kv_heads=3, dim=16, vdim=12, rot_dims=0, **MOE_ALONE),
        latent(heads=2, dim=24, rot_dim=4, vdim=8, kv_rank=24, window=0, **MOE_GROUPS_OF_ONE),
    ]
    return FimilornSpec(width=width, vocab=vocab, base_layers=layers, loop=loop, rms_eps=eps)


def tile_spec(width=128, vocab=256, loop=(0, 4, 2)):
    """sizes that the tensor-core kernels take"""
    return FimilornSpec(width=width, vocab=vocab, rms_eps=1e-6, loop=loop, base_layers=[
        retention(heads=2, dim=64, vdim=64, rot_dims=32, decay=(0.98, 0.75), ff="dense", ff_dim=256, ff_limit=1.1),
        attn(heads=4, kv_heads=2, dim=64, vdim=128, rot_dims=64, scale=0.125, ff="moe", ff_dim=64, n_experts=8, top_k=2,
             n_groups=2, keep_groups=1, shared_ff=64),
        latent(heads=4, dim=64, rot_dim=64, vdim=64, kv_rank=64, window=50, scale=0.09, ff="moe", ff_dim=64, n_experts=8,
               top_k=3, n_groups=4, keep_groups=2, shared_ff=128),
        retention(heads=1, dim=128, vdim=96, rot_dims=128, decay=(0.995,)),
    ])


def checkpoint(spec, seed=0):
    """random bf16-representable weights (so the fp32 engine and the fp64 oracle read the same numbers)"""
    return random_checkpoint(spec, seed=seed, device="cpu")


def calm_routers(spec, sd):
    """the same weights with choices that no rounding turns over: the experts' corrections rise (or fall) by more than a score
    can, so experts and groups rank by their numbers whatever the token"""
    sd = dict(sd)
    for i, ly in enumerate(spec.base_layers):
        if ly.ff == "moe":
            c = 2.0 * torch.arange(ly.n_experts) - 5.0
            sd[f"l{i}.mlp.correction"] = (c if i % 2 else c.flip(0)).to(torch.bfloat16)
    return sd


def rel_err(got, want):
    """rms of the difference over the rms of the expected rows, worst row"""
    got = np.asarray(got, dtype=np.float64)
    want = np.asarray(want, dtype=np.float64)
    num = np.sqrt(((got - want) ** 2).mean(-1))
    den = np.sqrt((want ** 2).mean(-1)) + 1e-30
    return float((num / den).max())


def tokens(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()
