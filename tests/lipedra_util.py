"""Shared helpers of the Lipedra tests: small configurations whose sizes differ from one another (key heads fewer than
heads or as many, value size unlike key size, rotation over part of a map or all of it or none, taps from none to more
than the vectorised kernel takes, borrowed keys and values, layers without feed-forward), random checkpoints, error
measures."""
import numpy as np
import torch

from llmq_b200.lipedra import LipedraLayer, LipedraSpec, random_checkpoint

DENSE = dict(ff="dense", ff_dim=72, ff_limit=1.5)


def attn(heads=6, kv_heads=2, dim=20, vdim=36, scale=0.3, diff=0.35, taps=4, rot_dims=12, rot_base=500.0, factor=3.0,
         original=64.0, fast=8.0, slow=1.0, kv_from=-1, **ff):
    rot = dict(rot_dims=rot_dims, rot_base=rot_base) if rot_dims else {}
    if rot_dims and original:
        rot.update(rot_factor=factor, rot_original=original, rot_fast=fast, rot_slow=slow)
    return LipedraLayer(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff, conv_taps=taps,
                        kv_from=kv_from, **rot, **ff)


def small_spec(width=96, vocab=211, layers=None, eps=1e-5, embed_scale=3.0):
    layers = layers or [
        attn(**DENSE),
        attn(heads=3, kv_heads=3, dim=14, vdim=10, taps=2, rot_dims=14, diff=0.6, original=0.0, ff="dense", ff_dim=128,
             ff_limit=0.7),                                            # plain frequencies, gate and up in blocks of 128
        attn(taps=3, kv_from=0, diff=0.1),                             # layer 0's keys and values, no feed-forward
        attn(heads=5, kv_heads=1, dim=8, vdim=52, taps=0, rot_dims=0, **DENSE),      # no convolution, no rotation
        attn(heads=4, kv_heads=2, dim=12, vdim=12, taps=6, rot_dims=2, scale=0.5, **DENSE),
        attn(taps=1, kv_from=0, scale=0.2, **DENSE),                   # a second reader of layer 0
    ]
    return LipedraSpec(width=width, vocab=vocab, layers=layers, rms_eps=eps, embed_scale=embed_scale)


def tile_spec(width=128, vocab=256):
    """map and value sizes the tensor-core attention kernels take, exactly and padded; more heads on one key head than a
    decode tile has rows; more taps than the vectorised preparation takes; borrowed keys and values"""
    layers = [attn(heads=4, kv_heads=2, dim=64, vdim=128, taps=4, rot_dims=32, scale=0.1, ff="dense", ff_dim=128,
                   ff_limit=2.0),
              attn(heads=10, kv_heads=1, dim=16, vdim=32, taps=2, rot_dims=16, scale=0.25, ff="dense", ff_dim=64,
                   ff_limit=1.0),
              attn(heads=4, kv_heads=2, dim=64, vdim=128, taps=3, rot_dims=32, scale=0.12, kv_from=0),
              attn(heads=3, kv_heads=3, dim=32, vdim=64, taps=5, rot_dims=6, scale=0.2, ff="dense", ff_dim=256,
                   ff_limit=1.0),
              attn(heads=2, kv_heads=1, dim=96, vdim=64, taps=0, rot_dims=0, scale=0.1, ff="dense", ff_dim=64, ff_limit=3.0),
              attn(heads=2, kv_heads=2, dim=128, vdim=128, taps=1, rot_dims=128, scale=0.09)]
    return LipedraSpec(width=width, vocab=vocab, layers=layers, rms_eps=1e-5, embed_scale=2.0)


def checkpoint(spec, seed=0):
    """random bf16-representable weights (so the fp32 engine and the fp64 oracle read the same numbers)"""
    return random_checkpoint(spec, seed=seed, device="cpu")


def rel_err(got, want):
    """rms of the difference over the rms of the expected rows, worst row"""
    got = np.asarray(got, dtype=np.float64)
    want = np.asarray(want, dtype=np.float64)
    num = np.sqrt(((got - want) ** 2).mean(-1))
    den = np.sqrt((want ** 2).mean(-1)) + 1e-30
    return float((num / den).max())


def tokens(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()
