"""CPU tests of the Lipedra host code: the config reader, the registry, the mapping of checkpoint tensors to engine
weights, the rotation frequencies the engine uploads, and the oracle's own consistency (causality, convolution,
borrowed keys and values, combination of the maps, clamps)."""
import ctypes as C
import json
import math

import pytest
import torch

from llmq_b200 import lib as L
from llmq_b200 import lipedra as P
from oracle import lipedra as O
from tests.lipedra_util import DENSE, attn, checkpoint, small_spec, tile_spec, tokens


def _with(cfg, path, value):
    bad = json.loads(json.dumps(cfg))
    at = bad
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    return bad


def test_config_round_trip_and_descriptions():
    spec = small_spec()
    cfg = json.loads(json.dumps(spec.to_config()))
    back = P.LipedraSpec.from_config(cfg)
    assert back.layers == spec.layers
    assert (back.width, back.vocab, back.rms_eps, back.embed_scale) == (96, 211, 1e-5, 3.0)
    assert back.layers[2].ff is None and back.layers[2].kv_from == 0 and back.layers[1].rot_original == 0.0
    with pytest.raises(ValueError):
        P.LipedraSpec.from_config({**cfg, "architecture": "Other"})
    for path, value in ((("layers", 0, "type"), "unknown"), (("layers", 0, "mixer", "kv_heads"), 4),
                        (("layers", 0, "mixer", "rot", "dims"), 11), (("layers", 0, "mixer", "rot", "dims"), 22),
                        (("layers", 0, "mixer", "conv"), 17), (("layers", 2, "mixer", "kv_from"), 2),
                        (("layers", 2, "mixer", "kv_from"), 1), (("layers", 5, "mixer", "kv_from"), 2),
                        (("layers", 2, "mixer", "dim"), 24), (("layers", 2, "mixer", "heads"), 4),
                        (("layers", 2, "mixer", "rot", "base"), 7.0), (("layers", 0, "mlp", "kind"), "other")):
        with pytest.raises(ValueError):
            P.LipedraSpec.from_config(_with(cfg, path, value))
    # what a config leaves out is off
    bare = json.loads(json.dumps(cfg))
    del bare["layers"][0]["mixer"]["rot"]["scaling"], bare["layers"][3]["mixer"]["kv_heads"], bare["embedding"]
    bare["layers"] = [bare["layers"][0], bare["layers"][3]]
    sp = P.LipedraSpec.from_config(bare)
    assert (sp.layers[0].rot_factor, sp.layers[0].rot_original, sp.layers[0].rot_dims) == (0.0, 0.0, 12)
    assert (sp.layers[1].kv_heads, sp.layers[1].rot_dims, sp.layers[1].conv_taps, sp.embed_scale) == (5, 0, 0, 1.0)
    ex = spec.config_extras()
    assert (ex["arch"], ex["layer_form"], ex["shared_norm"], ex["embed_scale"]) == (L.ARCH_LIPEDRA, L.FORM_PARALLEL, 1, 3.0)
    d0, d2 = spec.layers[0].desc(), spec.layers[2].desc()
    assert (d0.mixer, d0.heads, d0.kv_heads, d0.dim, d0.vdim, d0.conv_taps, d0.rot_dims, d0.kv_from, d0.ff, d0.ff_dim) == \
        (L.MIXER_DIFF_ATTN, 6, 2, 20, 36, 4, 12, -1, L.FF_CLAMPED, 72)
    assert (d0.rot_base, d0.rot_factor, d0.rot_original, d0.rot_fast, d0.rot_slow) == (500.0, 3.0, 64.0, 8.0, 1.0)
    assert abs(d0.diff - 0.35) < 1e-6 and abs(d0.ff_limit - 1.5) < 1e-6 and abs(d0.attn_scale - 0.3) < 1e-6
    assert (d2.kv_from, d2.conv_taps, d2.ff) == (0, 3, L.FF_NONE)


def test_structs_match_the_header(tmp_path):
    import os
    import subprocess
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    src = tmp_path / "t.c"
    src.write_text('#include "b200q.h"\n#include <stdio.h>\n#include <stddef.h>\n'
                   'int main(void){printf("%zu %zu %zu %zu %zu\\n", sizeof(b200q_layer_desc), offsetof(b200q_layer_desc, '
                   'diff), offsetof(b200q_layer_desc, ff_limit), sizeof(b200q_model_config), '
                   'offsetof(b200q_model_config, shared_norm));return 0;}\n')
    exe = tmp_path / "t"
    subprocess.run(["gcc", "-std=c99", "-I", os.path.join(root, "include"), str(src), "-o", str(exe)], check=True)
    got = [int(x) for x in subprocess.run([str(exe)], capture_output=True, text=True, check=True).stdout.split()]
    assert got == [C.sizeof(L.LayerDesc), L.LayerDesc.diff.offset, L.LayerDesc.ff_limit.offset, C.sizeof(L.ModelConfig),
                   L.ModelConfig.shared_norm.offset]


def test_resolve_model_picks_the_class_by_config(tmp_path):
    from llmq_b200.model import BUILTIN_SPECS, resolve_model
    spec = small_spec()
    sd = checkpoint(spec, 2)
    (tmp_path / "config.json").write_text(json.dumps(spec.to_config()))
    P.save_checkpoint(str(tmp_path / "model.safetensors"), sd)
    got, d = resolve_model(str(tmp_path))
    assert isinstance(got, P.LipedraSpec) and got.layers == spec.layers and d == str(tmp_path)
    assert BUILTIN_SPECS["lipedra-1b"].layered and resolve_model("random:lipedra-1b")[1] is None
    loaded = P.load_checkpoint(str(tmp_path / "model.safetensors"))
    assert set(loaded) == set(sd) and all(torch.equal(loaded[k], sd[k]) for k in sd)


def test_engine_weights_shapes_and_fusions():
    spec = small_spec()
    sd = checkpoint(spec, 3)
    ew = dict(spec.engine_weights(sd))
    W = spec.width
    l0 = spec.layers[0]
    nq, nk, nv = 6 * 2 * 20, 2 * 2 * 20, 2 * 36
    assert l0.channels == nq + nk + nv and l0.proj_rows % 64 == 0 and l0.proj_rows >= l0.channels + 6
    w, b = ew["layers.0.in"], ew["layers.0.in_b"]
    NP = l0.proj_rows
    assert w.shape == (NP + 144, W) and b.shape == (NP + 144,) and b.dtype == torch.float32
    assert torch.equal(w[:nq], sd["l0.mix.q"]) and torch.equal(w[nq:nq + nk], sd["l0.mix.k"])
    assert torch.equal(w[l0.channels:l0.channels + 6], sd["l0.mix.g"])
    assert float(w[l0.channels + 6:NP].abs().max()) == 0.0 and float(b[l0.channels:NP].abs().max()) == 0.0
    assert torch.equal(w[NP + 72:], sd["l0.mlp.up"]) and torch.equal(b[NP:NP + 72], sd["l0.mlp.gate.b"].float())
    assert torch.equal(b[nq + nk:nq + nk + nv], sd["l0.mix.v.b"].float())
    conv = ew["layers.0.mix.conv"].view(4, l0.channels)
    assert torch.equal(conv[1, nq:nq + nk], sd["l0.mix.k.conv"][:, 1].float())
    out = ew["layers.0.out"]
    assert out.shape == (W, 6 * 36 + 72) and torch.equal(out[:, :216], sd["l0.mix.o"]) and \
        torch.equal(out[:, 216:], sd["l0.mlp.down"])
    lam = float(ew["layers.0.mix.lambda"])
    want = math.exp(float((sd["l0.mix.lq1"].double() * sd["l0.mix.lk1"].double()).sum())) - \
        math.exp(float((sd["l0.mix.lq2"].double() * sd["l0.mix.lk2"].double()).sum())) + 0.35
    assert abs(lam - want) < 1e-9
    # a borrowing layer projects queries only; without a feed-forward there is no unit and no output bias
    l2 = spec.layers[2]
    assert ew["layers.2.in"].shape == (l2.proj_rows, W) and l2.channels == nq and "layers.2.out_b" not in ew
    assert ew["layers.2.mix.conv"].shape == (3 * nq,) and ew["layers.2.out"] is sd["l2.mix.o"]
    assert "layers.3.mix.conv" not in ew
    # gate and up rows (and their biases) alternate in blocks of 128 when ff is a multiple of 128
    il, NP1 = ew["layers.1.in_il"], spec.layers[1].proj_rows
    assert "layers.1.in" not in ew and torch.equal(il[NP1:NP1 + 128], sd["l1.mlp.gate"]) and \
        torch.equal(il[NP1 + 128:], sd["l1.mlp.up"])
    sp2 = tile_spec()
    sd2 = checkpoint(sp2, 4)
    ew2, n3 = dict(sp2.engine_weights(sd2)), sp2.layers[3].proj_rows
    il, ib = ew2["layers.3.in_il"][n3:], ew2["layers.3.in_b"][n3:]
    for j, (name, lo) in enumerate((("gate", 0), ("up", 0), ("gate", 128), ("up", 128))):
        assert torch.equal(il[128 * j:128 * (j + 1)], sd2[f"l3.mlp.{name}"][lo:lo + 128])
        assert torch.equal(ib[128 * j:128 * (j + 1)], sd2[f"l3.mlp.{name}.b"][lo:lo + 128].float())
    big = attn(heads=16, kv_heads=4, dim=64, vdim=128)
    assert big.channels == 3072 and big.proj_rows == 3328                # whole 256-row tiles from 1024 rows up
    assert spec.weight_bytes_per_token() > 0


def test_rotation_frequencies_match_the_plain_form():
    lib = L.load()
    for rot in (dict(dims=12, base=700.0), dict(dims=8, base=90.0, scaling=dict(factor=3.0, original=64, fast=8.0, slow=1.0)),
                dict(dims=30, base=30000.0, scaling=dict(factor=6.0, original=8192, fast=24.0, slow=2.0)),
                dict(dims=4, base=50.0, scaling=dict(factor=1.0, original=16, fast=1.0, slow=1.0))):
        sc = rot.get("scaling") or {}
        want, mag = O.frequencies(rot)
        n = rot["dims"] // 2
        out, m = (C.c_double * n)(), C.c_float()
        L.check(lib.b200q_rot_frequencies(rot["dims"], rot["base"], sc.get("factor", 0.0), sc.get("original", 0.0),
                                          sc.get("fast", 0.0), sc.get("slow", 0.0), C.addressof(out), C.addressof(m)))
        assert max(abs(out[i] - float(want[i])) / float(want[i]) for i in range(n)) < 1e-14
        assert abs(m.value - mag) < 1e-7


def _changed(spec, sd, n, at):
    a = tokens(n, spec.vocab, 1)
    b = list(a)
    b[at] = (b[at] + 1) % spec.vocab
    la, lb = O.forward(spec.to_config(), sd, a), O.forward(spec.to_config(), sd, b)
    return [i for i in range(n) if float((la[i] - lb[i]).abs().max()) > 1e-9]


def test_oracle_is_causal_and_sees_every_earlier_key():
    spec = small_spec(width=64, vocab=50)
    assert _changed(spec, checkpoint(spec, 4), 30, 9) == list(range(9, 30))


def test_oracle_convolution_reaches_taps_back_and_no_further():
    w = torch.tensor([[0.5, -2.0, 3.0]], dtype=torch.float64)
    u = torch.zeros(6, 1, dtype=torch.float64)
    u[1] = 1.0
    assert O.short_conv(u, w)[:, 0].tolist() == [0.0, 3.0, -2.0, 0.5, 0.0, 0.0]   # the last tap is the current value
    u = torch.ones(4, 1, dtype=torch.float64)
    assert O.short_conv(u, w)[:, 0].tolist() == [3.0, 1.0, 1.5, 1.5]              # zeros before the start
    assert O.short_conv(u[:1], w)[:, 0].tolist() == [3.0]


def test_oracle_borrowed_keys_and_values_are_the_lenders():
    """keys and values of layer 0 are made from the embedding alone: what the reader sees of another token is that token's
    embedding, whatever layer 0 added to it"""
    spec = small_spec(width=64, vocab=50, layers=[attn(**DENSE), attn(kv_from=0)])
    sd = checkpoint(spec, 5)
    cfg, toks = spec.to_config(), tokens(12, 50, 3)
    h0 = O.centered_norm(sd["embed"].double()[toks] * spec.embed_scale, sd["l0.norm1"].double(), spec.rms_eps)
    kv = O.keys_and_values(h0, {k: v.double() for k, v in sd.items()}, "l0.mix.", cfg["layers"][0]["mixer"])
    out = []
    O.forward(cfg, sd, toks, torch.float64, out)
    h1 = O.centered_norm(out[0], sd["l1.norm1"].double(), spec.rms_eps)
    y = O.differential_attention(h1, {k: v.double() for k, v in sd.items()}, "l1.mix.", cfg["layers"][1]["mixer"],
                                 spec.rms_eps, kv)
    assert torch.allclose(out[1], out[0] + y)
    assert "l1.mix.k" not in sd and "l1.mix.v.conv" not in sd and "l1.mix.q.conv" in sd


def test_oracle_maps_combine_and_units_clamp():
    a1, a2 = torch.tensor([[3.0, 4.0]]), torch.tensor([[1.0, 0.0]])
    got = O.combine_maps(a1, a2, 0.5, 0.2, 0.0)
    v = torch.tensor([[2.5, 4.0]])
    assert torch.allclose(got, v / torch.sqrt((v * v).mean()) * 0.8)
    g, u = torch.tensor([5.0, -5.0, 0.5]), torch.tensor([9.0, -9.0, 0.25])
    got = O.clamped_unit(g, u, 2.0)
    sig = lambda z: 1.0 / (1.0 + math.exp(-1.702 * z))
    for i, (gg, uu) in enumerate(((2.0, 2.0), (-5.0, -2.0), (0.5, 0.25))):        # the gate has no lower clamp
        assert abs(float(got[i]) - gg * sig(gg) * (uu + 1.0)) < 1e-6
    # two maps with equal queries and keys and lambda 1 cancel
    q = torch.randn(5, 2, 3, dtype=torch.float64)
    a = O.causal_map(q, q[:, :1], torch.randn(5, 1, 4, dtype=torch.float64), 0.7)
    assert float(O.combine_maps(a, a, 1.0, 0.3, 1e-5).abs().max()) == 0.0


def test_oracle_turns_neighbouring_pairs_by_position():
    f, mag = O.frequencies(dict(dims=4, base=100.0))
    assert mag == 1.0
    e = torch.zeros(3, 1, 2, 6, dtype=torch.float64)
    e[:, 0, :, 0] = 1.0
    r = O.turn_pairs(e, f)
    assert abs(float(r[2, 0, 0, 1]) - math.sin(2.0)) < 1e-12 and float(r[2, 0, 1, 2:].abs().max()) == 0.0
    x = torch.randn(9, 1, 2, 6, dtype=torch.float64, generator=torch.Generator().manual_seed(0))
    x[:] = x[0]
    r = O.turn_pairs(x, f, 1.5)
    assert torch.allclose(r[..., 4:], x[..., 4:]) and torch.allclose(r[0, ..., :4], 1.5 * x[0, ..., :4])
    dots = torch.einsum("ihmd,jhmd->mij", r, r)
    for d in range(1, 4):
        diag = torch.diagonal(dots, offset=d, dim1=1, dim2=2)
        assert float((diag - diag[:, :1]).abs().max()) < 1e-9               # the distance alone counts
