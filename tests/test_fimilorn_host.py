"""CPU tests of the Fimilorn host code: the config reader, the layer runs, the registry, the mapping of checkpoint tensors to
engine weights, and the oracle's own consistency (causality, windows, sinks, retention against its direct sum, rotations
that depend on the distance only, routing, clamps, repeated layers)."""
import ctypes as C
import json

import pytest
import torch

from llmq_b200 import fimilorn as F
from llmq_b200 import lib as L
from oracle import fimilorn as O
from tests.fimilorn_util import (DENSE, MOE, MOE_ALONE, MOE_GROUPS_OF_ONE, attn, checkpoint, latent, retention, small_spec,
                                 tokens)


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
    back = F.FimilornSpec.from_config(cfg)
    assert back.base_layers == spec.base_layers and back.layers == spec.layers
    assert (back.width, back.vocab, back.rms_eps, back.loop) == (96, 211, 1e-5, (1, 4, 3))
    with pytest.raises(ValueError):
        F.FimilornSpec.from_config({**cfg, "architecture": "Other"})
    for path, value in ((("layers", 0, "type"), "unknown"), (("layers", 2, "mixer", "kv_heads"), 4),
                        (("layers", 0, "mixer", "rot", "dims"), 13), (("layers", 0, "mixer", "rot", "dims"), 22),
                        (("layers", 1, "mixer", "rot", "dims"), 10), (("layers", 0, "mixer", "decay"), [0.5]),
                        (("layers", 1, "mlp", "router", "groups", "count"), 5),
                        (("layers", 1, "mlp", "router", "groups", "keep"), 5), (("layers", 1, "mlp", "router", "top"), 7),
                        (("layers", 0, "mlp", "kind"), "other"), (("loop", "stop"), 7), (("loop", "start"), 4),
                        (("loop", "times"), 0)):
        with pytest.raises(ValueError):
            F.FimilornSpec.from_config(_with(cfg, path, value))
    # what a config leaves out is off: no loop, no window, no rotation, as many key heads as heads, one group, no shared expert
    bare = json.loads(json.dumps(cfg))
    del bare["loop"], bare["layers"][0]["mixer"]["rot"], bare["layers"][1]["mixer"]["mask"]
    del bare["layers"][2]["mixer"]["kv_heads"], bare["layers"][1]["mlp"]["router"]["groups"], bare["layers"][1]["mlp"]["shared"]
    sp = F.FimilornSpec.from_config(bare)
    assert sp.loop is None and sp.n_layers == 6 and all(ly.step is None for ly in sp.layers)
    assert sp.layers[0].rot_dims == 0 and sp.layers[1].window == 0 and sp.layers[2].kv_heads == 6
    assert (sp.layers[1].n_groups, sp.layers[1].keep_groups, sp.layers[1].shared_ff) == (1, 1, 0)
    ex = spec.config_extras()
    assert (ex["arch"], ex["layer_form"], ex["norm_kind"]) == (L.ARCH_FIMILORN, L.FORM_SANDWICH, L.NORM_RMS)
    d = [ly.desc() for ly in spec.layers]
    assert (d[0].mixer, d[0].heads, d[0].dim, d[0].vdim, d[0].rot_dims, d[0].ff, d[0].ff_dim, d[0].inject) == \
        (L.MIXER_RETENTION, 3, 20, 28, 12, L.FF_CLAMPED, 72, L.INJECT_NONE)
    assert abs(d[0].ff_limit - 0.8) < 1e-6 and d[0].rot_base == 300.0
    assert (d[1].mixer, d[1].q_rank, d[1].kv_rank, d[1].rot_dim, d[1].window, d[1].rot_half, d[1].sink, d[1].head_gate,
            d[1].inject) == (L.MIXER_LATENT_ATTN, 0, 40, 8, 19, 1, 1, 0, L.INJECT_STEP)
    assert (d[1].ff, d[1].n_experts, d[1].top_k, d[1].n_groups, d[1].keep_groups, d[1].shared_dim) == \
        (L.FF_MOE_GATED, 12, 3, 4, 2, 40)
    assert (d[2].mixer, d[2].kv_heads, d[2].qk_norm, d[2].bare, d[2].channel_gate, d[2].sink, d[2].window, d[2].inject) == \
        (L.MIXER_WINDOW_ATTN, 2, 1, 1, 1, 1, 0, L.INJECT_NONE)


def test_layer_runs():
    spec = small_spec()
    assert [(ly.src, ly.step) for ly in spec.layers] == [
        (0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None), (1, 2), (2, None), (3, None), (4, None), (5, None)]
    assert [(i, t) for i, t in O.layer_runs(spec.to_config())] == [(ly.src, ly.step) for ly in spec.layers]
    inj = [ly.desc().inject for ly in spec.layers]
    assert inj == [0, L.INJECT_STEP, 0, 0, L.INJECT_STEP_EMBED, 0, 0, L.INJECT_STEP_EMBED, 0, 0, 0, 0]
    once = small_spec(loop=(0, 6, 1))
    assert once.n_layers == 6 and once.layers[0].step == 0 and once.layers[0].desc().inject == L.INJECT_STEP


def test_layer_description_matches_the_header(tmp_path):
    import os
    import subprocess
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    src = tmp_path / "t.c"
    src.write_text('#include "b200q.h"\n#include <stdio.h>\n#include <stddef.h>\n'
                   'int main(void){printf("%zu %zu %zu %zu %d %d %d\\n", sizeof(b200q_layer_desc), offsetof(b200q_layer_desc, '
                   'sink), offsetof(b200q_layer_desc, channel_gate), offsetof(b200q_layer_desc, rot_half), '
                   'B200Q_MIXER_RETENTION, B200Q_FF_MOE_GATED, B200Q_INJECT_STEP_EMBED);return 0;}\n')
    exe = tmp_path / "t"
    subprocess.run(["gcc", "-std=c99", "-I", os.path.join(root, "include"), str(src), "-o", str(exe)], check=True)
    got = [int(x) for x in subprocess.run([str(exe)], capture_output=True, text=True, check=True).stdout.split()]
    assert got == [C.sizeof(L.LayerDesc), L.LayerDesc.sink.offset, L.LayerDesc.channel_gate.offset, L.LayerDesc.rot_half.offset,
                   L.MIXER_RETENTION, L.FF_MOE_GATED, L.INJECT_STEP_EMBED]


def test_resolve_model_picks_the_class_by_config(tmp_path):
    from llmq_b200.model import BUILTIN_SPECS, resolve_model
    spec = small_spec()
    sd = checkpoint(spec, 2)
    (tmp_path / "config.json").write_text(json.dumps(spec.to_config()))
    F.save_checkpoint(str(tmp_path / "model.safetensors"), sd)
    got, d = resolve_model(str(tmp_path))
    assert isinstance(got, F.FimilornSpec) and got.layers == spec.layers and d == str(tmp_path)
    assert BUILTIN_SPECS["fimilorn-1b"].layered and resolve_model("random:fimilorn-1b")[1] is None
    loaded = F.load_checkpoint(str(tmp_path / "model.safetensors"))
    assert set(loaded) == set(sd) and all(torch.equal(loaded[k], sd[k]) for k in sd)


def test_engine_weights_shapes_fusions_and_sharing():
    spec = small_spec()
    sd = checkpoint(spec, 3)
    ew = dict(spec.engine_weights(sd))
    W = spec.width
    assert ew["lm_head"] is ew["embed"]
    r = spec.layers[0]
    hd, hv = r.heads * r.dim, r.heads * r.vdim
    proj = ew["layers.0.mix.proj"]
    assert proj.shape == ((2 * hd + 2 * hv + 63) // 64 * 64, W)
    assert torch.equal(proj[hd:2 * hd], sd["l0.mix.k"]) and torch.equal(proj[2 * hd + hv:2 * hd + 2 * hv], sd["l0.mix.g"])
    assert ew["layers.0.mix.decay"].dtype == torch.float32 and ew["layers.0.mix.decay"].tolist() == [0.5, 0.875, 0.96875]
    assert ew["layers.0.mlp.gate_up"].shape == (144, W) and torch.equal(ew["layers.0.mlp.gate_up"][72:], sd["l0.mlp.up"])
    a = spec.layers[2]
    qd, gd, gv, av = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim, a.heads * a.vdim
    proj = ew["layers.2.mix.proj"]
    assert proj.shape == ((qd + gd + gv + av + 63) // 64 * 64, W)
    assert torch.equal(proj[qd + gd + gv:qd + gd + gv + av], sd["l2.mix.g"])
    assert ew["layers.2.mix.q_norm"].shape == (qd,) and ew["layers.2.mix.k_norm"].shape == (gd,)
    c = spec.layers[1]
    nq, rp = c.heads * (c.dim + c.rot_dim), c.kv_rank + c.rot_dim
    down = ew["layers.1.mix.down"]
    assert down.shape == ((nq + rp + 63) // 64 * 64, W) and torch.equal(down[nq:nq + rp], sd["l1.mix.dkv"])
    ukt = ew["layers.1.mix.uk_t"]
    assert torch.equal(ukt[c.kv_rank:2 * c.kv_rank].T, sd["l1.mix.uk"][c.dim:2 * c.dim])
    # a shared expert of the experts' size is one more of the stack, one of another size has products of its own
    gu, down = ew["layers.1.mlp.experts_gate_up"], ew["layers.1.mlp.experts_down"]
    assert gu.shape == (13 * 80, W) and down.shape == (13 * W, 40) and "layers.1.mlp.shared_down" not in ew
    assert torch.equal(gu[5 * 80:5 * 80 + 40], sd["l1.mlp.e5.gate"]) and torch.equal(gu[12 * 80 + 40:], sd["l1.mlp.shared.up"])
    assert torch.equal(down[12 * W:], sd["l1.mlp.shared.down"])
    assert ew["layers.2.mlp.experts_gate_up"].shape == (6 * 48, W) and ew["layers.2.mlp.shared_gate_up"].shape == (112, W)
    assert "layers.3.norm2" not in ew and "layers.3.mlp.router" not in ew
    assert "layers.10.mlp.shared_gate_up" not in ew
    router = ew["layers.1.mlp.router"]
    assert router.shape == (64, W) and torch.equal(router[:12], sd["l1.mlp.router"]) and float(router[12:].abs().max()) == 0.0
    # runs of one layer share their tensors; every pass has its own step vector
    for n in ("mix.down", "mlp.experts_gate_up", "norm1b"):
        assert ew[f"layers.1.{n}"] is ew[f"layers.4.{n}"] is ew[f"layers.7.{n}"]
    for run, t in ((1, 0), (4, 1), (7, 2)):
        assert torch.equal(ew[f"layers.{run}.step"], sd["loop.step"][t])
    assert "layers.0.step" not in ew and "layers.2.step" not in ew
    # a dense unit whose size is a multiple of 128: gate and up rows alternate in blocks of 128
    sp2 = small_spec(layers=[retention(ff="dense", ff_dim=256, ff_limit=1.0)], loop=None)
    sd2 = checkpoint(sp2, 4)
    il = dict(sp2.engine_weights(sd2))["layers.0.mlp.gate_up_il"]
    assert torch.equal(il[:128], sd2["l0.mlp.gate"][:128]) and torch.equal(il[384:], sd2["l0.mlp.up"][128:])
    assert spec.weight_bytes_per_token() > 0


def _changed(spec, sd, n, at, vocab=50):
    a = tokens(n, vocab, 1)
    b = list(a)
    b[at] = (b[at] + 1) % vocab
    la, lb = O.forward(spec.to_config(), sd, a), O.forward(spec.to_config(), sd, b)
    return [i for i in range(n) if float((la[i] - lb[i]).abs().max()) > 1e-9]


def test_oracle_reach_of_a_changed_token():
    def one(*layers, loop=None):
        spec = small_spec(width=64, vocab=50, layers=list(layers), loop=loop)
        return spec, checkpoint(spec, 4)
    assert _changed(*one(latent(window=7, **DENSE)), 30, 5) == list(range(5, 12))
    assert _changed(*one(attn(**MOE)), 30, 5) == list(range(5, 30))
    assert _changed(*one(retention()), 30, 5) == list(range(5, 30))
    # every pass has keys of its own: two passes of a window of 4 reach twice as far
    assert _changed(*one(latent(window=4), loop=(0, 1, 2)), 30, 5) == list(range(5, 12))


def test_oracle_sink_takes_weight_and_adds_no_value():
    q = torch.zeros(1, 2, 4, dtype=torch.float64)
    k, v = torch.zeros(1, 1, 4, dtype=torch.float64), torch.ones(1, 1, 3, dtype=torch.float64)
    sink = torch.tensor([0.0, 1.0], dtype=torch.float64)
    out = O.sink_attention(q, k, v, O.visible(1), 0.5, sink)
    assert torch.allclose(out[0, 0], torch.full((3,), 0.5, dtype=torch.float64))
    assert torch.allclose(out[0, 1], torch.full((3,), 1 / (1 + 2.718281828459045), dtype=torch.float64))
    assert torch.allclose(O.sink_attention(q, k, v, O.visible(1), 0.5), torch.ones(1, 2, 3, dtype=torch.float64))


def test_oracle_retention_equals_its_direct_sum():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(9, 2, n, generator=g, dtype=torch.float64) for n in (5, 5, 3))
    lam = torch.tensor([0.9, 0.2], dtype=torch.float64)
    got = O.retention_scan(q, k, v, lam)
    for i in range(9):
        want = sum(lam[:, None] ** (i - j) * (q[i] * k[j]).sum(-1, keepdim=True) * v[j] for j in range(i + 1))
        assert torch.allclose(got[i], want)


def test_oracle_rotation_depends_on_the_distance_only():
    g = torch.Generator().manual_seed(0)
    x = torch.randn(12, 2, 10, generator=g, dtype=torch.float64)
    x[:] = x[0]
    f = O.frequencies({"dims": 6, "base": 100.0})
    assert f.tolist() == [1.0, 100.0 ** (-1 / 3), 100.0 ** (-2 / 3)] and O.frequencies(None).numel() == 0
    r = O.turn(x, f)
    assert torch.equal(r[..., 6:], x[..., 6:]) and torch.equal(r[0], x[0])
    dots = torch.einsum("ihd,jhd->hij", r, r)
    for d in range(1, 5):
        diag = torch.diagonal(dots, offset=d, dim1=1, dim2=2)
        assert float((diag - diag[:, :1]).abs().max()) < 1e-9
    e = torch.zeros(2, 1, 6, dtype=torch.float64)
    e[:, 0, 0] = 1.0
    assert float(O.turn(e, f)[1, 0, 3]) > 1e-3 and float(O.turn(e, f)[1, 0, 1]) == 0.0


def test_oracle_routing_and_units():
    z = torch.tensor([[4.0, -4.0, 1.0, 0.5, 0.9, 0.8]], dtype=torch.float64)
    s = torch.sigmoid(z)
    zero = torch.zeros(6, dtype=torch.float64)
    # groups of two: the sums of the pairs rank them, not the largest score: experts 0, 1 lose against 2, 3 and 4, 5
    idx, w = O.route(z, zero, 3, 3, 2)
    assert sorted(idx[0].tolist()) == [2, 4, 5] and torch.allclose(w[0].sort().values, s[0, [2, 4, 5]].sort().values)
    assert O.route(z, zero, 1)[0].tolist() == [[0]]
    # a correction steers the choice and not the weight; masked experts lose even against negative choices
    corr = torch.tensor([-9.0, -9.0, -3.0, -3.0, -5.0, -5.0], dtype=torch.float64)
    idx, w = O.route(z, corr, 2, 3, 1)
    assert sorted(idx[0].tolist()) == [2, 3] and torch.allclose(w[0].sort().values, s[0, [2, 3]].sort().values)
    # groups of one expert: their sum is the one score
    assert sorted(O.route(z, zero, 2, 6, 2)[0][0].tolist()) == [0, 2]
    g, u = torch.tensor([5.0, -5.0], dtype=torch.float64), torch.tensor([9.0, -9.0], dtype=torch.float64)
    want = torch.tensor([2.0 / (1 + torch.exp(torch.tensor(-3.404))) * 3.0, -5.0 / (1 + torch.exp(torch.tensor(8.51))) * -1.0])
    assert torch.allclose(O.clamped_unit(g, u, 2.0).float(), want.float())
    spec = small_spec(width=64, vocab=50, layers=[attn(**MOE_ALONE), latent(**MOE_GROUPS_OF_ONE)], loop=None)
    assert O.forward(spec.to_config(), checkpoint(spec, 1), [1, 2, 3]).shape == (3, 50)


def test_op_arguments_are_checked_before_any_launch():
    lib = L.load()
    assert lib.b200q_retention_scratch_floats(3, 8, 16) == 3 * 48
    assert lib.b200q_retention(None, 0, 1, 8, 8, 0, None, None, None, 0, None, None, 1, 1, 1e-5, None, None, 1, 0, None) == -1
    assert b"retention" in lib.b200q_last_error()
    assert lib.b200q_moe_route_gated(None, 6, None, 1, 6, 2, 4, 1, 0, *([None] * 8)) == -1
    assert lib.b200q_sandwich_close(None, None, 0, 1, None, None, 0, None, None, None, None, 1, 8, 1e-5, 0, None) == -1
    assert lib.b200q_pass_begin(None, None, None, None, None, None, 1, 8, 1e-5, 0, None) == -1
