"""GPU tests of the Lipedra path: the engine (scheduler, paged caches, carried convolution inputs, kernels) against
oracle/lipedra.py — a plain fp64 restatement that recomputes every position from the tokens, with no cache and no
batching.  The configurations are small, differ from one another in every size, and are drawn here; the fp32 engine is
held to a tight bound, the bf16 engine to a rounding-sized one."""
import json

import numpy as np
import pytest
import torch

from oracle import lipedra as O
from tests.lipedra_util import DENSE, attn, checkpoint, rel_err, small_spec, tile_spec, tokens

pytestmark = pytest.mark.gpu
F32_TOL, BF16_TOL = 2e-4, 6e-2


def build(spec, sd, dtype=torch.float32, max_tokens=512, max_seqs=4, num_blocks=None):
    from llmq_b200.model import BLOCK_SIZE, Engine, NativeModel

    nb = num_blocks or (max_tokens // BLOCK_SIZE + max_seqs)
    model = NativeModel(spec, spec.engine_weights(sd), max_tokens=max_tokens, max_seqs=max_seqs,
                        max_model_len=max_tokens, num_blocks=nb, dtype=dtype, max_logit_rows=max_tokens)
    eng = Engine(model, max_num_seqs=max_seqs, max_num_batched_tokens=max_tokens, max_model_len=model.max_model_len)
    return model, eng


def oracle_logits(spec, sd, toks):
    return O.forward(spec.to_config(), sd, toks, torch.float64).numpy()


def replay_cut(eng, rid, toks, cuts):
    """feed toks to request rid in portions of the given sizes (the rest one by one); logits of every place"""
    out, at, cuts = [], 0, list(cuts)
    while at < len(toks):
        n = min(cuts.pop(0) if cuts else 1, len(toks) - at)
        out.append(eng.step_replay([(rid, toks[at:at + n], list(range(n)))]))
        at += n
    return np.concatenate(out)


def check_close(got, want, dtype, what=""):
    err = rel_err(got, want)
    assert err < (F32_TOL if dtype == torch.float32 else BF16_TOL), f"{what}: {err}"


def _ops():
    from llmq_b200 import lib as L
    return L, L.load()


# ---- every mechanism alone: a one-layer model around it --------------------------------------------------
ONE_LAYER = {
    "attention": [attn()],
    "as_many_key_heads_whole_map_turned_plain_frequencies": [attn(heads=3, kv_heads=3, dim=14, vdim=10, rot_dims=14,
                                                                  original=0.0)],
    "one_head": [attn(heads=1, kv_heads=1, dim=18, vdim=70, rot_dims=4)],
    "no_convolution_no_rotation": [attn(heads=5, kv_heads=1, dim=8, vdim=52, taps=0, rot_dims=0)],
    "one_tap": [attn(taps=1)],
    "two_taps": [attn(taps=2)],
    "many_taps": [attn(taps=9, heads=2, kv_heads=1)],
    "odd_sizes": [attn(heads=4, kv_heads=2, dim=11, vdim=7, rot_dims=6)],
    "many_heads_per_key_head_wide_values": [attn(heads=18, kv_heads=2, dim=8, vdim=140, rot_dims=2)],
    "equal_frequency_bounds": [attn(fast=2.0, slow=2.0)],
    "strong_difference_weak_rest": [attn(diff=0.9, scale=1.1)],
    "borrowed_keys_and_values": [attn(**DENSE), attn(taps=2, kv_from=0, scale=0.15, diff=0.0)],
    "tiles": [attn(heads=4, kv_heads=2, dim=64, vdim=128, rot_dims=32, scale=0.1)],
    "tiles_padded": [attn(heads=6, kv_heads=1, dim=32, vdim=64, rot_dims=10, taps=3)],
    "tiles_many_heads_per_key_head": [attn(heads=22, kv_heads=1, dim=16, vdim=32, rot_dims=16, taps=2)],
    "tiles_wide_maps": [attn(heads=2, kv_heads=1, dim=128, vdim=128, rot_dims=64, scale=0.08)],
    "tiles_more_taps_than_the_vector_kernel": [attn(heads=2, kv_heads=2, dim=16, vdim=96, rot_dims=8, taps=7)],
    "feed_forward": [attn(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2, **DENSE)],
    "feed_forward_tight_limit_blocks": [attn(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2, ff="dense", ff_dim=256,
                                             ff_limit=0.4)],
}


@pytest.mark.parametrize("name", sorted(ONE_LAYER))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_mechanism_alone(cuda, name, dtype):
    spec = small_spec(width=80, vocab=97, layers=ONE_LAYER[name])
    sd = checkpoint(spec, seed=11)
    toks = tokens(45, spec.vocab, 5)
    model, eng = build(spec, sd, dtype)
    tap = torch.zeros(spec.n_layers, len(toks), spec.width, device=cuda)
    model.set_layer_tap(tap)
    got = eng.step_replay([(1, toks, list(range(len(toks))))])
    model.set_layer_tap(None)
    stream = []
    want = O.forward(spec.to_config(), sd, toks, torch.float64, stream)
    assert len(stream) == spec.n_layers
    check_close(tap.cpu().numpy()[-1], stream[-1].numpy(), dtype, name)
    check_close(got, want.numpy(), dtype, name)
    # the same tokens one by one through the cache
    again = replay_cut(eng, 2, toks, [])
    check_close(again, want.numpy(), dtype, name + " token by token")
    eng.close()
    model.close()


# ---- op level: made-up inputs that make a fault show ----------------------------------------------------
def _permute(row, r, mask):
    """a cache row [2*dim + vdim] as the kernels store row r of a page"""
    e = torch.arange(row.shape[-1])
    out = torch.empty_like(row)
    out[..., e ^ ((r & mask) << 3)] = row
    return out


def _diff_op(cuda, q, k, v, lam, mult, eps, gate, scale, dtype, portions, block_size=16, companion=False, seed=0):
    """run b200q_diff_attn for one sequence whose keys and values lie in a paged cache with shuffled pages (unused places
    hold garbage).  q [T, H, 2, D], k [T, G, 2, D], v [T, G, V], gate [T, H]; portions: the token counts of successive
    steps; companion puts another sequence's single token (one key, value 1) first in every step."""
    L, lib = _ops()
    T, H, _, D = q.shape
    G, V = k.shape[1], v.shape[2]
    tdt = torch.float32 if dtype == L.DTYPE_F32 else torch.bfloat16
    tiled = lib.b200q_diff_attn_tiled(D, V, block_size, dtype)
    mask, RW = (7 if tiled else 0), 2 * D + V
    nb = (T + block_size - 1) // block_size
    pages = np.random.default_rng(seed).permutation(nb + 4)[:nb + 1].astype(np.int32)
    cache = torch.full((nb + 4, G, block_size, RW), 1e4)
    rows = torch.cat([k.reshape(T, G, 2 * D), v], -1)
    for t in range(T):
        cache[int(pages[t // block_size]), :, t % block_size] = _permute(rows[t], t % block_size, mask)
    ones = torch.cat([torch.zeros(G, 2 * D), torch.arange(1.0, V + 1).expand(G, V)], -1)
    cache[int(pages[nb]), :, 0] = _permute(ones, 0, mask)
    cache = cache.to(tdt).to(cuda).contiguous()
    bt = torch.zeros(2, nb, dtype=torch.int32)
    bt[0, 0] = int(pages[nb])
    bt[1] = torch.tensor(pages[:nb])
    bt = bt.to(cuda).contiguous()
    qd = (q * scale * (1.4426950408889634 if tiled else 1.0)).to(tdt if tiled else torch.float32).to(cuda)
    lamd = torch.tensor([lam], dtype=torch.float32, device=cuda)
    got, at = torch.zeros(T, H, V), 0
    for n in portions:
        n = min(n, T - at)
        if n <= 0:
            break
        c = 1 if companion else 0
        q_step = torch.zeros(c + n, H, 2, D, dtype=qd.dtype, device=cuda)
        q_step[c:] = qd[at:at + n]
        g_step = torch.zeros(c + n, H + 3, dtype=tdt, device=cuda)
        g_step[c:, :H] = gate[at:at + n].to(tdt).to(cuda)
        row_seq = torch.tensor([0] * c + [c] * n, dtype=torch.int32, device=cuda)
        pos = torch.tensor([0] * c + list(range(at, at + n)), dtype=torch.int32, device=cuda)
        desc = torch.tensor(([[0, 1, 0, 0]] if c else []) + [[c, n, at, c]], dtype=torch.int32, device=cuda)
        table = bt if c else bt[1:].contiguous()
        out = torch.zeros(c + n, H * V + 8, dtype=tdt, device=cuda)
        L.check(lib.b200q_diff_attn(q_step.data_ptr(), cache.data_ptr(), table.data_ptr(), nb, row_seq.data_ptr(),
                                    pos.data_ptr(), desc.data_ptr(), 1 + c, n if at % 2 else 0, c + n, H, G, D, V,
                                    block_size, lamd.data_ptr(), mult, eps, g_step.data_ptr(), H + 3, out.data_ptr(), H * V + 8, dtype, None))
        torch.cuda.synchronize()
        assert float(out[:, H * V:].float().abs().max()) == 0.0            # nothing behind the heads is touched
        if c:                                                              # its only key, gate 0: a half
            one = torch.arange(1.0, V + 1).to(tdt).double() * (1.0 - lam)
            one = one / torch.sqrt((one * one).mean() + eps) * mult * 0.5
            assert torch.allclose(out[0, :H * V].double().cpu().view(H, V), one.expand(H, V), atol=2e-2, rtol=2e-2)
        got[at:at + n] = out[c:, :H * V].float().cpu().view(n, H, V)
        at += n
    assert lib.b200q_wait_failures() == 0
    return got


def _standout(T, H, G, D, V, marks, seed):
    """small random queries and keys; at the marked positions of a map the key points along the map's query direction and
    is large, so whoever sees it is dominated by it; every position has a random value vector of its own, so the
    direction of an output names the keys it saw"""
    g = torch.Generator().manual_seed(seed)
    u = torch.randn(G, 2, D, generator=g)
    u = u / u.norm(dim=-1, keepdim=True)
    q = 0.05 * torch.randn(T, H, 2, D, generator=g) + 6.0 * u.repeat_interleave(H // G, 0)[None]
    k = 0.3 * torch.randn(T, G, 2, D, generator=g)
    for mp in (0, 1):
        for j in marks[mp]:
            k[j, :, mp] = 4.0 * u[:, mp]
    v = torch.randn(T, G, V, generator=g)
    return q, k, v, torch.randn(T, H, generator=g)


def _want(q, k, v, lam, mult, eps, gate, scale):
    q, k, v = q.double(), k.double(), v.double()
    a1, a2 = (O.causal_map(q[:, :, m], k[:, :, m], v, scale) for m in (0, 1))
    return O.rms(a1 - lam * a2, eps) * mult * torch.sigmoid(gate.double())[:, :, None]


DIFF_CASES = [
    # (T, H, G, D, V, block size, marked keys of map 1, of map 2)
    (150, 4, 2, 24, 40, 16, [2, 47, 100], [3, 63, 64]),              # sizes no tile takes
    (300, 4, 2, 64, 128, 16, [0, 15, 63, 127], [16, 64, 128, 255]),  # tile sizes: marks at page and tile borders
    (420, 2, 1, 64, 64, 16, [5], [17]),                              # one far key among hundreds in each map
    (200, 12, 1, 32, 128, 16, [1, 31, 96], [0, 32, 130]),            # padded maps, more heads than a decode tile
    (170, 3, 3, 128, 128, 16, [7, 64, 65], [8, 16, 111]),            # the widest tile
    (140, 16, 2, 16, 32, 16, [0, 79], [1, 80]),                      # the smallest tile
    (90, 6, 2, 11, 7, 8, [0, 7, 8], [15, 16]),                       # odd sizes, pages of 8
    (130, 2, 2, 40, 300, 32, [31, 32], [63]),                        # wide values, pages of 32
    (70, 4, 4, 64, 128, 32, [31, 32], [3]),                          # tile sizes in pages the tiles do not take
]


@pytest.mark.parametrize("case", range(len(DIFF_CASES)))
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("how", ["whole", "portions", "single"])
def test_far_keys_pages_tiles_and_both_maps(cuda, case, dtype, how):
    """a key that dominates whoever sees it, in one map only: visible from its own position on and not one before, at
    page borders and tile borders, far back among hundreds; whole, in portions of 1 to 130 tokens beside another
    sequence, and token by token"""
    L, _ = _ops()
    T, H, G, D, V, bs, m1, m2 = DIFF_CASES[case]
    q, k, v, gate = _standout(T, H, G, D, V, (m1, m2), seed=case)
    dt = L.DTYPE_F32 if dtype == "f32" else L.DTYPE_BF16
    if dtype == "bf16":                                                   # what cache and rows can hold
        k, v, gate = (x.bfloat16().float() for x in (k, v, gate))
    lam, mult, eps, scale = 0.55, 0.65, 1e-5, 0.9
    want = _want(q, k, v, lam, mult, eps, gate, scale)
    portions = {"whole": [T], "portions": [1, 2, 16, 3, 70, 17, 1, 1, 33, 130, 64, 5] * 4, "single": [1] * T}[how]
    got = _diff_op(cuda, q, k, v, lam, mult, eps, gate, scale, dt, portions, bs, companion=how != "whole", seed=case)
    assert rel_err(got.reshape(-1, V), want.reshape(-1, V)) < (1e-4 if dtype == "f32" else 4e-2)
    # the marks do what they are meant to: a mark one place off, or in the other map, would show
    for wrong in (([m1[0] + 1] + m1[1:], m2), (m1, m2[:-1] + [m2[-1] + 1]), (m2, m1)):
        qq, kk, vv, _ = _standout(T, H, G, D, V, wrong, seed=case)
        assert rel_err(_want(qq, kk, vv, lam, mult, eps, gate, scale).reshape(-1, V), want.reshape(-1, V)) > 0.3


PREP_CASES = [
    # (H, G, D, V, taps, rotated dims, own keys)
    (4, 2, 64, 128, 4, 32, True), (3, 1, 16, 32, 2, 16, True), (2, 2, 32, 64, 3, 10, True), (2, 1, 16, 96, 1, 6, True),
    (4, 2, 64, 128, 4, 64, False), (2, 1, 48, 32, 0, 0, True), (3, 3, 16, 32, 7, 4, True), (4, 2, 11, 7, 3, 6, True),
    (6, 2, 20, 36, 5, 12, False),
]


@pytest.mark.parametrize("case", range(len(PREP_CASES)))
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("cuts", [[70], [2, 3, 1, 1, 40, 2, 1, 17, 3], [1] * 20])
def test_preparation_continues_across_portions(cuda, case, dtype, cuts):
    """biases, convolution, rotation and cache rows of a sequence in portions, beside a second sequence of other lengths,
    with dirty state slots: queries and cache rows equal those of the whole sequence, the carried values are the last
    projected ones"""
    L, lib = _ops()
    H, G, D, V, taps, rd, own = PREP_CASES[case]
    dt, tdt = (L.DTYPE_F32, torch.float32) if dtype == "f32" else (L.DTYPE_BF16, torch.bfloat16)
    bs, T = 16, sum(cuts)
    tiled = lib.b200q_diff_attn_tiled(D, V, bs, dt)
    mask, RW, NQ = (7 if tiled else 0), 2 * D + V, H * 2 * D
    C = NQ + (G * RW if own else 0)
    ld = C + H + -(C + H) % 8
    g = torch.Generator().manual_seed(case)
    proj = torch.randn(2, T, ld, generator=g).to(tdt)
    bias = torch.randn(ld, generator=g) * 0.4
    conv = torch.randn(max(taps, 1), C, generator=g) * 0.5
    freq = O.frequencies(dict(dims=rd, base=60.0, scaling=dict(factor=2.0, original=32, fast=4.0, slow=1.0)))[0] \
        if rd else torch.zeros(0, dtype=torch.float64)
    mag, scale = 1.2, 0.3
    slots = 3
    stride = max(taps - 1, 0) * C + 4
    state = torch.full((slots * stride,), 77.0, device=cuda)
    nb = (T + bs - 1) // bs
    pages = np.random.default_rng(case).permutation(2 * nb + 2)
    cache = torch.full((2 * nb + 2, G, bs, RW), 5.0, dtype=tdt, device=cuda)
    bd, cd, fd = bias.to(cuda), conv.to(cuda).contiguous(), freq.to(cuda)
    qs = [[], []]
    at = [0, 0]
    for i, n in enumerate(cuts):
        ns = [n, min([1, 2, 5, 0][i % 4], T - at[1])]                     # the companion: 0 = sits the step out
        part = [s for s in (0, 1) if ns[s] > 0]
        desc, row, rseq, pos, smap = [], 0, [], [], []
        for r, s in enumerate(part):
            desc.append([row, ns[s], at[s], 2 - s])
            row += ns[s]
            rseq += [r] * ns[s]
            pos += list(range(at[s], at[s] + ns[s]))
            smap += [int(pages[s * nb + p // bs]) * bs + p % bs for p in range(at[s], at[s] + ns[s])]
        pr = torch.cat([proj[s, at[s]:at[s] + ns[s]] for s in part]).to(cuda).contiguous()
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=cuda)
        descd, rseqd, posd, smapd = i32(desc), i32(rseq), i32(pos), i32(smap)
        tab = torch.zeros(max(row * rd, 1), device=cuda)
        if rd:
            L.check(lib.b200q_rot_table(fd.data_ptr(), mag, posd.data_ptr(), row, rd // 2, tab.data_ptr(), None))
        q = torch.zeros(row, NQ, dtype=tdt if tiled else torch.float32, device=cuda)
        L.check(lib.b200q_diff_attn_prep(pr.data_ptr(), ld, bd.data_ptr(), cd.data_ptr() if taps else None, taps,
                                         state.data_ptr() if taps > 1 else None, stride, int(own), H, G, D, V, rd,
                                         tab.data_ptr() if rd else None, scale, descd.data_ptr(), rseqd.data_ptr(),
                                         len(part), max(ns) if i % 2 else 0, smapd.data_ptr(), bs, q.data_ptr(),
                                         cache.data_ptr() if own else None, row, dt, None))
        torch.cuda.synchronize()
        for r, s in enumerate(part):
            qs[s].append(q[desc[r][0]:desc[r][0] + ns[s]].float().cpu())
            at[s] += ns[s]
    tol = 2e-5 if dtype == "f32" else 3e-2
    qmul = scale * (1.4426950408889634 if tiled else 1.0)
    for s in (0, 1):
        n = at[s]
        u = proj[s, :n, :C].double() + bias[:C].double()
        y = O.short_conv(u, conv.double().t()) if taps else u
        qw = y[:, :NQ].view(n, H, 2, D)
        kw = y[:, NQ:NQ + G * 2 * D].view(n, G, 2, D) if own else None
        if rd:
            qw = O.turn_pairs(qw, freq, mag)
            kw = O.turn_pairs(kw, freq, mag) if own else None
        assert float((torch.cat(qs[s]).double() - qw.reshape(n, NQ) * qmul).abs().max()) < tol
        if own:
            rows = torch.cat([kw.reshape(n, G, 2 * D), y[:, NQ + G * 2 * D:].view(n, G, V)], -1)
            cc = cache.float().cpu()
            for p in range(n):
                e = torch.arange(RW) ^ ((p % bs & mask) << 3)
                have = cc[int(pages[s * nb + p // bs]), :, p % bs][:, e]
                assert float((have.double() - rows[p]).abs().max()) < tol * 4
        if taps > 1:                                                      # zeros stand for what lies before the start
            st = state[(2 - s) * stride:(2 - s) * stride + (taps - 1) * C].view(taps - 1, C).cpu().double()
            w = torch.zeros(taps - 1, C, dtype=torch.float64)
            m = min(n, taps - 1)
            w[taps - 1 - m:] = u[n - m:]
            if n >= taps - 1:
                assert float((st - w).abs().max()) < 1e-5
            else:
                assert float((st[taps - 1 - m:] - w[taps - 1 - m:]).abs().max()) < 1e-5
    assert float(state[:stride].min()) == 77.0                            # slot 0 is nobody's
    assert float(cache[int(pages[2 * nb])].float().min()) == 5.0          # nor is this page


def test_closing_sum_units_and_tables(cuda):
    """the elementwise kernels against their formulas: both dtypes, widths that are and are not multiples of four, partial
    sums, biases or none, gate and up side by side or in blocks, strided rows"""
    L, lib = _ops()
    g = torch.Generator().manual_seed(1)
    for W, T in ((52, 9), (37, 5), (9000, 2)):
        x, bias, w = torch.randn(T, W, generator=g) * 2, torch.randn(W, generator=g), torch.randn(W, generator=g) * 0.3
        for dt, tdt, tol in ((L.DTYPE_F32, torch.float32, 1e-5), (L.DTYPE_BF16, torch.bfloat16, 3e-2)):
            for splits in (0, 1, 3):                                      # 0: one row in the model dtype
                y = torch.randn(max(splits, 1), T, W, generator=g)
                y = y.to(tdt) if splits == 0 else y
                for b in (None, bias):
                    for nxt in (True, False):
                        xd, yd = x.to(cuda).clone(), y.to(cuda).contiguous()
                        bd, wd = bias.to(cuda), w.to(cuda)
                        out = torch.full((T, W), 7.0, dtype=tdt, device=cuda)
                        L.check(lib.b200q_layer_close(xd.data_ptr(), yd.data_ptr(), int(splits > 0), max(splits, 1),
                                                      bd.data_ptr() if b is not None else None, wd.data_ptr(),
                                                      out.data_ptr() if nxt else None, T, W, 1e-5, dt, None))
                        torch.cuda.synchronize()
                        xw = x.double() + y.double().sum(0) + (b.double() if b is not None else 0.0)
                        assert float((xd.cpu().double() - xw).abs().max()) < 1e-5
                        if nxt:
                            assert float((out.cpu().double() - O.centered_norm(xw, w.double(), 1e-5)).abs().max()) < tol
                        else:
                            assert float(out.float().min()) == 7.0
    for F, block, off in ((48, 8, 8), (48, 0, 8), (45, 0, 3), (45, 9, 1), (256, 128, 16)):
        T, ld = 6, 2 * F + off
        for dt, tdt, tol in ((L.DTYPE_F32, torch.float32, 1e-5), (L.DTYPE_BF16, torch.bfloat16, 3e-2)):
            gu, bias = (torch.randn(T, ld, generator=g) * 2).to(tdt), torch.randn(2 * F, generator=g)
            for b in (None, bias):
                gud, bd = gu.to(cuda), bias.to(cuda)
                out = torch.full((T, F + off), 7.0, dtype=tdt, device=cuda)
                L.check(lib.b200q_clamped_glu_ex(gud.data_ptr(), ld, bd.data_ptr() if b is not None else None,
                                                 out.data_ptr(), F + off, T, F, block, 1.3, dt, None))
                torch.cuda.synchronize()
                v = gu[:, :2 * F].double() + (b.double() if b is not None else 0.0)
                v = v.view(T, F // block, 2, block).transpose(1, 2).reshape(T, 2, F) if block else v.view(T, 2, F)
                assert float((out[:, :F].cpu().double() - O.clamped_unit(v[:, 0], v[:, 1], 1.3)).abs().max()) < tol
                assert float(out[:, F:].float().min()) == 7.0
    pos = torch.tensor([0, 1, 7, 100000], dtype=torch.int32, device=cuda)
    freq = torch.tensor([1.0, 0.37, 1e-4], dtype=torch.float64, device=cuda)
    tab = torch.zeros(4, 3, 2, device=cuda)
    L.check(lib.b200q_rot_table(freq.data_ptr(), 1.25, pos.data_ptr(), 4, 3, tab.data_ptr(), None))
    torch.cuda.synchronize()
    a = pos.cpu().double()[:, None] * freq.cpu()[None]
    assert float((tab.cpu().double() - torch.stack([a.cos(), a.sin()], -1) * 1.25).abs().max()) < 1e-6


@pytest.mark.parametrize("M,F,W", [(5, 128, 64), (200, 256, 192), (700, 384, 128), (4096, 6144, 128)])
def test_product_with_the_clamped_unit_in_its_epilogue(cuda, M, F, W):
    """1-CTA and CTA-pair kernels, rows behind another block of columns, gate and up rows in blocks of 128"""
    from llmq_b200.kabavik import _interleave
    L, lib = _ops()
    gen = torch.Generator().manual_seed(M)
    a = torch.randn(M, W, generator=gen).bfloat16()
    gw, uw = ((torch.randn(F, W, generator=gen) * 0.2).bfloat16() for _ in range(2))
    gb, ub = torch.randn(F, generator=gen), torch.randn(F, generator=gen)
    ld, off = F + 72, 64
    out = torch.full((M, ld), 7.0, dtype=torch.bfloat16, device=cuda)
    ad, wd = a.to(cuda), _interleave(gw, uw).to(cuda).contiguous()
    bd = _interleave(gb[:, None], ub[:, None]).reshape(-1).to(cuda).contiguous()
    L.check(lib.b200q_gemm_clamped_glu_bf16(ad.data_ptr(), wd.data_ptr(), bd.data_ptr(), out.data_ptr() + off * 2, ld, M,
                                            2 * F, W, 1.1, None))
    torch.cuda.synchronize()
    x = ad.double()
    want = O.clamped_unit(x @ gw.to(cuda).double().t() + gb.to(cuda).double(),
                          x @ uw.to(cuda).double().t() + ub.to(cuda).double(), 1.1)
    got = out[:, off:off + F].double()
    assert float((got - want).abs().max()) < 2e-2 * float(want.abs().max())
    assert float(out[:, :off].float().min()) == 7.0 and float(out[:, off + F:].float().min()) == 7.0


# ---- whole models ------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def small():
    spec = small_spec()
    return spec, checkpoint(spec, seed=21)


@pytest.fixture(scope="module")
def tiles():
    spec = tile_spec()
    return spec, checkpoint(spec, seed=31)


@pytest.mark.parametrize("which", ["small", "tiles"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_whole_prompt_every_layer(cuda, request, which, dtype):
    spec, sd = request.getfixturevalue(which)
    toks = tokens(150, spec.vocab, 1)
    model, eng = build(spec, sd, dtype)
    tap = torch.zeros(spec.n_layers, len(toks), spec.width, device=cuda)
    model.set_layer_tap(tap)
    got = eng.step_replay([(1, toks, list(range(len(toks))))])
    model.set_layer_tap(None)
    stream = []
    want = O.forward(spec.to_config(), sd, toks, torch.float64, stream)
    for i in range(spec.n_layers):
        check_close(tap[i].cpu().numpy(), stream[i].numpy(), dtype, f"layer {i}")
    check_close(got, want.numpy(), dtype)
    eng.close()
    model.close()


@pytest.mark.parametrize("which,dtype", [("small", torch.float32), ("tiles", torch.bfloat16)])
@pytest.mark.parametrize("cuts", [[], [1, 1], [2, 2, 2, 3, 5], [16, 16, 1, 15], [3, 1, 64, 2], [64, 2], [65, 90]])
def test_portions_and_token_by_token(cuda, request, which, dtype, cuts):
    """a prompt cut into portions (down to two tokens, shorter than the convolutions reach back, across page and tile
    edges) and then decoded token by token gives the logits of the whole prompt; [] = every token alone from the first"""
    spec, sd = request.getfixturevalue(which)
    toks = tokens(100, spec.vocab, 2)
    want = oracle_logits(spec, sd, toks)
    model, eng = build(spec, sd, dtype)
    got = replay_cut(eng, 1, toks, cuts)
    check_close(got, want, dtype, str(cuts))
    eng.close()
    model.close()


@pytest.mark.parametrize("which", ["small", "tiles"])
def test_long_decoding_past_pages_and_tiles(cuda, request, which):
    spec, sd = request.getfixturevalue(which)
    toks = tokens(330, spec.vocab, 3)
    want = oracle_logits(spec, sd, toks)
    for dtype in (torch.float32, torch.bfloat16):
        model, eng = build(spec, sd, dtype)
        got = replay_cut(eng, 1, toks, [3])
        check_close(got, want, dtype)
        eng.close()
        model.close()


def test_decoding_far_enough_for_a_second_block_of_page_numbers(cuda):
    """a decode warp holds 32 page numbers at a time: single tokens past 32 * 4 pages, after a long prompt, with the
    fused product of long steps; gate and up in blocks"""
    layers = [attn(heads=4, kv_heads=1, dim=32, vdim=64, rot_dims=8, scale=0.2, ff="dense", ff_dim=128, ff_limit=1.0),
              attn(heads=2, kv_heads=1, dim=64, vdim=128, rot_dims=16, scale=0.1, ff="dense", ff_dim=256, ff_limit=2.0)]
    spec = small_spec(width=64, vocab=64, layers=layers)
    sd = checkpoint(spec, seed=9)
    toks = tokens(2100, spec.vocab, 4)
    want = oracle_logits(spec, sd, toks)
    model, eng = build(spec, sd, torch.bfloat16, max_tokens=2176)
    for rid, cuts in ((1, [2040]), (2, [600, 511, 300, 2, 680])):
        got = replay_cut(eng, rid, toks, cuts)
        eng.abort(rid)
        check_close(got, want, torch.bfloat16, str(cuts))
    eng.close()
    model.close()


@pytest.mark.parametrize("which,dtype", [("small", torch.float32), ("tiles", torch.float32), ("tiles", torch.bfloat16)])
def test_mixed_batches_pages_and_slots_reused(cuda, request, which, dtype):
    """up to three live requests in a pool too small for all of them: portions of some beside single tokens of
    others, requests that sit a step out, finished requests whose pages and state slots go to the next one (pool and
    slots start dirty).  Every request must come out as if it had run alone."""
    spec, sd = request.getfixturevalue(which)
    rng = np.random.default_rng(7)
    lens = [37, 5, 64, 18, 1, 49, 33, 2, 80]
    reqs = {i: tokens(n, spec.vocab, 100 + i) for i, n in enumerate(lens)}
    want = {i: oracle_logits(spec, sd, t) for i, t in reqs.items()}
    model, eng = build(spec, sd, dtype, max_tokens=160, max_seqs=3, num_blocks=13)   # 208 token places for 289 tokens
    model.kv.view(torch.int16).fill_(0x4E4E)                                  # large values in either dtype
    model.state.fill_(1e6)
    got = {i: [] for i in reqs}
    at = {i: 0 for i in reqs}
    waiting, live = list(reqs), []
    while waiting or live:
        while waiting and len(live) < 3:
            need = sum((len(reqs[i]) + 15) // 16 for i in live) + (len(reqs[waiting[0]]) + 15) // 16
            if need > 13:
                break
            live.append(waiting.pop(0))
        entries, done = [], []
        for i in live:
            if len(live) > 1 and rng.random() < 0.2:
                continue                                                       # sits this step out
            left = len(reqs[i]) - at[i]
            n = min(left, int(rng.choice([1, 1, 2, 3, 9, 16, 40])))
            entries.append((i, reqs[i][at[i]:at[i] + n], list(range(n))))
        if not entries:
            continue
        out = eng.step_replay(entries)
        row = 0
        for i, t, w in entries:
            got[i].append(out[row:row + len(w)])
            row += len(w)
            at[i] += len(t)
            if at[i] == len(reqs[i]):
                done.append(i)
        for i in done:
            eng.abort(i)
            live.remove(i)
    for i in reqs:
        check_close(np.concatenate(got[i]), want[i], dtype, f"request {i}")
    assert eng.stats().free_blocks == 13
    eng.close()
    model.close()


def test_model_without_convolutions_and_with_units_of_one(cuda):
    """no carried state at all; scale, embedding scale and frequencies' factor 1, diff 0"""
    layers = [attn(heads=2, kv_heads=2, dim=16, vdim=32, taps=0, scale=1.0, diff=0.0, rot_dims=16, factor=1.0, ff="dense",
                   ff_dim=64, ff_limit=1.0),
              attn(heads=3, kv_heads=1, dim=6, vdim=9, taps=1, scale=1.0, diff=0.0, rot_dims=0)]
    spec = small_spec(width=64, vocab=128, layers=layers, embed_scale=1.0)
    sd = checkpoint(spec, seed=5)
    toks = tokens(60, spec.vocab, 8)
    want = oracle_logits(spec, sd, toks)
    for dtype in (torch.float32, torch.bfloat16):
        model, eng = build(spec, sd, dtype)
        assert not hasattr(model, "state") or model.state is None
        check_close(replay_cut(eng, 1, toks, [40, 2, 9]), want, dtype)
        eng.close()
        model.close()


# ---- generation through the engine's own scheduler, sampler and model directory reader ----------------
def _generate(eng, prompts, n_new):
    for i, p in enumerate(prompts):
        eng.add_request(i, p, n_new, ignore_eos=True)
    outs = {i: [] for i in range(len(prompts))}
    while eng.has_work():
        ids, toks, _ = eng.step()
        for i, t in zip(ids.tolist(), toks.tolist()):
            outs[i].append(t)
    return outs


def test_greedy_generation_from_a_model_directory(cuda, small, tmp_path):
    """config.json + model.safetensors on disk -> resolve_model -> NativeModel -> Engine.add_request/step:
    chunked prefill under a small token budget, continuous batching of unequal requests, decode-only steps (graphs),
    more requests than may be live at once"""
    from llmq_b200.lipedra import save_checkpoint
    from llmq_b200.model import Engine, NativeModel, checkpoint_engine_weights, resolve_model

    spec, sd = small
    d = tmp_path / "model"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(spec.to_config()))
    save_checkpoint(str(d / "model.safetensors"), sd)
    spec2, model_dir = resolve_model(str(d))
    assert spec2.layers == spec.layers and spec2.layered and spec2.arch == "lipedra"
    prompts = [tokens(n, spec.vocab, 40 + n) for n in (3, 41, 1, 26, 17, 9)]
    n_new = 24
    model = NativeModel(spec2, checkpoint_engine_weights(spec2, model_dir), max_tokens=32, max_seqs=4,
                        max_model_len=128, num_blocks=24, dtype=torch.float32)
    eng = Engine(model, max_num_seqs=4, max_num_batched_tokens=32)
    outs = _generate(eng, prompts, n_new)
    for i, p in enumerate(prompts):
        assert outs[i] == O.greedy(spec.to_config(), sd, p, n_new), f"request {i}"
    eng.close()
    model.close()


def test_greedy_generation_bf16_matches_its_own_replay(cuda, tiles):
    """bf16 serving on the tensor-core kernels: what the scheduler generates is what a replay of the same tokens predicts
    (sampling, async stepping and graphs change nothing)"""
    spec, sd = tiles
    prompts = [tokens(n, spec.vocab, 60 + n) for n in (12, 30)]
    model, eng = build(spec, sd, torch.bfloat16, max_tokens=64)
    outs = _generate(eng, prompts, 20)
    for i, p in enumerate(prompts):
        full = p + outs[i]
        lg = eng.step_replay([(100 + i, full, list(range(len(full))))])
        eng.abort(100 + i)
        top2 = np.sort(lg[len(p) - 1:-1], -1)[:, -2:]
        clear = (top2[:, 1] - top2[:, 0]) > 0.05 * np.abs(lg).max()         # skip near-ties of bf16 rounding
        pred = lg[len(p) - 1:-1].argmax(-1)
        assert clear.sum() > 3 and (pred[clear] == np.asarray(outs[i])[clear]).all()
    eng.close()
    model.close()
