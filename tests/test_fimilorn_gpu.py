"""GPU tests of the Fimilorn path: the engine (scheduler, paged caches, state slots, kernels) against oracle/fimilorn.py — a
plain fp64 restatement that recomputes every position from the tokens, with no cache, no state and no batching.  The
configurations are small, differ from one another in every size, and are drawn here; the fp32 engine is held to a tight
bound, the bf16 engine to a rounding-sized one."""
import json

import numpy as np
import pytest
import torch

from oracle import fimilorn as O
from tests.fimilorn_util import (DENSE, MOE, MOE_ALL, MOE_ALONE, MOE_GROUPS_OF_ONE, MOE_OTHER_SHARED, attn, calm_routers,
                                 checkpoint, latent, rel_err, retention, small_spec, tile_spec, tokens)

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
    """fp32: every row within the tight bound.  bf16: 97 rows in a hundred within the rounding-sized one and none beyond
    twice that (a head whose output is small before it is divided by its own size carries rounding on, enlarged)"""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    rows = np.sqrt(((got - want) ** 2).mean(-1)) / (np.sqrt((want ** 2).mean(-1)) + 1e-30)
    if dtype == torch.float32:
        assert rows.max() < F32_TOL, f"{what}: {rows.max()}"
    else:
        assert np.quantile(rows, 0.97) < BF16_TOL and rows.max() < 2 * BF16_TOL, f"{what}: {rows.max()}"


def _ops():
    from llmq_b200 import lib as L
    return L, L.load()


# ---- every mechanism alone: a one-layer model around it --------------------------------------------------
TINY = dict(heads=1, dim=8, vdim=8, rot_dims=4, decay=(0.5,))
ONE_LAYER = {
    "retention": ([retention()], None),
    "retention_no_rotation": ([retention(heads=2, dim=72, vdim=8, rot_dims=0, decay=(0.999, 0.25))], None),
    "retention_odd_values": ([retention(heads=1, dim=7, vdim=33, rot_dims=2, decay=(0.9,))], None),
    "retention_wide_keys": ([retention(heads=2, dim=200, vdim=20, rot_dims=200, decay=(1.0, 0.01))], None),
    "retention_wide_values": ([retention(heads=1, dim=16, vdim=1100, rot_dims=16, decay=(0.95,))], None),
    "retention_tiles": ([retention(heads=2, dim=64, vdim=96, rot_dims=48, decay=(0.99, 0.5))], None),
    "retention_tiles_wide": ([retention(heads=1, dim=128, vdim=64, rot_dims=0, decay=(0.97,))], None),
    "attention": ([attn()], None),
    "attention_no_rotation": ([attn(heads=2, kv_heads=1, dim=72, vdim=24, rot_dims=0)], None),
    "attention_as_many_key_heads": ([attn(heads=3, kv_heads=3, dim=10, vdim=6, rot_dims=10)], None),
    "attention_many_heads_per_key": ([attn(heads=18, kv_heads=2, dim=8, vdim=8, rot_dims=2)], None),
    "attention_window": ([attn(window=9)], None),
    "attention_tiles": ([attn(heads=4, kv_heads=1, dim=64, vdim=64, rot_dims=32, scale=0.2)], None),
    "attention_tiles_wide": ([attn(heads=2, kv_heads=2, dim=128, vdim=128, rot_dims=128, scale=0.1)], None),
    "latent": ([latent()], None),
    "latent_window_of_one": ([latent(window=1)], None),
    "latent_every_key": ([latent(heads=5, dim=8, rot_dim=12, vdim=40, kv_rank=24, window=0)], None),
    "latent_partly_rotated": ([latent(rot_dim=12, rot_dims=4)], None),
    "latent_tiles": ([latent(heads=3, dim=64, rot_dim=64, vdim=64, kv_rank=64, window=33, scale=0.1)], None),
    "dense": ([retention(**TINY, **DENSE)], None),
    "dense_blocks": ([retention(**TINY, ff="dense", ff_dim=128, ff_limit=0.5)], None),
    "experts": ([retention(**TINY, **MOE)], None),
    "experts_other_shared": ([retention(**TINY, **MOE_OTHER_SHARED)], None),
    "experts_without_shared": ([retention(**TINY, **MOE_ALONE)], None),
    "experts_groups_of_one": ([retention(**TINY, **MOE_GROUPS_OF_ONE)], None),
    "experts_all_chosen": ([retention(**TINY, **MOE_ALL)], None),
    "one_layer_five_passes": ([attn(**DENSE)], (0, 1, 5)),
    "one_pass_has_its_step_too": ([latent(**DENSE)], (0, 1, 1)),
}


@pytest.mark.parametrize("name", sorted(ONE_LAYER))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_mechanism_alone(cuda, name, dtype):
    """whole, and token by token: every layer run's residual and the logits (bf16 experts: with choices that rounding does
    not turn over)"""
    layers, loop = ONE_LAYER[name]
    wide = "tiles" in name or "blocks" in name
    spec = small_spec(width=128 if wide else 80, vocab=97, layers=layers, loop=loop)
    sd = checkpoint(spec, seed=11)
    if dtype == torch.bfloat16:
        sd = calm_routers(spec, sd)
    toks = tokens(75 if wide else 45, spec.vocab, 5)
    model, eng = build(spec, sd, dtype)
    tap = torch.zeros(spec.n_layers, len(toks), spec.width, device=cuda)
    model.set_layer_tap(tap)
    got = eng.step_replay([(1, toks, list(range(len(toks))))])
    model.set_layer_tap(None)
    stream = []
    want = O.forward(spec.to_config(), sd, toks, torch.float64, stream).numpy()
    assert len(stream) == spec.n_layers
    for i in range(spec.n_layers):
        check_close(tap[i].cpu().numpy(), stream[i].numpy(), dtype, f"{name}, run {i}")
    check_close(got, want, dtype, name)
    eng.abort(1)
    check_close(replay_cut(eng, 2, toks, []), want, dtype, name + ", token by token")
    eng.close()
    model.close()


# ---- op level: made-up inputs that make a fault show ----------------------------------------------------
class Paged:
    """one sequence's rows in a paged cache with shuffled pages (unused places hold garbage) beside a companion sequence
    of a single token, and the step metadata of any portion"""

    def __init__(self, cuda, rows, companion_row, tdt, seed, bs=16):
        T = rows.shape[0]
        self.cuda, self.bs, self.nb = cuda, bs, (T + bs - 1) // bs
        pages = np.random.default_rng(seed).permutation(self.nb + 4)[:self.nb + 1].astype(np.int32)
        self.cache = torch.full(((self.nb + 4) * bs, rows.shape[1]), 1e4, dtype=tdt, device=cuda)
        for t in range(T):
            self.cache[int(pages[t // bs]) * bs + t % bs] = rows[t].to(tdt)
        self.cache[int(pages[self.nb]) * bs] = companion_row.to(tdt)
        bt = torch.zeros(2, self.nb, dtype=torch.int32)
        bt[0, 0] = int(pages[self.nb])
        bt[1] = torch.tensor(pages[:self.nb])
        self.bt = bt.to(cuda).contiguous()

    def step(self, at, n, companion):
        c = 1 if companion else 0
        row_seq = torch.tensor([0] * c + [c] * n, dtype=torch.int32, device=self.cuda)
        pos = torch.tensor([0] * c + list(range(at, at + n)), dtype=torch.int32, device=self.cuda)
        desc = torch.tensor(([[0, 1, 0, 0]] if c else []) + [[c, n, at, c]], dtype=torch.int32, device=self.cuda)
        return c, row_seq, pos, desc, (self.bt if c else self.bt[1:].contiguous())


def portions_of(T, how):
    sizes = {"whole": [T], "portions": [1, 2, 16, 3, 70, 17, 1, 1, 33, 64, 5] * 4, "single": [1] * T}[how]
    at = 0
    for n in sizes:
        n = min(n, T - at)
        if n <= 0:
            return
        yield at, n
        at += n


def standout(T, H, G, D, V, marks, seed):
    """small random queries and keys; at every marked position the key points along the (shared) query direction of its
    group and is large, so whoever sees it is dominated by it; the value of position j is j in every channel, so an
    output row names the keys it saw"""
    g = torch.Generator().manual_seed(seed)
    u = torch.randn(G, D, generator=g)
    u = u / u.norm(dim=-1, keepdim=True)
    qs = 0.05 * torch.randn(T, H, D, generator=g) + 6.0 * u.repeat_interleave(H // G, 0)[None]
    keys = 0.3 * torch.randn(T, G, D, generator=g)
    for j in marks:
        keys[j] = 4.0 * u
    vals = torch.arange(T, dtype=torch.float32)[:, None, None].expand(T, G, V).clone()
    return qs, keys, vals


ATTENTION_CASES = [
    # (T, H, G, D, V, window, marked keys[, first keys that stay visible behind the window])
    (150, 4, 2, 24, 40, 0, [0, 15, 16, 63, 64, 100]),              # sizes no tile takes
    (200, 2, 1, 64, 64, 64, [0, 15, 16, 63, 64, 127, 128, 135]),   # a window of one tile, pages at its edges
    (300, 4, 4, 128, 128, 0, [7]),                                 # every earlier key: one far back among hundreds
    (300, 4, 2, 128, 64, 80, [3, 79, 80, 83, 159, 160, 200]),
    (260, 3, 3, 16, 8, 21, [0, 20, 21, 47, 63, 64, 100, 200]),
    (90, 16, 1, 64, 128, 17, [0, 16, 17, 33, 50]),                 # sixteen heads on one key head
    (70, 24, 1, 128, 64, 0, [0, 18, 40]),                          # more heads per key head than a decode tile has rows
    (200, 4, 2, 64, 64, 33, [0, 2, 3, 40, 100], 3),                # kept first keys beside a sink
    (150, 2, 1, 128, 64, 20, [4, 5, 70], 5),
]


def _attention_want(qs, keys, vals, window, sink, gate, kept=0):
    T, H, D = qs.shape
    G, V = keys.shape[1], vals.shape[2]
    see = O.visible(T, window) | (O.visible(T) & (torch.arange(T)[None, :] < kept))
    out = O.sink_attention(qs.double(), keys.double(), vals.double(), see, 1.0,
                           sink.double() if sink is not None else None)
    return out * torch.sigmoid(gate.double()).view(T, H, V) if gate is not None else out


@pytest.mark.parametrize("case", range(len(ATTENTION_CASES)))
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("how", ["whole", "portions", "single"])
def test_attention_sinks_gates_edges_pages_and_far_keys(cuda, case, dtype, how):
    """a key that dominates whoever sees it, at page, tile and window borders and far back, under sinks that range from
    nothing to as strong as that key, with a gate value per channel: whole, in portions beside another sequence, and
    token by token"""
    L, lib = _ops()
    T, H, G, D, V, window, marks, kept = (ATTENTION_CASES[case] + (0,))[:8]
    qs, keys, vals = standout(T, H, G, D, V, marks, seed=case)
    g = torch.Generator().manual_seed(100 + case)
    dt, tdt = (L.DTYPE_F32, torch.float32) if dtype == "f32" else (L.DTYPE_BF16, torch.bfloat16)
    keys, vals = keys.to(tdt).float(), vals.to(tdt).float()
    gate = torch.randn(T, H * V + 6, generator=g).to(tdt).float()
    # head h's sink: -20 (nothing), then up to 24, the score of a marked key
    sink = torch.linspace(-20.0, 24.0, H) if H > 1 else torch.tensor([24.0])
    want = _attention_want(qs, keys, vals, window, sink, gate[:, :H * V], kept)
    without = _attention_want(qs, keys, vals, window, None, gate[:, :H * V], kept)
    assert float((want - without).abs().max()) > 1.0             # the sinks bite
    paged = Paged(cuda, torch.cat([keys.reshape(T, -1), vals.reshape(T, -1)], 1),
                  torch.cat([torch.zeros(G * D), torch.ones(G * V)]), tdt, case)
    sd = sink.to(cuda)
    got = torch.zeros(T, H * V)
    for at, n in portions_of(T, how):
        c, row_seq, pos, desc, table = paged.step(at, n, how != "whole")
        q = torch.zeros(c + n, H, D, device=cuda)
        q[c:] = qs[at:at + n].to(cuda)
        gs = torch.zeros(c + n, H * V + 6, dtype=tdt, device=cuda)
        gs[c:] = gate[at:at + n].to(tdt).to(cuda)
        o = torch.zeros(c + n, H * V, dtype=tdt, device=cuda)
        L.check(lib.b200q_window_attn_sink(q.data_ptr(), paged.cache.data_ptr(), table.data_ptr(), paged.nb,
                                           row_seq.data_ptr(), pos.data_ptr(), desc.data_ptr(), 1 + c, c + n, H, G, D, V,
                                           paged.bs, window, kept, 0.0, sd.data_ptr(), gs.data_ptr(), H * V + 6, 1, n,
                                           o.data_ptr(), dt, None))
        torch.cuda.synchronize()
        if c:   # one key of zeros against the sink: 1 / (1 + exp(sink)), half of it behind the gate
            alone = (0.5 / (1.0 + torch.exp(sink.double())))[:, None].expand(H, V).reshape(-1)
            assert float((o[0].cpu().double() - alone).abs().max()) < 3e-3, "the companion saw foreign keys"
        got[at:at + n] = o[c:].float().cpu()
    tol = 2e-4 if dtype == "f32" else 2e-2
    assert float((got.double().view(T, H, V) - want).abs().max()) < tol * T
    for i in range(T) if H > 1 else []:                         # the marks do what they are meant to (head 0: no sink)
        seen = [m for m in marks if m <= i and (not window or i - m < window or m < kept)]
        if seen:
            assert abs(float(want[i, 0, 0] / torch.sigmoid(gate[i, 0].double())) - sum(seen) / len(seen)) < 0.5


LATENT_CASES = [
    # (T, H, latent size, rotated size, window, marked keys)
    (150, 3, 40, 8, 19, [0, 18, 19, 47, 63, 64, 100]),          # sizes no tile takes
    (200, 5, 64, 64, 64, [0, 15, 16, 63, 64, 127, 128, 135]),   # tile sizes, a window of one tile
    (250, 9, 128, 64, 80, [3, 79, 80, 83, 159, 160, 200]),
    (256, 2, 128, 16, 0, [5]),                                  # every earlier key: one far back among hundreds
    (120, 20, 256, 64, 33, [0, 32, 33, 64, 65, 97]),            # more heads than one tile has rows
    (300, 16, 512, 64, 129, [0, 127, 128, 129, 255, 256]),
    (200, 6, 192, 32, 70, [0, 69, 70, 71, 139, 140]),           # tiles, but no whole eighths of the latent
    (150, 33, 384, 48, 0, [9]),
]


@pytest.mark.parametrize("case", range(len(LATENT_CASES)))
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("how", ["whole", "portions", "single"])
def test_latent_sinks_edges_pages_and_far_keys(cuda, case, dtype, how):
    """a marked row dominates whoever sees it and the first latent channel holds the row's position (the query ignores that
    channel), so an output names the rows it saw; sinks from nothing to as strong as a marked row"""
    L, lib = _ops()
    T, H, R, P, window, marks = LATENT_CASES[case]
    RP = R + P
    g = torch.Generator().manual_seed(case)
    u = torch.randn(RP, generator=g)
    u[0] = 0.0
    u = u / u.norm()
    qa = 0.05 * torch.randn(T, H, RP, generator=g) + 6.0 * u
    qa[..., 0] = 0.0
    rows = 0.3 * torch.randn(T, RP, generator=g)
    for j in marks:
        rows[j] = 4.0 * u
    rows[:, 0] = torch.arange(T, dtype=torch.float32)
    dt, tdt = (L.DTYPE_F32, torch.float32) if dtype == "f32" else (L.DTYPE_BF16, torch.bfloat16)
    rows = rows.to(tdt).float()
    sink = torch.linspace(-20.0, 0.9 * 24.0, H)
    want = O.sink_attention(qa.double(), rows[:, None].double(), rows[:, None, :R].double(), O.visible(T, window), 0.9,
                            sink.double())
    assert float((want - O.sink_attention(qa.double(), rows[:, None].double(), rows[:, None, :R].double(),
                                          O.visible(T, window), 0.9)).abs().max()) > 1.0
    paged = Paged(cuda, rows, torch.ones(RP), tdt, case)
    sd = sink.to(cuda)
    got = torch.zeros(T, H * R)
    for at, n in portions_of(T, how):
        c, row_seq, pos, desc, table = paged.step(at, n, how != "whole")
        q = torch.zeros(c + n, H, RP, device=cuda)
        q[c:] = qa[at:at + n].to(cuda)
        o = torch.zeros(c + n, H * R, dtype=tdt, device=cuda)
        L.check(lib.b200q_latent_attn_sink(q.data_ptr(), paged.cache.data_ptr(), table.data_ptr(), paged.nb,
                                           row_seq.data_ptr(), pos.data_ptr(), c + n, H, R, P, paged.bs, window, 0.9,
                                           sd.data_ptr(), None, 0, o.data_ptr(), dt, None))
        torch.cuda.synchronize()
        if c:   # one row of ones, score 0: 1 / (1 + exp(sink))
            alone = (1.0 / (1.0 + torch.exp(sink.double())))[:, None].expand(H, R).reshape(-1)
            assert float((o[0].cpu().double() - alone).abs().max()) < 5e-3, "the companion saw foreign rows"
        got[at:at + n] = o[c:].float().cpu()
    tol = 2e-4 if dtype == "f32" else 2e-2
    assert float((got.double().view(T, H, R) - want).abs().max()) < tol * T
    for i in range(T):                                          # the marks do what they are meant to (head 0: no sink)
        seen = [m for m in marks if m <= i and (not window or i - m < window)]
        if seen:
            assert abs(float(want[i, 0, 0]) - sum(seen) / len(seen)) < 0.5


EXPANDED_CASES = [
    # (T, H, unrotated, rotated, values, latent size, window, marked keys)
    (200, 2, 64, 64, 64, 64, 64, [0, 15, 16, 63, 64, 127, 128, 135]),
    (300, 3, 128, 64, 128, 128, 80, [3, 79, 80, 83, 159, 160, 200]),
    (256, 8, 40, 24, 64, 64, 0, [5]),                            # a key of 64 whose parts are no multiples of 16
    (150, 2, 96, 96, 128, 192, 19, [0, 18, 19, 47, 63, 64, 100]),
]


@pytest.mark.parametrize("case", range(len(EXPANDED_CASES)))
@pytest.mark.parametrize("how", ["whole", "portions"])
def test_latent_portions_over_expanded_rows(cuda, case, how):
    """the rows a portion sees are gathered from their pages in order, every sequence's span where it should be; keys of two
    parts (expanded, and shared in the cache), a dominating key at window, page and tile edges, sinks and gates per head;
    single tokens of the step are left alone"""
    L, lib = _ops()
    T, H, D, P, V, R, window, marks = EXPANDED_CASES[case]
    assert lib.b200q_latent_expand_ok(H, D, P, V, R, 16, L.DTYPE_BF16) == 1
    g = torch.Generator().manual_seed(case)
    u = torch.randn(D + P, generator=g)
    u = u / u.norm()
    q = (0.05 * torch.randn(T, H, D + P, generator=g) + 6.0 * u).bfloat16().float()
    keys = 0.3 * torch.randn(T, H, D + P, generator=g)
    keys[..., D:] = keys[:, :1, D:]                              # the rotated part is shared by the heads
    for j in marks:
        keys[j] = 4.0 * u
    keys = keys.bfloat16().float()
    vals = torch.arange(T, dtype=torch.float32)[:, None, None].expand(T, H, V).bfloat16().float()
    lat = torch.randn(T, R, generator=g).bfloat16().float()
    gate = torch.randn(T, H + 3, generator=g).bfloat16().float()
    sink = torch.linspace(-20.0, 21.6, H)
    want = O.sink_attention(q.double(), keys.double(), vals.double(), O.visible(T, window), 0.9, sink.double())
    want = want * torch.sigmoid(gate[:, :H].double())[:, :, None]
    paged = Paged(cuda, torch.cat([lat, keys[:, 0, D:]], 1), torch.ones(R + P), torch.bfloat16, case)
    sd = sink.to(cuda)
    for at, n in portions_of(T, how):
        if n == 1:
            continue
        c, row_seq, pos, desc, table = paged.step(at, n, how != "whole")
        lo = max(0, at - window + 1) if window else 0
        count = at + n - lo
        rows = torch.full((T + 64, R), 9.0, dtype=torch.bfloat16, device=cuda)
        span = torch.full((2 * (c + 1),), -1, dtype=torch.int32, device=cuda)
        L.check(lib.b200q_latent_gather(paged.cache.data_ptr(), table.data_ptr(), paged.nb, desc.data_ptr(), 1 + c, count, window,
                                        16, R, P, T + 64, rows.data_ptr(), span.data_ptr(), None))
        torch.cuda.synchronize()
        assert span.cpu().tolist() == [-1, -1] * c + [0, lo]
        assert torch.equal(rows[:count].float().cpu(), lat[lo:lo + count]) and float(rows[count:].float().min()) == 9.0
        ldq = H * (D + P) + 8
        q16 = torch.zeros(c + n, ldq, dtype=torch.bfloat16, device=cuda)
        q16[c:, :H * (D + P)] = q[at:at + n].reshape(n, -1).bfloat16().to(cuda)
        qa = torch.full((c + n, H, R + P), 1e4, device=cuda)
        qa[c:, :, R:] = q[at:at + n, :, D:].to(cuda)
        kx = keys[lo:lo + count, :, :D].bfloat16().to(cuda).contiguous()
        vx = vals[lo:lo + count].bfloat16().to(cuda).contiguous()
        gs = torch.zeros(c + n, H + 3, dtype=torch.bfloat16, device=cuda)
        gs[c:] = gate[at:at + n].bfloat16().to(cuda)
        o = torch.full((c + n, H * V), 77.0, dtype=torch.bfloat16, device=cuda)
        L.check(lib.b200q_latent_portion_attn(q16.data_ptr(), ldq, qa.data_ptr(), kx.data_ptr(), vx.data_ptr(), span.data_ptr(),
                                              paged.cache.data_ptr(), table.data_ptr(), paged.nb, desc.data_ptr(), 1 + c, n, H, D,
                                              P, V, R, 16, window, 0.9, sd.data_ptr(), gs.data_ptr(), H + 3, o.data_ptr(), None))
        torch.cuda.synchronize()
        assert float((o[c:].float().cpu().double().view(n, H, V) - want[at:at + n]).abs().max()) < 2e-2 * T
        if c:
            assert float(o[0].float().min()) == 77.0
    for i in range(T):                                          # the marks do what they are meant to (head 0: no sink)
        seen = [m for m in marks if m <= i and (not window or i - m < window)]
        if seen:
            assert abs(float(want[i, 0, 0] / torch.sigmoid(gate[i, 0].double())) - sum(seen) / len(seen)) < 0.6


def test_latent_spans_of_several_portions(cuda):
    """rows of three portions behind two single tokens: each sequence's rows follow the one before, windows cut them"""
    L, lib = _ops()
    R, P, bs = 64, 8, 16
    cache = torch.randn(40 * bs, R + P).bfloat16()
    bt = torch.randperm(40)[:35].view(5, 7).to(torch.int32)
    seqs = [(1, 30), (1, 0), (5, 0), (40, 33), (2, 90)]          # (tokens, position of the first)
    at, desc = 0, []
    for i, (n, p0) in enumerate(seqs):
        desc.append([at, n, p0, i])
        at += n
    cd, btd, dd = cache.to(cuda), bt.to(cuda), torch.tensor(desc, dtype=torch.int32, device=cuda)
    for window in (0, 20):
        want, spans = [], [[-1, -1], [-1, -1]]
        for i, (n, p0) in enumerate(seqs[2:], 2):
            lo = max(0, p0 - window + 1) if window else 0
            spans.append([len(want), lo])
            want += [cache[int(bt[i, p // bs]) * bs + p % bs, :R] for p in range(lo, p0 + n)]
        out = torch.zeros(len(want) + 3, R, dtype=torch.bfloat16, device=cuda)
        span = torch.full((10,), -1, dtype=torch.int32, device=cuda)
        L.check(lib.b200q_latent_gather(cd.data_ptr(), btd.data_ptr(), 7, dd.data_ptr(), 5, 100, window, bs, R, P, len(want) + 3,
                                        out.data_ptr(), span.data_ptr(), None))
        torch.cuda.synchronize()
        assert span.cpu().view(5, 2).tolist() == spans
        assert torch.equal(out.cpu()[:len(want)], torch.stack(want)) and float(out[len(want):].float().abs().max()) == 0.0


RETENTION_CASES = [
    # (heads, dim, vdim, rotated, decays, dtype)
    (3, 12, 20, 8, (0.9, 0.5, 1.0), "f32"),
    (2, 64, 64, 64, (0.99, 0.25), "f32"),
    (1, 7, 33, 0, (0.8,), "f32"),
    (3, 12, 20, 8, (0.9, 0.5, 1.0), "bf16"),             # sizes the chunks do not take
    (2, 64, 64, 32, (0.99, 0.25), "bf16"),               # chunks
    (3, 64, 96, 64, (0.9995, 0.05, 1.0), "bf16"),        # chunks over narrow value blocks
    (2, 128, 32, 128, (0.97, 0.9), "bf16"),
    (1, 128, 128, 0, (0.999,), "bf16"),
]


@pytest.mark.parametrize("case", range(len(RETENTION_CASES)))
@pytest.mark.parametrize("how", ["whole", "portions", "single"])
def test_retention_across_portions_and_dirty_slots(cuda, case, how):
    """queries and keys turned, the state carried from portion to portion beside a second sequence whose single tokens go
    to another slot; a sequence's first portion ignores what its slot held; an old, strong token is remembered"""
    L, lib = _ops()
    H, D, V, rd, decay, dtype = RETENTION_CASES[case]
    T = 330
    g = torch.Generator().manual_seed(case)
    dt, tdt = (L.DTYPE_F32, torch.float32) if dtype == "f32" else (L.DTYPE_BF16, torch.bfloat16)
    NC = 2 * H * (D + V)
    ld = NC + 8

    def draw(n):
        p = torch.randn(n, ld, generator=g)
        p[min(2, n - 1), H * D:2 * H * D] *= 6.0                 # a strong key near the start
        return p.to(tdt)

    def want_of(p):
        p = p.double()
        f = O.frequencies({"dims": rd, "base": 50.0}) if rd else O.frequencies(None)
        n = p.shape[0]
        q = O.turn(p[:, :H * D].reshape(n, H, D), f)
        k = O.turn(p[:, H * D:2 * H * D].reshape(n, H, D), f) * D ** -0.5
        o = O.retention_scan(q, k, p[:, 2 * H * D:2 * H * D + H * V].reshape(n, H, V), torch.tensor(decay, dtype=torch.float64))
        return O.rms(o, 1e-5).reshape(n, -1) * O.silu(p[:, NC - H * V:NC])

    proj = draw(T)
    want = want_of(proj)
    steps = list(portions_of(T, how))
    comp = draw(len(steps))
    comp_want = want_of(comp)
    lam = torch.tensor(decay, dtype=torch.float32, device=cuda)
    stride = H * D * V + 4
    state = torch.full((5, stride), 1e3, device=cuda)
    freq = O.frequencies({"dims": rd, "base": 50.0}).to(cuda) if rd else None
    got, comp_got = torch.zeros(T, H * V), torch.zeros(len(steps), H * V)
    for s, (at, n) in enumerate(steps):
        c = 0 if how == "whole" else 1
        p = torch.cat(([comp[s:s + 1]] if c else []) + [proj[at:at + n]]).to(cuda).contiguous()
        pos = torch.tensor(([s] if c else []) + list(range(at, at + n)), dtype=torch.int32, device=cuda)
        table = torch.zeros(c + n, max(rd, 2), device=cuda)
        if rd:
            L.check(lib.b200q_rot_table(freq.data_ptr(), 1.0, pos.data_ptr(), c + n, rd // 2, table.data_ptr(), None))
        desc = torch.tensor(([[0, 1, s, 4]] if c else []) + [[c, n, at, 1]], dtype=torch.int32, device=cuda)
        row_seq = torch.tensor([0] * c + [c] * n, dtype=torch.int32, device=cuda)
        scratch = torch.zeros(int(lib.b200q_retention_scratch_floats(H, D, V)) * (c + n), device=cuda)
        o = torch.full((c + n, H * V), 77.0, dtype=tdt, device=cuda)
        L.check(lib.b200q_retention(p.data_ptr(), ld, H, D, V, rd, table.data_ptr() if rd else None, lam.data_ptr(),
                                    state.data_ptr(), stride, desc.data_ptr(), row_seq.data_ptr(), 1 + c, n, 1e-5,
                                    scratch.data_ptr(), o.data_ptr(), c + n, dt, None))
        torch.cuda.synchronize()
        got[at:at + n] = o[c:].float().cpu()
        if c:
            comp_got[s] = o[0].float().cpu()
    tol = 1e-4 if dtype == "f32" else 2e-2
    assert rel_err(got, want) < tol
    if how != "whole":
        assert rel_err(comp_got, comp_want) < tol
    # slots of no sequence, and the space behind a slot's state, are untouched
    assert float(state[[0, 2, 3]].min()) == 1e3 and float(state[1, H * D * V:].min()) == 1e3
    assert float(state[1, :H * D * V].abs().max()) < 1e3


def test_retention_state_in_32_bit_over_chunks(cuda):
    """the tensor-core chunks keep the state to fp32: over 700 tokens of a slow decay it stays within 1e-4 of the fp64 one"""
    L, lib = _ops()
    H, D, V, T = 2, 64, 64, 700
    g = torch.Generator().manual_seed(9)
    ld = 2 * H * (D + V)
    proj = torch.randn(T, ld, generator=g).bfloat16()
    lam = (0.9995, 0.97)
    p = proj.double()
    f = O.frequencies({"dims": 64, "base": 1000.0})
    k = O.turn(p[:, H * D:2 * H * D].reshape(T, H, D), f) * D ** -0.5
    v = p[:, 2 * H * D:2 * H * D + H * V].reshape(T, H, V)
    S = torch.zeros(H, D, V, dtype=torch.float64)
    for t in range(T):
        S = torch.tensor(lam, dtype=torch.float64)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
    state = torch.zeros(1, H * D * V, device=cuda)
    freq, lamd, pd = f.to(cuda), torch.tensor(lam, device=cuda), proj.to(cuda)
    at = 0
    for n in (300, 2, 1, 64, 333):
        pos = torch.arange(at, at + n, dtype=torch.int32, device=cuda)
        table = torch.zeros(n, 64, device=cuda)
        L.check(lib.b200q_rot_table(freq.data_ptr(), 1.0, pos.data_ptr(), n, 32, table.data_ptr(), None))
        desc = torch.tensor([[0, n, at, 0]], dtype=torch.int32, device=cuda)
        row_seq = torch.zeros(n, dtype=torch.int32, device=cuda)
        scratch = torch.zeros(int(lib.b200q_retention_scratch_floats(H, D, V)) * n, device=cuda)
        o = torch.zeros(n, H * V, dtype=torch.bfloat16, device=cuda)
        part = pd[at:at + n].contiguous()
        L.check(lib.b200q_retention(part.data_ptr(), ld, H, D, V, 64, table.data_ptr(), lamd.data_ptr(), state.data_ptr(),
                                    H * D * V, desc.data_ptr(), row_seq.data_ptr(), 1, n, 1e-5, scratch.data_ptr(),
                                    o.data_ptr(), n, L.DTYPE_BF16, None))
        torch.cuda.synchronize()
        at += n
    assert at == T
    assert rel_err(state.cpu().numpy().reshape(1, -1), S.reshape(1, -1).numpy()) < 1e-4


def test_routing_by_groups(cuda):
    """sigmoid scores, corrections, groups by the sum of their two largest choices, masked groups under negative choices,
    ties to the lowest index, the shared expert's pair, and the grouping of the pairs"""
    L, lib = _ops()
    g = torch.Generator().manual_seed(4)
    for E, top, n_groups, keep, shared in ((12, 3, 4, 2, 1), (7, 2, 7, 3, 0), (5, 4, 1, 1, 1), (64, 8, 8, 3, 0), (40, 2, 2, 1, 1)):
        T = 37
        z = torch.randn(T, E, generator=g)
        corr = torch.randn(E, generator=g) * 0.4 - 2.0           # every choice score is negative
        z[0] = 1.0
        c0 = corr.clone()
        for equal in (False, True):
            corr = torch.full((E,), -2.0) if equal else c0       # row 0 with equal corrections: all choices tie
            K, N = top + shared, E + shared
            ints = lambda n: torch.full((n,), -1, dtype=torch.int32, device=cuda)
            idx, off, perm, pair, tab, nt = ints(T * K), ints(N + 1), ints(T * K), ints(T * K), ints((T * K // 128 + N + 1) * 4), ints(4)
            wts = torch.zeros(T * K, device=cuda)
            zd, cd = torch.cat([z, torch.full((T, 3), 50.0)], 1).to(cuda), corr.to(cuda)   # (rows are wider than E)
            L.check(lib.b200q_moe_route_gated(zd.data_ptr(), E + 3, cd.data_ptr(), T, E, top, n_groups, keep, shared, idx.data_ptr(),
                                              wts.data_ptr(), off.data_ptr(), perm.data_ptr(), pair.data_ptr(), tab.data_ptr(),
                                              nt.data_ptr(), None))
            torch.cuda.synchronize()
            want_i, want_w = O.route(z.double(), corr.double(), top, n_groups, keep)
            gi, gw = idx.cpu().view(T, K), wts.cpu().view(T, K)
            for t in range(1 if equal else 0, T):
                if t == 0 and not equal:
                    continue                                     # near-ties of the corrected equal scores
                assert sorted(gi[t, :top].tolist()) == sorted(want_i[t].tolist())
                order = gi[t, :top].argsort()
                assert torch.allclose(gw[t, :top][order].double(), want_w[t][want_i[t].argsort()], atol=1e-6)
            if equal:
                assert gi[0, :top].tolist() == list(range(top))
            if shared:
                assert (gi[:, top] == E).all() and (gw[:, top] == 1.0).all()
            o, pm, pr = off.cpu(), perm.cpu(), pair.cpu().view(T, K)
            for t in range(T):
                for k in range(K):
                    e, at = int(gi[t, k]), int(pr[t, k])
                    assert int(o[e]) <= at < int(o[e + 1]) and int(pm[at]) == t
            assert int(nt.cpu()[0]) == sum((int(o[e + 1]) - int(o[e]) + 127) // 128 for e in range(N))


@pytest.mark.parametrize("W", [64, 90, 320, 1300, 5000])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_closing_sums_and_pass_openings(cuda, W, dtype):
    """x += norm(y), next norm: y a row, split partial sums, a routed sum with and without a second row; x += x0 + step with
    the kept row — against the plain forms, at widths that stay in registers and one that does not"""
    L, lib = _ops()
    dt, tdt = (L.DTYPE_F32, torch.float32) if dtype == "f32" else (L.DTYPE_BF16, torch.bfloat16)
    tol = 1e-5 if dtype == "f32" else 1e-2
    g = torch.Generator().manual_seed(W)
    T, K = 5, 3
    x = torch.randn(T, W, generator=g)
    pw, nw = torch.rand(W, generator=g) + 0.5, torch.rand(W, generator=g) + 0.5
    y, y2 = torch.randn(T, W, generator=g).to(tdt), torch.randn(T, W, generator=g).to(tdt)
    parts = torch.randn(4, T, W, generator=g)
    eo = torch.randn(T * K, W, generator=g).to(tdt)
    pair = torch.randperm(T * K, generator=g).to(torch.int32)
    wts = torch.rand(T * K, generator=g)
    routed = (eo.double()[pair.long()] * wts.double()[:, None]).view(T, K, W).sum(1)
    pwd, nwd, yd, y2d, prd, ed, paird, wd = (t.to(cuda) for t in (pw, nw, y, y2, parts, eo, pair, wts))
    forms = {
        "row": ((yd.data_ptr(), 0, 1, None, None, 0, None), y.double()),
        "parts": ((prd.data_ptr(), 1, 4, None, None, 0, None), parts.double().sum(0)),
        "routed": ((ed.data_ptr(), 0, 1, paird.data_ptr(), wd.data_ptr(), K, None), routed),
        "routed_and_row": ((ed.data_ptr(), 0, 1, paird.data_ptr(), wd.data_ptr(), K, y2d.data_ptr()), routed + y2.double()),
    }
    for name, (args, yv) in forms.items():
        for last in (False, True):
            xd = x.to(cuda)
            out = torch.full((T, W), 7.0, dtype=tdt, device=cuda)
            L.check(lib.b200q_sandwich_close(xd.data_ptr(), *args, pwd.data_ptr(), None if last else nwd.data_ptr(),
                                             out.data_ptr(), T, W, 1e-5, dt, None))
            torch.cuda.synchronize()
            xw = x.double() + O.rms(yv, 1e-5) * pw.double()
            assert float((xd.cpu().double() - xw).abs().max()) < 2e-5, name
            if last:
                assert float(out.float().min()) == 7.0
            else:
                assert rel_err(out.float().cpu(), (O.rms(xw, 1e-5) * nw.double()).numpy()) < tol, name
    x0, step = torch.randn(T, W, generator=g), torch.randn(W, generator=g)
    x0d, sd = x0.to(cuda), step.to(cuda)
    for add in (False, True):
        xd, keep = x.to(cuda), torch.zeros(T, W, device=cuda)
        out = torch.zeros(T, W, dtype=tdt, device=cuda)
        L.check(lib.b200q_pass_begin(xd.data_ptr(), x0d.data_ptr() if add else None, sd.data_ptr(), keep.data_ptr(),
                                     nwd.data_ptr(), out.data_ptr(), T, W, 1e-5, dt, None))
        torch.cuda.synchronize()
        xw = x.double() + (x0.double() if add else 0.0) + step.double()
        assert torch.equal(keep.cpu(), x) and float((xd.cpu().double() - xw).abs().max()) < 1e-5
        assert rel_err(out.float().cpu(), (O.rms(xw, 1e-5) * nw.double()).numpy()) < tol


def test_preparations_read_the_table(cuda):
    """q / k norms over the whole projection and half-split turns by the step's table (window attention), and the latent row
    with its shared key and the turned query parts (latent attention), at scattered positions and cache places"""
    L, lib = _ops()
    g = torch.Generator().manual_seed(2)
    T = 6
    pos = torch.tensor([0, 1, 7, 200, 1000, 123456], dtype=torch.int32)
    slots = torch.tensor([9, 3, -1, 4, 0, 7], dtype=torch.int32)
    posd, slotd = pos.to(cuda), slots.to(cuda)

    def table_of(rd, base):
        f = O.frequencies({"dims": rd, "base": base})
        t = torch.zeros(T, rd, device=cuda)
        fd = f.to(cuda)
        L.check(lib.b200q_rot_table(fd.data_ptr(), 1.0, posd.data_ptr(), T, rd // 2, t.data_ptr(), None))
        torch.cuda.synchronize()
        return f, t

    def turn(v, f):
        n = f.numel()
        a = pos.double()[:, None] * f[None, :]
        c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
        u, w = v[..., :n], v[..., n:2 * n]
        return torch.cat([u * c - w * s, w * c + u * s, v[..., 2 * n:]], -1)

    H, G, D, V = 4, 2, 12, 6
    HD, GD, GV = H * D, G * D, G * V
    ld = HD + GD + GV + 3
    proj = torch.randn(T, ld, generator=g)
    wq, wk = torch.rand(HD, generator=g) + 0.5, torch.rand(GD, generator=g) + 0.5
    f, tab = table_of(8, 50.0)
    q = turn((O.rms(proj[:, :HD].double(), 1e-5) * wq.double()).view(T, H, D), f) * 0.3
    k = turn((O.rms(proj[:, HD:HD + GD].double(), 1e-5) * wk.double()).view(T, G, D), f)
    pd, wqd, wkd = proj.to(cuda), wq.to(cuda), wk.to(cuda)
    qs, cache = torch.zeros(T, HD, device=cuda), torch.full((10, GD + GV), 5.0, device=cuda)
    L.check(lib.b200q_window_attn_prep_tab(pd.data_ptr(), ld, 0, HD, HD + GD, None, H, G, D, V, 1, wqd.data_ptr(),
                                           wkd.data_ptr(), 1e-5, 8, tab.data_ptr(), slotd.data_ptr(), 0.3, qs.data_ptr(),
                                           cache.data_ptr(), T, L.DTYPE_F32, None))
    torch.cuda.synchronize()
    assert float((qs.cpu().double().view(T, H, D) - q).abs().max()) < 1e-5
    for t in range(T):
        if slots[t] >= 0:
            row = cache[int(slots[t])].cpu().double()
            assert float((row[:GD] - k[t].reshape(-1)).abs().max()) < 1e-5
            assert float((row[GD:] - proj[t, HD + GD:HD + GD + GV].double()).abs().max()) < 1e-6
    assert float(cache[[1, 2, 5, 6, 8]].min()) == 5.0 and float(cache[[1, 2, 5, 6, 8]].max()) == 5.0

    D, P, R = 6, 10, 14
    ld = H * (D + P) + R + P + 5
    proj = torch.randn(T, ld, generator=g)
    wc = torch.rand(R, generator=g) + 0.5
    for rd in (8, 10, 0):
        f, tab = table_of(rd, 30.0) if rd else (O.frequencies(None), torch.zeros(1, device=cuda))
        qv = turn(proj[:, :H * (D + P)].double().view(T, H, D + P)[..., D:], f)
        lat = proj[:, H * (D + P):].double()
        c, kr = O.rms(lat[:, :R], 1e-5) * wc.double(), turn(lat[:, R:R + P].reshape(T, 1, P), f)[:, 0]
        pd, wd = proj.to(cuda), wc.to(cuda)
        qa, cache = torch.full((T, H, R + P), 3.0, device=cuda), torch.full((10, R + P), 5.0, device=cuda)
        L.check(lib.b200q_latent_prep_tab(pd.data_ptr(), ld, H, D, R, P, rd, tab.data_ptr(), slotd.data_ptr(), wd.data_ptr(),
                                          qa.data_ptr(), cache.data_ptr(), T, 1e-5, L.DTYPE_F32, None))
        torch.cuda.synchronize()
        assert float((qa.cpu().double()[..., R:] - qv).abs().max()) < 1e-5 and float(qa[..., :R].min()) == 3.0
        for t in range(T):
            if slots[t] >= 0:
                row = cache[int(slots[t])].cpu().double()
                assert float((row - torch.cat([c[t], kr[t]])).abs().max()) < 1e-5
        assert float(cache[[1, 2, 5, 6, 8]].min()) == 5.0 and float(cache[[1, 2, 5, 6, 8]].max()) == 5.0


@pytest.mark.parametrize("H,G,D,V,rd,norm", [(4, 2, 64, 64, 32, 1), (3, 1, 24, 40, 16, 1), (16, 4, 128, 128, 128, 1),
                                              (2, 2, 48, 8, 0, 1), (5, 5, 16, 16, 16, 0), (40, 20, 128, 128, 64, 1)])
def test_query_and_key_preparation_bf16(cuda, H, G, D, V, rd, norm):
    """eight values per thread: norms over the whole projection, turned and unturned pieces, values, places that no token
    names, a token without a place, sizes whose units exceed a block's"""
    L, lib = _ops()
    g = torch.Generator().manual_seed(H)
    T, HD, GD, GV = 5, H * D, G * D, G * V
    ld = HD + GD + GV + 8
    proj = torch.randn(T, ld, generator=g).bfloat16()
    wq, wk = torch.rand(HD, generator=g) + 0.5, torch.rand(GD, generator=g) + 0.5
    pos = torch.tensor([0, 3, 40, 999, 70000], dtype=torch.int32)
    slots = torch.tensor([6, 2, -1, 0, 4], dtype=torch.int32)
    f = O.frequencies({"dims": rd, "base": 100.0}) if rd else O.frequencies(None)
    a = pos.double()[:, None] * f[None, :]
    tab = torch.stack([torch.cos(a), torch.sin(a)], -1).float().contiguous()

    def turn(v):
        n = f.numel()
        c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
        return torch.cat([v[..., :n] * c - v[..., n:2 * n] * s, v[..., n:2 * n] * c + v[..., :n] * s, v[..., 2 * n:]], -1)

    q, k = proj[:, :HD].double(), proj[:, HD:HD + GD].double()
    if norm:
        q, k = O.rms(q, 1e-5) * wq.double(), O.rms(k, 1e-5) * wk.double()
    q, k = turn(q.view(T, H, D)) * 0.3, turn(k.view(T, G, D))
    pd, wqd, wkd, td, sl = (t.to(cuda) for t in (proj, wq, wk, tab, slots))
    qs = torch.zeros(T, HD, device=cuda)
    cache = torch.full((8, GD + GV), 5.0, dtype=torch.bfloat16, device=cuda)
    L.check(lib.b200q_window_attn_prep_tab(pd.data_ptr(), ld, 0, HD, HD + GD, None, H, G, D, V, norm, wqd.data_ptr(),
                                           wkd.data_ptr(), 1e-5, rd, td.data_ptr() if rd else None, sl.data_ptr(), 0.3,
                                           qs.data_ptr(), cache.data_ptr(), T, L.DTYPE_BF16, None))
    torch.cuda.synchronize()
    assert float((qs.cpu().double().view(T, H, D) - q).abs().max()) < 1e-5
    for t in range(T):
        if slots[t] >= 0:
            row = cache[int(slots[t])].float().cpu()
            assert float((row[:GD].double() - k[t].reshape(-1)).abs().max()) < 2e-2
            assert torch.equal(row[GD:], proj[t, HD + GD:HD + GD + GV].float())
    assert float(cache[[1, 3, 5, 7]].float().min()) == 5.0 and float(cache[[1, 3, 5, 7]].float().max()) == 5.0


def test_gated_product_without_biases(cuda):
    """the clamped unit in the product's epilogue with no biases equals the plain form"""
    L, lib = _ops()
    g = torch.Generator().manual_seed(6)
    M, F, K = 300, 256, 128
    a, w = torch.randn(M, K, generator=g).bfloat16(), (torch.randn(2 * F, K, generator=g) * 0.2).bfloat16()
    y = a.double() @ w.double().T
    il = w.view(F // 128, 2, 128, K)
    gate, up = il[:, 0].reshape(F, K), il[:, 1].reshape(F, K)
    want = O.clamped_unit(a.double() @ gate.double().T, a.double() @ up.double().T, 1.5)
    ad, wd = a.to(cuda), w.to(cuda)
    out = torch.zeros(M, F, dtype=torch.bfloat16, device=cuda)
    L.check(lib.b200q_gemm_clamped_glu_bf16(ad.data_ptr(), wd.data_ptr(), None, out.data_ptr(), F, M, 2 * F, K, 1.5, None))
    torch.cuda.synchronize()
    assert y.shape == (M, 2 * F) and rel_err(out.float().cpu(), want.numpy()) < 1e-2


# ---- whole models ------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def small():
    spec = small_spec()
    return spec, checkpoint(spec, seed=21)


@pytest.fixture(scope="module")
def tiles():
    spec = tile_spec()
    return spec, calm_routers(spec, checkpoint(spec, seed=31))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_whole_prompt_every_layer_run(cuda, small, dtype):
    spec, sd = small
    if dtype == torch.bfloat16:
        sd = calm_routers(spec, sd)
    toks = tokens(70, spec.vocab, 1)
    model, eng = build(spec, sd, dtype)
    tap = torch.zeros(spec.n_layers, len(toks), spec.width, device=cuda)
    model.set_layer_tap(tap)
    got = eng.step_replay([(1, toks, list(range(len(toks))))])
    model.set_layer_tap(None)
    stream = []
    want = O.forward(spec.to_config(), sd, toks, torch.float64, stream)
    assert len(stream) == spec.n_layers == 12
    for i in range(spec.n_layers):
        check_close(tap[i].cpu().numpy(), stream[i].numpy(), dtype, f"run {i}")
    check_close(got, want.numpy(), dtype)
    eng.close()
    model.close()


@pytest.mark.parametrize("loop", [None, (0, 6, 2), (0, 1, 3), (5, 6, 2), (2, 3, 1), (0, 6, 1)])
def test_where_the_loop_lies(cuda, loop):
    """no loop, all layers, the first, the last, one pass only: what comes ahead of a pass, and the last layer's sum"""
    spec = small_spec(loop=loop)
    sd = checkpoint(spec, seed=41)
    toks = tokens(40, spec.vocab, 6)
    model, eng = build(spec, sd)
    check_close(replay_cut(eng, 1, toks, [9, 2, 20]), oracle_logits(spec, sd, toks), torch.float32, str(loop))
    eng.close()
    model.close()


@pytest.mark.parametrize("cuts", [[], [1, 1], [2, 2, 2, 3, 5], [16, 16, 1, 15], [20, 2, 21], [19, 19, 2], [64], [7, 90]])
@pytest.mark.parametrize("which,dtype", [("small", torch.float32), ("tiles", torch.bfloat16)])
def test_portions_and_token_by_token(cuda, small, tiles, cuts, which, dtype):
    """a prompt cut into portions (down to two tokens, across page, window and chunk edges) and then decoded token by token
    gives the logits of the whole prompt; [] = every token alone from the first"""
    spec, sd = small if which == "small" else tiles
    toks = tokens(100, spec.vocab, 2)
    model, eng = build(spec, sd, dtype)
    check_close(replay_cut(eng, 1, toks, cuts), oracle_logits(spec, sd, toks), dtype)
    eng.close()
    model.close()


@pytest.mark.parametrize("which,dtype", [("small", torch.float32), ("tiles", torch.float32), ("tiles", torch.bfloat16)])
def test_long_decoding_past_windows_and_pages(cuda, small, tiles, which, dtype):
    spec, sd = small if which == "small" else tiles
    toks = tokens(330, spec.vocab, 3)
    model, eng = build(spec, sd, dtype)
    check_close(replay_cut(eng, 1, toks, [3]), oracle_logits(spec, sd, toks), dtype)
    eng.close()
    model.close()


@pytest.mark.parametrize("which,dtype", [("small", torch.float32), ("tiles", torch.float32), ("tiles", torch.bfloat16)])
def test_mixed_batches_pages_and_slots_reused(cuda, small, tiles, which, dtype):
    """up to three live requests in a pool too small for all of them: portions of some beside single tokens of others,
    requests that sit a step out, finished requests whose pages and slots go to the next one (pool and slots start
    dirty).  Every request must come out as if it had run alone."""
    spec, sd = small if which == "small" else tiles
    rng = np.random.default_rng(7)
    lens = [37, 5, 64, 18, 1, 49, 33, 2, 80, 70]
    reqs = {i: tokens(n, spec.vocab, 100 + i) for i, n in enumerate(lens)}
    want = {i: oracle_logits(spec, sd, t) for i, t in reqs.items()}
    model, eng = build(spec, sd, dtype, max_tokens=160, max_seqs=3, num_blocks=13)   # 208 token places for 359 tokens
    model.kv.view(torch.int16).fill_(0x4E4E)                                  # large values in either dtype
    model.state.fill_(1e3)
    got, at = {i: [] for i in reqs}, {i: 0 for i in reqs}
    waiting, live = list(reqs), []
    while waiting or live:
        while waiting and len(live) < 3:
            need = sum((len(reqs[i]) + 15) // 16 for i in live + [waiting[0]])
            if need > 13:
                break
            live.append(waiting.pop(0))
        entries = []
        for i in live:
            if len(live) > 1 and rng.random() < 0.2:
                continue                                                       # sits this step out
            n = min(len(reqs[i]) - at[i], int(rng.choice([1, 1, 2, 3, 9, 16, 40, 70])))
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
                eng.abort(i)
                live.remove(i)
    for i in reqs:
        check_close(np.concatenate(got[i]), want[i], dtype, f"request {i}")
    assert eng.stats().free_blocks == 13
    eng.close()
    model.close()


def test_a_model_without_any_state_and_one_without_any_cache(cuda):
    for layers in ([attn(**DENSE), latent(**MOE)], [retention(**MOE), retention(heads=1, dim=6, vdim=10, rot_dims=6, decay=(0.7,))]):
        spec = small_spec(layers=layers, loop=(0, 2, 2))
        sd = checkpoint(spec, seed=51)
        toks = tokens(60, spec.vocab, 9)
        model, eng = build(spec, sd)
        check_close(replay_cut(eng, 1, toks, [30, 2]), oracle_logits(spec, sd, toks), torch.float32)
        eng.close()
        model.close()


def test_long_portions_take_the_fused_product(cuda):
    """portions of 512 tokens and more run the dense unit in its product's epilogue (bf16, sizes in blocks of 128), shorter
    ones beside it: one prompt whole, cut in two long portions, and cut short; retention walks many chunks"""
    layers = [retention(heads=2, dim=64, vdim=64, rot_dims=64, decay=(0.998, 0.9), ff="dense", ff_dim=256, ff_limit=0.9),
              attn(heads=2, kv_heads=1, dim=64, vdim=64, rot_dims=32, ff="dense", ff_dim=128, ff_limit=2.0),
              latent(heads=2, dim=32, rot_dim=64, vdim=64, kv_rank=64, window=300, ff="moe", ff_dim=64, n_experts=4, top_k=2,
                     n_groups=1, keep_groups=1, shared_ff=64)]
    spec = small_spec(width=128, vocab=256, layers=layers, loop=(1, 3, 2))
    sd = calm_routers(spec, checkpoint(spec, seed=9))
    toks = tokens(1100, spec.vocab, 4)
    want = oracle_logits(spec, sd, toks)
    for dtype in (torch.float32, torch.bfloat16):
        model, eng = build(spec, sd, dtype, max_tokens=1152)
        for rid, cuts in ((1, [1100]), (2, [520, 580]), (3, [300, 511, 289])):
            got = replay_cut(eng, rid, toks, cuts)
            eng.abort(rid)
            check_close(got, want, dtype, str(cuts))
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
    """config.json + model.safetensors on disk -> resolve_model -> NativeModel -> Engine.add_request/step: chunked prefill
    under a small token budget, continuous batching of unequal requests, decode-only steps from graphs, more requests
    than may be live at once"""
    from llmq_b200.fimilorn import save_checkpoint
    from llmq_b200.model import Engine, NativeModel, checkpoint_engine_weights, resolve_model

    spec, sd = small
    d = tmp_path / "model"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(spec.to_config()))
    save_checkpoint(str(d / "model.safetensors"), sd)
    spec2, model_dir = resolve_model(str(d))
    assert spec2.layers == spec.layers and spec2.layered and spec2.arch == "fimilorn"
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


@pytest.mark.parametrize("which", ["small", "tiles"])
def test_greedy_generation_bf16_matches_its_own_replay(cuda, small, tiles, which):
    """bf16 serving: what the scheduler generates is what a replay of the same tokens predicts (sampling, async stepping and
    graphs change nothing)"""
    spec, sd = small if which == "small" else tiles
    sd = calm_routers(spec, sd)
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
        assert (pred[clear] == np.asarray(outs[i])[clear]).all()
    eng.close()
    model.close()
