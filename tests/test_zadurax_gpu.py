"""Zadurax on the GPU against the plain implementation: the new kernels against float64 torch, every
mechanism alone, whole prompts against token-by-token decoding, portions down to two tokens, unequal
batches against each request alone, slots and pages used again, keys far away, at page borders and on
both sides of every window's edge with attention made sharp, single tokens that a memory must carry over
the borders of its chunks, sinks, long decoding, other sizes, greedy generation through the Python entry
point, and the replay program."""
import json
import math
import os
import random
import subprocess

import numpy as np
import pytest
import torch

import plain_zadurax as P
from helpers import BF16_REL_TO_MAX, TraceBuilder, check_logits, random_tokens, read_step, three_cuts
from zadurax_models import (CONFIGS, attention, config, dense, latent, load_weights, make_model, memory, read_config)

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]
F = torch.float64
DEV = torch.device("cuda:0")


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return {name: make_model(str(tmp_path_factory.mktemp(f"zadurax_{name}")), cfg, seed=900 + i)
            for i, (name, cfg) in enumerate(CONFIGS.items())}


_engines, _plain = {}, {}


def engine_for(models, name, dtype):
    from nnis_b200.engine import Engine
    if (name, dtype) not in _engines:
        _engines[(name, dtype)] = Engine.from_dir(models[name], dtype=dtype, max_tokens=64 * 96)
    return _engines[(name, dtype)]


def plain_of(model_dir, dtype, tokens):
    key = (model_dir, dtype, tuple(tokens))
    if key not in _plain:
        bf = dtype == "bfloat16"
        _plain[key] = P.forward(list(tokens), load_weights(model_dir, bf), read_config(model_dir), emulate_bf16=bf)
    return _plain[key]


def check_rows(model_dir, dtype, rows, what, beyond=0.0):
    """rows: (tokens of the request, position, logits row).  ``beyond``: the part of the bfloat16 rows that may
    lie outside the bound, up to three times it (where sharp attention carries one rounding far)."""
    got, want = np.stack([r for _, _, r in rows]), torch.stack([plain_of(model_dir, dtype, t)[p] for t, p, _ in rows])
    if dtype == "bfloat16" and beyond:
        off = (torch.from_numpy(got).double() - want).abs().max(-1).values
        bound = BF16_REL_TO_MAX * max(1.0, float(want.abs().max()))
        assert float((off > bound).double().mean()) <= beyond and float(off.max()) <= 3 * bound, (what, off.max(), bound)
        return
    check_logits(got, want, dtype, what)


def replay_and_check(models, name, dtype, trace, sequences, tmp_path, what, beyond=0.0):
    from nnis_b200.engine.replay import replay
    engine = engine_for(models, name, dtype)
    out = str(tmp_path / f"out_{name}_{dtype}")
    replay(engine, trace.lines, out)
    usage = engine.cache.usage()
    assert usage["slots_held"] == 0 and not any(usage["pages_held"]), usage
    engine.cache.check()
    vocab = read_config(models[name])["vocab"]
    rows = []
    for step, places in trace.rows.items():
        got = read_step(out, step, vocab)
        assert got.shape[0] == len(places)
        rows += [(sequences[rid], pos, got[i]) for i, (rid, pos) in enumerate(places)]
    check_rows(models[name], dtype, rows, f"{what} {name} {dtype}", beyond)


def run_whole(engine, tokens, want=None):
    from nnis_b200.engine import SequenceStep
    slot = engine.acquire_slot()
    try:
        return engine.step([SequenceStep(slot, tokens, list(range(len(tokens))) if want is None else want)]).cpu().numpy()
    finally:
        engine.release_slot(slot)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ---- the matrix memory ------------------------------------------------------------------------
class MemoryRun:
    """The memory kernels over rows [q | k | v | g | i | f | padding] of several sequences in slots of a
    state area, step by step."""

    def __init__(self, H, d, dv, cap, slots=7, pad=3, seed=0):
        from nnis_b200.csrc import ops
        self.ops, self.H, self.d, self.dv, self.cap, self.pad = ops, H, d, dv, cap, pad
        g = torch.Generator().manual_seed(seed)
        self.ib, self.fb = torch.randn(H, generator=g), torch.randn(H, generator=g)
        self.state = torch.zeros(slots, H, d, dv, device=DEV)
        self.n = torch.zeros(slots, 2, H, d, device=DEV)
        self.m = torch.zeros(slots, 2, H, device=DEV)
        self.at = {}  # slot -> tokens so far

    def plain(self, rows):
        """rows [T, cols] of one sequence, float64 -> outputs [T, H * dv] and the size of what they are sums of"""
        H, d, dv, cap, r = self.H, self.d, self.dv, self.cap, rows.double()
        T = r.shape[0]
        q, k = r[:, :H * d].view(T, H, d) * d ** -0.5, r[:, H * d:2 * H * d].view(T, H, d)
        v = r[:, 2 * H * d:2 * H * d + H * dv].view(T, H, dv)
        gates = r[:, 2 * H * (d + dv):]
        i = cap * torch.tanh((gates[:, :H] + self.ib.double()) / cap)
        f = torch.nn.functional.logsigmoid(cap * torch.tanh((gates[:, H:2 * H] + self.fb.double()) / cap))
        # what one rounding of every product may move an output by: the sums without their signs
        N, S = torch.zeros(H, d, dtype=F), torch.zeros(H, d, dv, dtype=F)
        n, m, bound = torch.zeros(H, d, dtype=F), torch.zeros(H, dtype=F), torch.zeros(T, H, dv, dtype=F)
        out = P.matrix_memory(q, k, v, i, f)
        for t in range(T):
            new = torch.maximum(f[t] + m, i[t])
            keep, take, m = torch.exp(f[t] + m - new), torch.exp(i[t] - new), new
            n = keep[:, None] * n + take[:, None] * k[t]
            N = keep[:, None] * N + take[:, None] * k[t].abs()
            S = keep[:, None, None] * S + take[:, None, None] * (k[t].abs()[:, :, None] * v[t].abs()[:, None, :])
            bottom = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
            bound[t] = ((S * q[t].abs()[:, :, None]).sum(1) + out[t].abs() * (N * q[t].abs()).sum(-1)[:, None]) / bottom[:, None]
        return out.reshape(T, -1), bound.reshape(T, -1)

    def step(self, parts, single=False):
        """parts: (slot, rows) of every sequence of the step -> its outputs; ``single``: by the kernel for single tokens."""
        ops, H = self.ops, self.H
        a = torch.cat([r for _, r in parts]).to(DEV)
        n, counts = a.shape[0], [r.shape[0] for _, r in parts]
        starts = [self.at.get(s, 0) for s, _ in parts]
        o = torch.full((n, H * self.dv), 77.0, device=DEV)
        slots = i32([s for s, _ in parts])
        args = (a, self.ib.to(DEV), self.fb.to(DEV), self.state, self.n, self.m)
        sizes = (H, self.d, self.dv, self.cap, self.d ** -0.5, 1e-6)
        if single:
            assert all(c == 1 for c in counts)
            ops.memory_step(*args, i32(starts), i32(list(range(len(parts)))), slots, o, *sizes)
        else:
            chunks, first = ops.scan_segments(counts, ops.memory_chunk_tokens())
            c = chunks.shape[0]
            ops.memory_prompt(*args, torch.from_numpy(chunks).to(DEV), torch.from_numpy(first).to(DEV), slots,
                              i32([sum(counts[:j]) for j in range(len(counts))]), i32(starts), i32(counts),
                              torch.full((3, n, H), math.nan, dtype=F, device=DEV),
                              torch.full((4, c, H), math.nan, dtype=F, device=DEV),
                              torch.full((c, H, self.d, self.dv), math.nan, device=DEV),
                              torch.full((c, H, self.d), math.nan, device=DEV), o, *sizes)
        for (s, r) in parts:
            self.at[s] = self.at.get(s, 0) + r.shape[0]
        return torch.split(o.cpu().double(), counts)


def memory_rows(T, H, d, dv, pad, g, i_size=2.0, f_centre=2.0, f_size=2.0):
    rows = torch.randn(T, 2 * H * (d + dv) + 2 * H + pad, generator=g)
    off = 2 * H * (d + dv)
    rows[:, off:off + H] *= i_size
    rows[:, off + H:off + 2 * H] = rows[:, off + H:off + 2 * H] * f_size + f_centre
    return rows


def close(got, want, bound, tol=5e-6):
    """Within ``tol`` of the size of the sums that an output is made of (cancellation in them, and a denominator
    near zero, leave fewer digits in the output)."""
    off = float(((got - want).abs() / (bound + 1e-3)).max())
    assert off < tol, off


MEMORY_SIZES = [(3, 20, 28, 6.0), (5, 9, 13, 20.0), (1, 34, 7, 2.5), (2, 64, 128, 12.0), (3, 72, 136, 8.0), (1, 136, 64, 10.0),
                (2, 1, 1, 5.0), (9, 32, 64, 15.0), (1, 300, 36, 15.0), (2, 128, 260, 15.0), (1, 33, 65, 9.0)]


@pytest.mark.parametrize("H, d, dv, cap", MEMORY_SIZES)
def test_the_memory_in_every_cut(H, d, dv, cap):
    """Whole prompts, portions that end at, before and after chunks' borders, single tokens by either kernel,
    unequal sequences in one step, slots used by others before (as the cache hands them out: zeroed)."""
    g = torch.Generator().manual_seed(H * 100 + d)
    run = MemoryRun(H, d, dv, cap, pad=(-2 * H) % 8, seed=d)
    rows = memory_rows(200, H, d, dv, run.pad, g)
    want, bound = run.plain(rows)

    def check(parts_of, cuts, slot):
        at = 0
        for c, single in cuts:
            got, = run.step([(slot, parts_of[at:at + c])], single)
            close(got, want[at:at + c], bound[at:at + c])
            at += c
        assert at == 200
        run.state[slot], run.n[slot], run.m[slot], run.at[slot] = 0.0, 0.0, 0.0, 0
    for slot, cuts in enumerate(([200], [64, 64, 64, 8], [63, 1, 1, 135], [2, 62, 2, 134], [65, 127, 8], [1, 199], [128, 72])):
        check(rows, [(c, False) for c in cuts], slot)
    check(rows, [(1, True)] * 70 + [(60, False)] + [(1, True)] * 3 + [(1, False)] * 2 + [(2, False)] + [(1, True)] * 63, 3)
    others = [memory_rows(n, H, d, dv, run.pad, g) for n in (1, 131, 64, 17)]
    wants = [run.plain(r) for r in others]
    slots = (4, 0, 6, 2)
    got = run.step([(s, r[:-1] if len(r) > 1 else r) for s, r in zip(slots, others)])
    for o, (w, b) in zip(got, wants):
        close(o, w[:o.shape[0]], b[:o.shape[0]])
    got = run.step([(s, r[-1:]) for s, r in zip(slots, others) if len(r) > 1], single=True)
    for o, (w, b) in zip(got, [w for w, r in zip(wants, others) if len(r) > 1]):
        close(o, w[-1:], b[-1:])
    # a row without a sequence is left alone, its slot too
    before = run.state.clone(), run.n.clone(), run.m.clone()
    o = torch.full((1, H * dv), 77.0, device=DEV)
    run.ops.memory_step(rows[:1].to(DEV), run.ib.to(DEV), run.fb.to(DEV), run.state, run.n, run.m, i32([-1]), i32([0]), i32([0]), o,
                        H, d, dv, cap, 1.0, 1e-6)
    assert (o == 77.0).all() and all(torch.equal(x, y) for x, y in zip(before, (run.state, run.n, run.m)))


@pytest.mark.parametrize("i_size, f_centre, f_size, cap", [(6.0, -8.0, 4.0, 14.0), (9.0, 0.0, 9.0, 14.0), (0.2, 9.0, 1.0, 14.0),
                                                           (3.0, 30.0, 5.0, 40.0), (8.0, -30.0, 40.0, 12.0), (5.0, 3.0, 3.0, 0.5)])
def test_the_memory_under_extreme_gates(i_size, f_centre, f_size, cap):
    """Gates that forget at once, that keep everything, that jump between both, and input gates over the
    whole of their range: long sums of log gates whose differences still count."""
    g = torch.Generator().manual_seed(int(i_size * 10 + f_size))
    H, d, dv = 4, 24, 20
    run = MemoryRun(H, d, dv, cap, pad=0, seed=1)
    rows = memory_rows(1500, H, d, dv, 0, g, i_size, f_centre, f_size)
    want, bound = run.plain(rows)
    for slot, cuts in enumerate(([1500], [700, 800], [5, 640, 855])):
        got, at = [], 0
        for c in cuts:
            got.append(run.step([(slot, rows[at:at + c])])[0])
            at += c
        close(torch.cat(got), want, bound, 1e-5)
    got = torch.cat([run.step([(5, rows[t:t + 1])], single=True)[0] for t in range(300)])
    close(got, want[:300], bound[:300], 1e-5)


@pytest.mark.parametrize("place", [0, 1, 62, 63, 64, 65, 127, 128, 150])
@pytest.mark.parametrize("cuts", [[260], [64, 196], [63, 197], [65, 1, 194], [150, 110]])
def test_one_token_is_carried_over_the_borders_of_chunks(place, cuts):
    """Every input gate nearly shut but one: until the end of the prompt, and in tokens decoded after it, the
    output is that token's value times its key's product with the query over the same."""
    H, d, dv, cap = 2, 16, 24, 12.0
    g = torch.Generator().manual_seed(place)
    run = MemoryRun(H, d, dv, cap, pad=4)
    run.ib.zero_()
    run.fb.fill_(40.0)  # keep everything
    rows = memory_rows(270, H, d, dv, 4, g, 0.0, 0.0, 0.0)
    off = 2 * H * (d + dv)
    rows[:, off:off + H] = -60.0
    rows[place, off:off + H] = 60.0
    (want, bound), got, at = run.plain(rows), [], 0
    for c in cuts:
        got.append(run.step([(1, rows[at:at + c])])[0])
        at += c
    got = torch.cat(got + [run.step([(1, rows[t:t + 1])], single=True)[0] for t in range(260, 270)])
    close(got, want, bound)
    v = rows[place, 2 * H * d:2 * H * d + H * dv].double().view(H, dv)
    q, k = rows[:, :H * d].double().view(-1, H, d) * d ** -0.5, rows[place, H * d:2 * H * d].double().view(H, d)
    sign = torch.sign((q * k).sum(-1))[..., None]
    strong = (q * k).sum(-1).abs() > 0.3
    after = torch.arange(270)[:, None] >= place
    assert float(((got.view(270, H, dv) - sign * v)[strong & after]).abs().max()) < 0.01
    assert float(got.view(270, H, dv)[~after.expand(270, H)].abs().max() if place else 0.0) < 0.05


def test_the_memorys_output_is_normed_weighed_and_gated():
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(3)
    for n, H, dv, off, extra in ((9, 3, 28, 7, 5), (70, 1, 130, 0, 0), (5, 8, 33, 12, 1)):
        o, a = torch.randn(n, H * dv, generator=g) * 3, torch.randn(n, off + H * dv + extra, generator=g)
        w = torch.rand(H * dv, generator=g) + 0.5
        pos = torch.arange(n, dtype=torch.int32)
        pos[2] = -1
        want = P.rms(o.double().view(n, H, dv), 1e-5).reshape(n, -1) * w.double() * torch.sigmoid(a[:, off:off + H * dv].double())
        want[2] = 0.0
        for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
            out = torch.full((n, H * dv), 9.0, dtype=dtype, device=DEV)
            ops.memory_finish(o.to(DEV), a.to(DEV), off, w.to(DEV), pos.to(DEV), out, H, dv, 1e-5)
            assert torch.allclose(out.cpu().double(), want, atol=tol, rtol=tol)


# ---- what the other mixers and the feed-forward gained ------------------------------------------
def _latent_reference(q, rows, dv, scale, sink):
    """q [T, H, dk], rows [T, dk] -> [T, H * dv]"""
    T, H = q.shape[:2]
    visible = torch.ones(T, T).tril().bool()
    out = [P.softmax_with_sink(((q[:, a] @ rows.T) * scale).masked_fill(~visible, -math.inf), float(sink[a])) @ rows[:, :dv]
           for a in range(H)]
    return torch.stack(out, 1).reshape(T, -1)


@pytest.mark.parametrize("H, dk, dv", [(3, 56, 48), (8, 33, 27), (16, 144, 128), (5, 40, 16), (64, 96, 64), (4, 304, 272),
                                       (2, 544, 512), (130, 24, 16), (1, 20, 20)])
def test_latent_attention_with_a_sink_in_every_cut(H, dk, dv):
    """Both kernels over scattered pages: whole prompts, later portions, single tokens, slices of the key range
    (the sink counts once, whatever the slices), a first token that has the sink and itself only."""
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(H + dk)
    S, scale = 260, 1.1 / math.sqrt(dk)
    pages = [5, 2, 9, 0, 7]
    r, q = torch.randn(S, dk, generator=g), torch.randn(S, H, dk, generator=g)
    sink = torch.randn(H, generator=g) * 3 + 2
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        rd, qd = r.to(dtype), q.to(dtype)
        cache = torch.full((10, 1, 64, dk), 50.0, dtype=dtype)
        for t in range(S):
            cache[pages[t // 64], 0, t % 64] = rd[t]
        want = _latent_reference(qd.double(), rd.double(), dv, scale, sink)
        assert float((want - _latent_reference(qd.double(), rd.double(), dv, scale, sink - 100)).abs().max()) > 0.1
        table = i32([[3] * 5, pages])
        for a, b, splits in ((0, 130, 1), (0, 1, 1), (0, 1, 2), (130, 190, 1), (190, 191, 1), (191, 192, 3), (0, 200, 4), (259, 260, 5)):
            n = b - a
            pos, seq = i32(list(range(a, b))), torch.ones(n, dtype=torch.int32, device=DEV)
            out = torch.full((n, H * dv), 9.0, dtype=dtype, device=DEV)
            partial = torch.empty(n * H * splits * (dv + 2), device=DEV) if splits > 1 else None
            args = (qd[a:b].reshape(n, -1).to(DEV), cache.to(DEV))
            ops.attention_latent(*args, pos, seq, table, out, H, dv, scale, splits, partial, sink=sink.to(DEV))
            assert torch.allclose(out.cpu().double(), want[a:b], atol=tol, rtol=tol), (dtype, a, b, splits)
            if dtype == torch.bfloat16 and ops.attention_latent_mma_takes(dk, dv, 64):
                out.fill_(9.0)
                if n == 1:  # a decode step: every row a token of its own
                    ops.attention_latent_mma(*args, None, None, None, None, pos, seq, table, out, H, dv, scale, splits, partial,
                                             sink=sink.to(DEV))
                else:
                    tiles = torch.from_numpy(ops.latent_tiles([1, n], [0, a], H, ops.latent_tile_rows(dv)))
                    tiles = tiles[tiles[:, 0] == 1].contiguous().to(DEV)
                    ops.attention_latent_mma(*args, tiles, i32([0, 0]), i32([0, a]), i32([1, n]), pos, seq, table, out, H, dv,
                                             scale, splits, partial, sink=sink.to(DEV))
                assert torch.allclose(out.cpu().double(), want[a:b], atol=tol, rtol=tol), ("mma", a, b, splits)


def test_the_latents_rows_are_turned_with_a_magnitude():
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(4)
    for H, dim, rot, rank, pad in ((3, 20, 8, 48, 4), (2, 9, 6, 27, 3), (1, 64, 32, 300, 8)):
        n, cfg = 70, {"base": 90.0, "dims": rot, "scaling": {"factor": 7.0, "original": 40, "fast": 3.0, "slow": 0.5}}
        freq, size = P.turning_rates(cfg)
        a = torch.randn(n, H * (dim + rot) + rank + rot + pad, generator=g)
        q, rows = torch.empty(n, H * dim, device=DEV), torch.zeros(n, H * (rank + rot), device=DEV)
        cache = torch.zeros(2, 1, 64, rank + rot, device=DEV)
        ops.latent_prep_direct(a.to(DEV), torch.ones(rank, device=DEV), torch.tensor(freq + [0.0], device=DEV), i32(list(range(n))),
                               torch.zeros(n, dtype=torch.int32, device=DEV), i32([[1, 0]]), q, rows, cache, None, H, dim, rank,
                               rot, rot, 1e-5, pairing="neighbours", magnitude=size)
        qa, down = a[:, :H * (dim + rot)].view(n, H, dim + rot), a[:, H * (dim + rot):]
        assert torch.equal(q.cpu().view(n, H, dim), qa[..., :dim])  # (the unturned part has no magnitude)
        assert torch.allclose(rows.cpu().view(n, H, -1)[..., rank:].double(), P.rotate(qa[..., dim:].double(), cfg), atol=1e-4)
        kr = P.rotate(down[:, None, rank:rank + rot].double(), cfg)[:, 0]
        got = torch.cat([cache[1, 0], cache[0, 0]])[:n].cpu().double()
        assert torch.allclose(got[:, rank:], kr, atol=1e-4)
        assert torch.allclose(got[:, :rank], P.rms(down[:, :rank].double(), 1e-5), atol=1e-5)


@pytest.mark.parametrize("n", [1, 9, 16, 17, 200])
def test_products_per_head_with_a_gate_per_value(n):
    """The three forms (few rows, many rows, tensor cores), gates some columns into the rows they lie in."""
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(n)
    for H, K, N, off in ((3, 48, 24, 5), (4, 128, 64, 0), (5, 27, 13, 11), (2, 512, 136, 32)):
        a, w = torch.randn(n, H * K, generator=g), torch.randn(H, N, K, generator=g) / K ** 0.5
        gate = torch.randn(n, off + H * N + 3, generator=g) * 2
        for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
            ad, wd = a.to(dtype), w.to(dtype)
            want = torch.einsum("mbk,bnk->mbn", ad.double().view(n, H, K), wd.double()).reshape(n, -1)
            out = torch.empty(n, H * N, dtype=dtype, device=DEV)
            ops.batched_linear(ad.to(DEV), K, wd.to(DEV), out, N)
            assert torch.allclose(out.cpu().double(), want, atol=tol, rtol=tol)
            ops.batched_linear(ad.to(DEV), K, wd.to(DEV), out, N, gate=gate.to(DEV), gate_off=off)
            want = want * torch.sigmoid(gate[:, off:off + H * N].double())
            assert torch.allclose(out.cpu().double(), want, atol=tol, rtol=tol), (dtype, H, K, N)


def test_keys_as_values_go_to_the_cache_as_projected():
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(8)
    for H, G, d, dims in ((4, 2, 16, 8), (3, 3, 11, 6), (6, 1, 40, 40), (2, 1, 7, 0)):
        n, rot = 70, {"base": 60.0, "dims": dims}
        a = torch.randn(n, (H + G) * d + H * d, generator=g) * 3
        wq, wk = torch.rand(d, generator=g) + 0.5, torch.rand(d, generator=g) - 0.5
        f = P.turning_rates(rot)[0] if dims else []
        q, gate = torch.empty(n, H * d, device=DEV), torch.empty(n, H * d, device=DEV)
        kc, vc = torch.zeros(2, G, 64, d, device=DEV), torch.zeros(2, G, 64, d, device=DEV)
        ops.qkv_prep(a.to(DEV), None, None, torch.tensor(f + [0.0], device=DEV), i32(list(range(n))),
                     torch.zeros(n, dtype=torch.int32, device=DEV), i32([[1, 0]]), q, kc, vc, gate, H, G, d, d, dims, 1e-5,
                     pairing="neighbours", head_weights=(wq.to(DEV), wk.to(DEV)), values_are_keys=True)
        turn = lambda x, heads, w: P.rotate(P.norm(x.double().view(n, heads, d), w, 1e-5), rot) if dims else \
            P.norm(x.double().view(n, heads, d), w, 1e-5)
        assert torch.allclose(q.cpu().double(), turn(a[:, :H * d], H, wq).reshape(n, -1), atol=1e-4)
        raw = a[:, H * d:(H + G) * d]
        rows = lambda c: torch.cat([c[1], c[0]], 1)[:, :n].transpose(0, 1).cpu()
        assert torch.allclose(rows(kc).double(), turn(raw, G, wk), atol=1e-4)
        assert torch.equal(rows(vc).reshape(n, -1), raw)
        assert torch.allclose(gate.cpu(), torch.sigmoid(a[:, (H + G) * d:]), atol=1e-6)


def test_the_gated_gelu_in_its_three_places():
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(2)
    for n, width, ff in ((300, 64, 96), (150, 256, 640), (8, 256, 512), (1, 128, 64), (64, 512, 1024), (700, 512, 2048)):
        h = torch.randn(n, width, generator=g).bfloat16()
        w = (torch.randn(2 * ff, width, generator=g) * 2 / width ** 0.5).bfloat16()
        z = h.double() @ w.double().T
        want = P.gelu_tanh(z[:, :ff]) * z[:, ff:]
        tol = dict(atol=2e-2, rtol=1e-2)
        for dtype in (torch.float32, torch.bfloat16):
            out = torch.empty(n, ff, dtype=dtype, device=DEV)
            ops.gelu_mul(z.float().to(DEV), out)
            assert torch.allclose(out.cpu().double(), want, **(dict(atol=1e-5, rtol=1e-5) if dtype == torch.float32 else tol))
        out = torch.full((n, ff), 9.0, dtype=torch.bfloat16, device=DEV)
        if ops.gemm_tc_takes(n, 2 * ff, width):
            ops.gemm_tc_gelu_gated(h.to(DEV), w.to(DEV), None, out)
            assert torch.allclose(out.cpu().double(), want, **tol), n
        if ops.gemv_takes(n, 2 * ff, width, ops.EPI_GATED, DEV):
            out.fill_(9.0)
            ops.gemv_bf16(w.to(DEV), None, out, ops.EPI_GATED, x=h.to(DEV), act=ops.GEMM_ACT_GELU_TANH)
            assert torch.allclose(out.cpu().double(), want, **tol), n
        ops.check_status(DEV)
    # far from zero: the gate's own value, or nothing
    big = torch.tensor([[-60.0, -9.0, 9.0, 60.0, 1.0, 1.0, 1.0, 1.0]], device=DEV)
    out = torch.empty(1, 4, device=DEV)
    ops.gelu_mul(big, out)
    assert torch.allclose(out.cpu(), torch.tensor([[0.0, 0.0, 9.0, 60.0]]), atol=1e-6)


# ---- the model ------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_each_configuration_alone(models, name, dtype, tmp_path):
    rng = random.Random(11)
    vocab = read_config(models[name])["vocab"]
    sequences, trace = {}, TraceBuilder()
    # the first tokens, a page's and a chunk's border, windows' edges
    for i, n in enumerate((1, 2, 3, 50, 63, 64, 65, 131, 300)):
        sequences[f"w{i}"] = random_tokens(rng, n, vocab)
        trace.step([(f"w{i}", sequences[f"w{i}"], range(n))], end=[f"w{i}"])
    toks = sequences["d"] = random_tokens(rng, 75, vocab)  # decoding from the second token on
    trace.step([("d", toks[:1], [0])])
    for t in range(1, 75):
        trace.step([("d", toks[t:t + 1], [0])], end=["d"] if t == 74 else [])
    replay_and_check(models, name, dtype, trace, sequences, tmp_path, "alone", beyond=0.02 if name == "sharp" else 0.0)


@pytest.mark.parametrize("name", ["mixed", "odd", "shared", "heads64"])
def test_the_stream_after_every_layer(models, name):
    """float32: the residual stream after each layer run, block by block."""
    from nnis_b200.engine import SequenceStep
    engine = engine_for(models, name, "float32")
    cfg = read_config(models[name])
    toks = random_tokens(random.Random(1), 90, cfg["vocab"])
    want = []
    P.forward(toks, load_weights(models[name], False), cfg, layers_out=want)
    got, saved = [], []
    for block in engine.model.blocks:
        saved.append((block, block.forward))

        def wrapped(hidden, ctx, cache, _f=block.forward):
            _f(hidden, ctx, cache)
            got.append(hidden.detach().cpu().clone())
        block.forward = wrapped
    try:
        slot = engine.acquire_slot()
        engine.step([SequenceStep(slot, toks, [89])])
        engine.release_slot(slot)
    finally:
        for block, f in saved:
            block.forward = f
    assert len(got) == len(want) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(got, want)):
        assert torch.allclose(a.double(), b, atol=1e-4 * float(b.abs().max())), i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "memories", "heads64"])
def test_whole_last_tokens_and_unequal_batches(models, name, dtype, tmp_path):
    vocab = read_config(models[name])["vocab"]
    trace, sequences = three_cuts(random.Random(3), vocab)
    replay_and_check(models, name, dtype, trace, sequences, tmp_path, "three cuts")


@pytest.mark.parametrize("name", ["mixed", "odd", "shared", "memories"])
def test_portions_batches_and_reuse_agree_with_each_request_alone(models, name):
    """float32: the same position's logits whatever the cut, the batch, the slot or the pages."""
    from nnis_b200.engine import SequenceStep
    engine = engine_for(models, name, "float32")
    vocab = read_config(models[name])["vocab"]
    rng = random.Random(9)
    prompts = [random_tokens(rng, n, vocab) for n in (200, 3, 67, 130)]
    alone = [run_whole(engine, p) for p in prompts]
    scale = max(float(np.abs(a).max()) for a in alone)
    for p, a in zip(prompts, alone):
        check_logits(a, plain_of(models[name], "float32", p), "float32", "alone")
    # portions of several sizes, down to two tokens and one
    for cuts in ([2, 2, 60, 1, 64, 71], [64, 64, 64, 8], [199, 1], [1, 199], [39, 2, 7, 152], [3, 17, 16, 164],
                 [1, 1, 1, 2, 130, 65], [2] * 100):
        slot = engine.acquire_slot()
        rows, at = [], 0
        for c in cuts:
            rows.append(engine.step([SequenceStep(slot, prompts[0][at:at + c], list(range(c)))]).cpu().numpy())
            at += c
        engine.release_slot(slot)
        assert at == 200 and np.abs(np.concatenate(rows) - alone[0]).max() < 5e-5 * scale, cuts
    # one batch of all four, then the same again in slots and pages that were used before
    for _ in range(2):
        slots = [engine.acquire_slot() for _ in prompts]
        heads = [max(1, len(p) - 20) for p in prompts]
        got = engine.step([SequenceStep(s, p[:h], list(range(h))) for s, p, h in zip(slots, prompts, heads)]).cpu().numpy()
        at = 0
        for i, h in enumerate(heads):
            assert np.abs(got[at:at + h] - alone[i][:h]).max() < 5e-5 * scale
            at += h
        live = list(range(len(prompts)))
        step = 0
        while live:  # decoded together; the shorter ones end earlier
            batch = [SequenceStep(slots[i], prompts[i][heads[i] + step:heads[i] + step + 1], [0]) for i in live]
            got = engine.step(batch).cpu().numpy()
            for r, i in enumerate(live):
                assert np.abs(got[r] - alone[i][heads[i] + step]).max() < 5e-5 * scale, (i, step)
            step += 1
            for i in list(live):
                if heads[i] + step == len(prompts[i]):
                    engine.release_slot(slots[i])
                    live.remove(i)
    assert engine.cache.usage()["slots_held"] == 0
    engine.cache.check()


def test_portions_of_one_sequence_beside_single_tokens_of_another(models):
    """A step in which one sequence brings many tokens and others one each: the prompt's kernels serve them all,
    at even and odd positions of every sequence."""
    from nnis_b200.engine import SequenceStep
    for name in ("mixed", "memories"):
        engine = engine_for(models, name, "float32")
        vocab = read_config(models[name])["vocab"]
        rng = random.Random(19)
        a, b, c = (random_tokens(rng, n, vocab) for n in (150, 40, 41))
        slots = [engine.acquire_slot() for _ in range(3)]
        rows, at = [], [0, 0, 0]
        for counts in ((1, 30, 1), (70, 1, 2), (1, 1, 33), (9, 1, 1), (68, 1, 1), (1, 6, 3)):
            got = engine.step([SequenceStep(s, t[p:p + n], list(range(n))) for s, t, p, n in
                               zip(slots, (a, b, c), at, counts)]).cpu().numpy()
            k = 0
            for i, (t, n) in enumerate(zip((a, b, c), counts)):
                rows += [(t, at[i] + j, got[k + j]) for j in range(n)]
                k += n
                at[i] += n
        for s in slots:
            engine.release_slot(s)
        assert at == [150, 40, 41]
        check_rows(models[name], "float32", rows, name)


def test_going_back_to_a_snapshot(models):
    """The state, the normaliser and the running maximum of even and of odd lengths come back."""
    from nnis_b200.engine import SequenceStep
    engine, vocab = engine_for(models, "shared", "float32"), 150
    rng = random.Random(23)
    base = random_tokens(rng, 71, vocab)
    for length in (70, 71):
        slot = engine.acquire_slot()
        engine.step([SequenceStep(slot, base[:length], [])])
        kept = engine.snapshot(slot)
        rows = []
        for other in (3, 40, 1):
            tail = random_tokens(rng, other, vocab)
            got = engine.step([SequenceStep(slot, tail, list(range(other)))]).cpu().numpy()
            rows += [(base[:length] + tail, length + j, got[j]) for j in range(other)]
            engine.restore(kept)
        engine.release_slot(slot)
        check_rows(models["shared"], "float32", rows, f"snapshot at {length}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_prompt_shape_that_recurs_is_captured_and_replayed(models, dtype):
    """A large prompt step whose shape comes a second time is recorded as a CUDA graph and replayed from
    the third time on.  Other tokens every time, the same shape."""
    from nnis_b200.engine import Engine, SequenceStep
    engine = Engine.from_dir(models["mixed"], dtype=dtype, max_tokens=64 * 64)
    rng = random.Random(77)
    graphs = []
    for round_ in range(4):
        a, b = random_tokens(rng, 300, 307), random_tokens(rng, 40, 307)
        slots = [engine.acquire_slot(), engine.acquire_slot()]
        got = engine.step([SequenceStep(slots[0], a[:290], [0, 150, 289]), SequenceStep(slots[1], b[:30], [29])]).cpu().numpy()
        more = engine.step([SequenceStep(slots[0], a[290:291], [0]), SequenceStep(slots[1], b[30:31], [0])]).cpu().numpy()
        for s_ in slots:
            engine.release_slot(s_)
        graphs.append(len(engine._step_graphs))
        rows = [(a, 0, got[0]), (a, 150, got[1]), (a, 289, got[2]), (b, 29, got[3]), (a, 290, more[0]), (b, 30, more[1])]
        check_rows(models["mixed"], dtype, rows, f"captured step, round {round_}")
    assert graphs == [0, 1, 1, 1], graphs


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "memories", "sharp"])
def test_long_decoding_lets_every_window_pass_over_decoded_tokens(models, name, dtype, tmp_path):
    vocab = read_config(models[name])["vocab"]
    toks = random_tokens(random.Random(21), 5 + 330, vocab)
    trace = TraceBuilder()
    trace.step([("a", toks[:5], [4])])
    for t in range(5, len(toks)):
        trace.step([("a", toks[t:t + 1], [0])], end=["a"] if t == len(toks) - 1 else [])
    replay_and_check(models, name, dtype, trace, {"a": toks}, tmp_path, "long decoding", beyond=0.02 if name == "sharp" else 0.0)


def _sharpen(model_dir, out_dir, query_pos, key_pos, tokens, cfg):
    """A copy of the model whose first layer has, in every head, one score that stands out: the query at
    ``query_pos`` against the key at ``key_pos``.  One row of W_q (a value that is not turned) lies along
    the normed embedding of the query's token, one of the keys' along the key's token's."""
    from safetensors.torch import load_file, save_file
    os.makedirs(out_dir, exist_ok=True)
    w = load_file(os.path.join(model_dir, "model.safetensors"))
    plain = {k: v.double() for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    h = P.norm(P.norm(plain["embed"][tokens], plain["embed.norm"], eps), plain["l0.norm1"], eps)
    centred = h - h.mean(0)  # (what all tokens share points every key the same way)
    hq, hk = (centred[t] / centred[t].norm() for t in (query_pos, key_pos))
    m = cfg["layers"][0]["mixer"]
    d = m["dim"]
    q = plain["l0.mix.q"].clone()
    if cfg["layers"][0]["type"] == "attention":
        k = plain["l0.mix.k"].clone()
        for a in range(m["heads"]):
            q[a * d + d - 1] = hq * 0.5
        for a in range(m["kv_heads"]):
            k[a * d + d - 1] = hk * 0.5
        w["l0.mix.k"] = k.to(torch.bfloat16)
        for name in ("l0.mix.q.norm", "l0.mix.k.norm"):
            w[name] = torch.full((d,), 0.4, dtype=torch.bfloat16)
            w[name][-1] = 1.2
    else:
        down, uk = plain["l0.mix.dkv"].clone(), plain["l0.mix.uk"].clone()
        down[0] = hk
        for a in range(m["heads"]):
            q[a * (d + m["rot_dim"]) + d - 1] = hq * 8.0
            uk[a * d + d - 1] = 0.0
            uk[a * d + d - 1, 0] = 1.0
        w["l0.mix.dkv"], w["l0.mix.uk"] = down.to(torch.bfloat16), uk.to(torch.bfloat16)
    w["l0.mix.q"] = q.to(torch.bfloat16)
    save_file(w, os.path.join(out_dir, "model.safetensors"))
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(cfg, f)
    return out_dir


def _edge(tmp_path, first, kp, qp, n, visible, seed, what):
    """The query at ``qp`` against the key at ``kp`` in a first layer made sharp there (the second layer sees one
    token only): against the plain implementation whole, decoded alone, and with portions that start at the
    query, after the key and at the key; and changing the key's token changes the query's logits if and
    only if the key is visible."""
    from nnis_b200.engine import Engine, SequenceStep
    cfg = config(97, 256, 1e-5, [(first, dense(48)), (attention(2, 1, 8, 1, 0.5), None)])
    base = make_model(str(tmp_path / "base"), cfg, seed)
    rng = random.Random(seed * 1000 + kp)
    toks = [rng.randrange(2, 97) for _ in range(n)]
    toks[kp], toks[qp] = 0, 1  # tokens that appear nowhere else
    d = _sharpen(base, str(tmp_path / "sharp"), qp, kp, toks, cfg)
    w = load_weights(d, False)
    probe = {}
    want = P.forward(toks, w, cfg, probe=probe)
    a = probe["weights"][0]  # layer 0, head 0
    if visible:
        assert float(a[qp, kp]) > 0.5, float(a[qp, kp])  # the key stands out
    else:
        assert float(a[qp, kp]) == 0.0
    other = list(toks)
    other[kp] = 50
    moved = float((P.forward(other, w, cfg)[qp] - want[qp]).abs().max())
    assert (moved > 1e-3) == visible, (moved, what)
    for dtype in DTYPES:
        engine = Engine.from_dir(d, dtype=dtype, max_tokens=1024)
        rows = []
        for cut in sorted({n, qp, qp - 1, kp + 1, kp} - {0}):
            slot = engine.acquire_slot()
            if cut == n:
                got = engine.step([SequenceStep(slot, toks, [qp, n - 1])]).cpu().numpy()
                rows += [(toks, qp, got[0]), (toks, n - 1, got[1])]
            else:
                engine.step([SequenceStep(slot, toks[:cut], [])])
                if cut == qp:
                    got = engine.step([SequenceStep(slot, toks[qp:qp + 1], [0])]).cpu().numpy()
                    rows.append((toks, qp, got[0]))
                    got = engine.step([SequenceStep(slot, toks[qp + 1:], [n - qp - 2])]).cpu().numpy()
                    rows.append((toks, n - 1, got[0]))
                else:
                    got = engine.step([SequenceStep(slot, toks[cut:], [qp - cut, n - 1 - cut])]).cpu().numpy()
                    rows += [(toks, qp, got[0]), (toks, n - 1, got[1])]
            engine.release_slot(slot)
        check_rows(d, dtype, rows, f"{what} {dtype}")
        if dtype == "float32":
            slot = engine.acquire_slot()
            changed = engine.step([SequenceStep(slot, other, [qp])]).cpu().numpy()
            engine.release_slot(slot)
            assert (float(np.abs(changed[0] - want[qp].numpy()).max()) > 1e-3) == visible


@pytest.mark.parametrize("window, distance", [(40, 39), (40, 40), (64, 63), (64, 64), (65, 64), (65, 65), (129, 128),
                                              (129, 129), (250, 249), (7, 6), (7, 7), (1, 1), (2, 1), (2, 2)])
@pytest.mark.parametrize("dim", [16, 64])
def test_a_key_just_inside_and_just_outside_the_window(window, distance, dim, tmp_path):
    n = 270
    qp = n - 3
    _edge(tmp_path, attention(4, 2, dim, window, {16: 0.75, 64: 0.375}[dim], 100.0, dim // 2), qp - distance, qp, n, distance < window, 31,
          f"window {window} distance {distance}")


@pytest.mark.parametrize("key, query", [(0, 267), (1, 267), (63, 200), (64, 128), (127, 128), (128, 192), (3, 64), (191, 267)])
def test_a_key_far_back_in_the_latents(key, query, tmp_path):
    """At the first tokens, at page borders and across several pages; every key stays visible."""
    _edge(tmp_path, latent(4, 16, 8, 24, 16, 0.5, 100.0, (4.0, 64, 8.0, 1.0)), key, query, 270, True, 43, f"key {key} query {query}")


def test_a_sink_that_takes_nearly_everything_and_one_that_takes_nothing(tmp_path):
    """Very large and very small sinks, per head: in prompts, portions, single tokens and slices."""
    from nnis_b200.engine import Engine, SequenceStep
    from safetensors.torch import load_file, save_file
    cfg = config(83, 64, 1e-5, [(latent(4, 16, 8, 24, 32, 0.3, 100.0), dense(40))])
    d = make_model(str(tmp_path / "m"), cfg, 5)
    w = load_file(os.path.join(d, "model.safetensors"))
    w["l0.mix.sink"] = torch.tensor([9.0, -90.0, 3.5, 60.0], dtype=torch.bfloat16)
    save_file(w, os.path.join(d, "model.safetensors"))
    toks = random_tokens(random.Random(2), 230, 83)
    probe = {}
    P.forward(toks, load_weights(d, False), cfg, probe=probe)
    sums = [float(a[225].sum()) for a in probe["weights"]]
    assert sums[0] < 0.5 and abs(sums[1] - 1) < 1e-12 and sums[3] < 1e-12, sums
    for dtype in DTYPES:
        engine = Engine.from_dir(d, dtype=dtype, max_tokens=1024)
        slot = engine.acquire_slot()
        got = [engine.step([SequenceStep(slot, toks[:150], list(range(150)))]).cpu().numpy(),
               engine.step([SequenceStep(slot, toks[150:220], list(range(70)))]).cpu().numpy()]
        got += [engine.step([SequenceStep(slot, toks[t:t + 1], [0])]).cpu().numpy() for t in range(220, 230)]
        engine.release_slot(slot)
        got = np.concatenate(got)
        check_rows(d, dtype, [(toks, i, got[i]) for i in range(230)], f"sinks {dtype}")


def test_far_keys_and_page_borders_with_sharp_attention(models):
    """Random sharp heads put most of a query's weight on single keys anywhere in their windows: prompts
    that end on both sides of page borders, portions that start there, and tokens decoded across them."""
    from nnis_b200.engine import SequenceStep
    vocab = read_config(models["sharp"])["vocab"]
    probe = {}
    toks = random_tokens(random.Random(5), 450, vocab)
    P.forward(toks, load_weights(models["sharp"], False), read_config(models["sharp"]), probe=probe)
    peak = torch.stack([m.max(-1).values for m in probe["weights"]])[:, 100:]
    assert float(peak.mean()) > 0.3  # sharp: much of a query's weight on one key, on average
    far = torch.stack([(m.argmax(-1) - torch.arange(450)).abs() for m in probe["weights"]])
    assert int(far.max()) > 250      # and some of those keys lie far back
    for dtype in DTYPES:
        engine = engine_for(models, "sharp", dtype)
        for cuts in ([450], [63, 1, 64, 1, 127, 194], [64, 64, 64, 64, 64, 64, 66], [128, 1, 1, 1, 62, 257], [300, 150]):
            slot = engine.acquire_slot()
            rows, at = [], 0
            for c in cuts:
                got = engine.step([SequenceStep(slot, toks[at:at + c], list(range(c)))]).cpu().numpy()
                rows += [(toks, at + i, got[i]) for i in range(c)]
                at += c
            engine.release_slot(slot)
            check_rows(models["sharp"], dtype, rows, f"sharp {dtype} {cuts}", beyond=0.02)


def _random_config(rng, middle=False):
    """``middle``: sizes of a small real model, at which the tensor-core products, the decode projections over
    tiles of rows and the tensor-core attention take over from the any-size kernels.  (Nothing that is normed
    has only one or two values: their norm is a sign.)"""
    pick = rng.choice
    width = pick([192, 256, 384, 512]) if middle else pick([40, 64, 76, 96, 128])
    layers = []
    for i in range(rng.randint(2, 4) if middle else rng.randint(1, 5)):
        if i and rng.random() < 0.25:
            layers.append(rng.randrange(i))
            continue
        mlp = None if rng.random() < 0.25 else dense(pick([256, 512, 640]) if middle else pick([6, 8, 12, 33, 64]))
        kind = rng.randrange(3)
        if kind == 0:
            kv = pick([1, 2, 4]) if middle else rng.randint(1, 3)
            dim = pick([32, 64, 80, 128]) if middle else pick([5, 6, 8, 16, 24, 40, 64, 130])
            dims = pick([0, dim // 2 * 2, dim // 4 * 2])
            mixer = attention(kv * rng.randint(1, 4), kv, dim, pick([1, 2, 17, 63, 64, 65, 100, 1000]),
                              pick([0.2, 0.5, 1.0]) / math.sqrt(dim), pick([10.0, 10000.0, 500000.0]), dims)
        elif kind == 1:
            dim = pick([32, 64]) if middle else pick([1, 5, 8, 16, 24, 40])
            rot = dim // 2 if middle else pick([0, 2, 4, 8, 16])
            scaling = (pick([1.0, 2.0, 16.0]), pick([20, 100, 4096]), pick([4.0, 32.0]), pick([0.5, 1.0, 3.0])) \
                if rng.random() < 0.7 else None
            mixer = latent(pick([4, 8, 16]) if middle else rng.randint(1, 6), dim, rot,
                           pick([32, 64]) if middle else pick([1, 4, 8, 13, 24, 64]),
                           pick([64, 128, 256]) if middle else pick([6, 10, 16, 24, 48, 130]),
                           pick([0.2, 0.5, 1.0]) / math.sqrt(dim + rot), pick([10.0, 10000.0, 500000.0]), scaling)
        else:
            mixer = memory(pick([2, 4, 8]) if middle else rng.randint(1, 6), pick([32, 64, 128]) if middle else
                           pick([1, 3, 8, 17, 40, 68]), pick([64, 128, 256]) if middle else pick([4, 6, 9, 32, 65, 100]),
                           pick([0.7, 4.0, 15.0, 30.0]))
        layers.append((mixer, mlp))
    return config(pick([1000, 2048, 4099]) if middle else pick([50, 131, 256, 577]), width, pick([1e-5, 1e-6]), layers)


@pytest.mark.parametrize("trial", range(16))
def test_configurations_drawn_at_random(trial, tmp_path):
    """A prompt in one step, a second portion and six tokens one by one, both dtypes, on a model
    whose sizes, layer order, sharing and constants are drawn at random: whatever kernels the sizes select."""
    from nnis_b200.engine import Engine, SequenceStep
    rng = random.Random(7100 + trial)
    cfg = _random_config(rng)
    d = make_model(str(tmp_path / "m"), cfg, seed=trial)
    toks = random_tokens(rng, 150, cfg["vocab"])
    for dtype in DTYPES:
        engine = Engine.from_dir(d, dtype=dtype, max_tokens=4096)
        slot = engine.acquire_slot()
        got = [engine.step([SequenceStep(slot, toks[:101], list(range(101)))]).cpu().numpy(),
               engine.step([SequenceStep(slot, toks[101:144], list(range(43)))]).cpu().numpy()]
        for t in range(144, 150):
            got.append(engine.step([SequenceStep(slot, toks[t:t + 1], [0])]).cpu().numpy())
        engine.release_slot(slot)
        engine.check_status()
        got = np.concatenate(got)
        check_rows(d, dtype, [(toks, i, got[i]) for i in range(150)], f"random configuration {trial} {dtype}: {json.dumps(cfg)}",
                   beyond=0.02)


@pytest.mark.parametrize("trial", range(8))
def test_middle_sizes_drawn_at_random(trial, tmp_path):
    """A batch of two prompts (one of them in two portions) and eight tokens decoded together, both
    dtypes, at sizes of a small real model."""
    from nnis_b200.engine import Engine, SequenceStep
    rng = random.Random(8200 + trial)
    cfg = _random_config(rng, middle=True)
    d = make_model(str(tmp_path / "m"), cfg, seed=40 + trial)
    a, b = random_tokens(rng, 208, cfg["vocab"]), random_tokens(rng, 77, cfg["vocab"])
    for dtype in DTYPES:
        engine = Engine.from_dir(d, dtype=dtype, max_tokens=2048)
        sa, sb = engine.acquire_slot(), engine.acquire_slot()
        rows = []  # (request's tokens, position, logits row)
        got = engine.step([SequenceStep(sa, a[:130], list(range(0, 130, 5))), SequenceStep(sb, b[:69], [0, 68])]).cpu().numpy()
        rows += [(a, 5 * i, got[i]) for i in range(26)] + [(b, 0, got[26]), (b, 68, got[27])]
        got = engine.step([SequenceStep(sa, a[130:200], [0, 69])]).cpu().numpy()
        rows += [(a, 130, got[0]), (a, 199, got[1])]
        for t in range(8):
            got = engine.step([SequenceStep(sa, a[200 + t:201 + t], [0]), SequenceStep(sb, b[69 + t:70 + t], [0])]).cpu().numpy()
            rows += [(a, 200 + t, got[0]), (b, 69 + t, got[1])]
        engine.release_slot(sa)
        engine.release_slot(sb)
        engine.check_status()
        check_rows(d, dtype, rows, f"middle size {trial} {dtype}: {json.dumps(cfg)}", beyond=0.02)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_point(models, dtype):
    from nnis_b200 import LLM
    d = models["mixed"]
    cfg = read_config(d)
    bf = dtype == "bfloat16"
    w = load_weights(d, bf)
    llm = LLM(d, dtype=dtype, max_tokens=64 * 32, max_batch=3)
    rng = random.Random(17)
    prompts = [[5, 9, 1, 200, 33], [7], random_tokens(rng, 160, 307), [250, 3], random_tokens(rng, 135, 307)]
    results = llm.generate(prompts, max_new_tokens=10, stop_token_ids=())
    for p, r in zip(prompts, results):
        assert r.ok and r.finish_reason == "length"
        if not bf:
            assert r.token_ids == P.greedy_generate(cfg, w, p, 10), (dtype, p)
        else:  # a bfloat16 near-tie may go either way: every pick is nearly the best
            logits = P.forward(p + r.token_ids, w, cfg, emulate_bf16=True)
            for i, t in enumerate(r.token_ids):
                row = logits[len(p) + i - 1]
                assert float(row.max() - row[t]) <= 0.05 * max(1.0, float(row.abs().max())), (p, i)
    # a session goes on from where generation left it
    from nnis_b200 import GenerationConfig
    session = llm.new_session()
    ids = session.generate(prompts[0], GenerationConfig(6))
    more = session.decode_one(17)
    if not bf:
        want = P.forward(prompts[0] + ids + [17], w, cfg)[-1]
        check_logits(np.asarray(more).reshape(1, -1), want[None, :], dtype, "session")
    assert llm.engine.cache.usage()["slots_held"] <= 1


def test_greedy_generation_over_pages_that_go_back(models):
    """200 tokens decoded as captured steps, float32: windows pass over decoded pages, which go back to the
    pools, and the memory is carried from step to step."""
    from nnis_b200 import LLM
    for name, vocab in (("mixed", 307), ("memories", 131)):
        d = models[name]
        llm = LLM(d, dtype="float32", max_tokens=64 * 20, max_batch=2)
        prompts = [random_tokens(random.Random(3), 20, vocab), random_tokens(random.Random(4), 90, vocab)]
        results = llm.generate(prompts, max_new_tokens=200, stop_token_ids=())
        w, cfg = load_weights(d, False), read_config(d)
        for p, r in zip(prompts, results):
            logits = P.forward(p + r.token_ids, w, cfg)
            for i, t in enumerate(r.token_ids):
                row = logits[len(p) + i - 1]
                assert float(row.max() - row[t]) <= 1e-4 * float(row.abs().max()), i


def test_sampled_generation_and_the_command_line(models):
    """Sampling with a seed repeats itself, and the command line's generate runs the design."""
    import sys
    from nnis_b200 import LLM
    from nnis_b200.sampling import SamplingConfig
    llm = LLM(models["odd"], dtype="bfloat16", max_tokens=2048, max_batch=2)
    policy = SamplingConfig.seeded(5).with_temperature(0.9).with_top_k(40)
    a = llm.generate([[1, 2, 3], [9, 8]], max_new_tokens=12, sampling=policy, stop_token_ids=())
    b = llm.generate([[1, 2, 3], [9, 8]], max_new_tokens=12, sampling=policy, stop_token_ids=())
    assert [r.token_ids for r in a] == [r.token_ids for r in b] and all(len(r.token_ids) == 12 for r in a)
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "nnis"), "generate", "--model", models["shared"],
                        "--prompt-ids", "4,5,6", "--max-new-tokens", "5", "--dtype", "float32"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    want = P.greedy_generate(read_config(models["shared"]), load_weights(models["shared"], False), [4, 5, 6], 5)
    assert r.stdout.split() == [str(t) for t in want]


def test_replay_program_runs_a_model_folder(models, tmp_path):
    cfg = read_config(models["shared"])
    toks = random_tokens(random.Random(4), 40, cfg["vocab"])
    trace = TraceBuilder()
    trace.step([("a", toks[:30], [0, 29]), ("b", toks[:7], [6])])
    trace.step([("a", toks[30:31], [0]), ("b", toks[7:8], [0])], end=["b"])
    trace.step([("a", toks[31:32], [])], end=["a"])
    out = str(tmp_path / "out")
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", models["shared"], "--dtype", "float32",
                        "--out", out, "--max-tokens", "256"], input="\n".join(trace.lines) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not os.path.exists(os.path.join(out, "2.f32"))
    want = plain_of(models["shared"], "float32", toks)
    check_logits(read_step(out, 0, cfg["vocab"]), torch.stack([want[0], want[29], want[6]]), "float32", "program")
    check_logits(read_step(out, 1, cfg["vocab"]), torch.stack([want[30], want[7]]), "float32", "program")
