"""Setenex on the GPU against the plain implementation: the new kernels against float64 torch, every
mechanism alone, whole prompts against token-by-token decoding, portions down to two tokens, unequal
batches against each request alone, slots and pages used again, keys far away, at page borders and on
both sides of every window's edge and of the kept first tokens with attention made sharp, long decoding,
other sizes, greedy generation through the Python entry point, and the replay program."""
import json
import math
import os
import random
import subprocess

import numpy as np
import pytest
import torch

import plain_setenex as P
from helpers import BF16_REL_TO_MAX, TraceBuilder, check_logits, random_tokens, read_step, three_cuts
from setenex_models import CONFIGS, attention, config, latent, load_weights, make_model, moe, read_config

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]
F = torch.float64
# a router's choice between two experts whose corrected scores lie closer than this may go either way
# in bfloat16; such positions are left out, and they must be a minority
CLOSE_CALL = 0.01


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return {name: make_model(str(tmp_path_factory.mktemp(f"setenex_{name}")), cfg, seed=700 + i)
            for i, (name, cfg) in enumerate(CONFIGS.items())}


_engines, _plain = {}, {}


def engine_for(models, name, dtype):
    from nnis_b200.engine import Engine
    if (name, dtype) not in _engines:
        _engines[(name, dtype)] = Engine.from_dir(models[name], dtype=dtype, max_tokens=64 * 96)
    return _engines[(name, dtype)]


def plain_of(model_dir, dtype, tokens):
    """(logits, smallest gap of any router's choice at each position)"""
    key = (model_dir, dtype, tuple(tokens))
    if key not in _plain:
        bf = dtype == "bfloat16"
        probe = {}
        logits = P.forward(list(tokens), load_weights(model_dir, bf), read_config(model_dir), emulate_bf16=bf, probe=probe)
        gaps = torch.stack(probe["gaps"]).min(0).values if probe.get("gaps") else torch.full((len(tokens),), math.inf)
        _plain[key] = (logits, gaps)
    return _plain[key]


def check_rows(model_dir, dtype, rows, what, beyond=0.0):
    """rows: (tokens of the request, position, logits row).  bfloat16 rows at a router's close call are
    left out (at most two fifths of them).  ``beyond``: the part of the bfloat16 rows that may lie outside the
    bound, up to three times it (where sharp attention carries one rounding far)."""
    keep, skipped = [], 0
    for toks, pos, row in rows:
        logits, gaps = plain_of(model_dir, dtype, toks)
        if dtype == "bfloat16" and float(gaps[pos]) < CLOSE_CALL:
            skipped += 1
            continue
        keep.append((row, logits[pos]))
    assert skipped <= max(2, 2 * len(rows) // 5), f"{what}: {skipped} of {len(rows)} rows at a close call"
    if keep:
        got, want = np.stack([r for r, _ in keep]), torch.stack([w for _, w in keep])
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


# ---- the new kernels against plain torch -------------------------------------------------------
DEV = torch.device("cuda:0")


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def test_embedding_times_a_number():
    from nnis_b200.csrc import ops
    table = torch.randn(50, 24)
    for dtype in (torch.float32, torch.bfloat16):
        hidden = torch.empty(3, 24, device=DEV)
        status = torch.zeros(1, dtype=torch.int32, device=DEV)
        ops.embed(table.to(dtype).to(DEV), i32([4, 9, 49]), hidden, status, 17.5)
        assert torch.equal(hidden.cpu(), table.to(dtype).float()[[4, 9, 49]] * 17.5) and int(status[0]) == 0


@pytest.mark.parametrize("outputs, top, groups, keep", [(8, 2, 2, 1), (12, 4, 3, 2), (16, 5, 4, 3), (6, 2, 1, 1), (9, 3, 9, 5),
                                                        (70, 6, 10, 4), (4, 4, 2, 2), (3, 1, 1, 1)])
def test_the_router_with_sigmoid_scores_and_groups_ranked_by_two(outputs, top, groups, keep):
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(outputs)
    for n, width in ((150, 76), (5, 64)):  # (several tokens a CTA, and one)
        h = torch.randn(n, width, generator=g)
        w = {"r.router": torch.randn(outputs, width, generator=g) * 0.2,
             "r.correction": torch.rand(outputs, generator=g) * 0.6 - 0.9}  # choice scores of either sign
        r = {"experts": outputs, "top": top, "groups": {"count": groups, "keep": keep}}
        probe = {}
        ids, weights = P.route(h.double(), {k: v.double() for k, v in w.items()}, "r", r, probe)
        pos = torch.arange(n, dtype=torch.int32)
        pos[3] = -1  # a padding row
        got_ids = torch.full((n, top), 99, dtype=torch.int32, device=DEV)
        got_w, passed = torch.empty(n, top, device=DEV), torch.empty(n, device=DEV)
        ops.moe_route_choice(h.to(DEV), w["r.router"].to(DEV), w["r.correction"].to(DEV), pos.to(DEV), got_ids, got_w,
                             passed, outputs, top, groups, keep, sigmoid_scores=True, group_top=2, renormalise=True)
        got_ids, got_w = got_ids.cpu(), got_w.cpu()
        assert (got_ids[3] == -1).all() and (passed == 0).all()
        clear = [t for t in range(n) if t != 3 and float(probe["gaps"][0][t]) > 1e-5]
        assert len(clear) > 0.9 * n - 2
        for t in clear:
            assert got_ids[t].tolist() == ids[t].tolist(), t
            assert torch.allclose(got_w[t].double(), weights[t], atol=1e-6) and abs(float(got_w[t].sum()) - 1) < 1e-5


def test_plain_gelu_experts_by_pairs_sorted_and_on_tcgen05():
    """The three ways of running the chosen experts against float64: a product per pair (both dtypes),
    sorted pairs on mma.sync tiles, sorted pairs on the tcgen05 kernel."""
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(6)
    for n, width, ff, E, top in ((300, 72, 40, 5, 2), (40, 128, 64, 4, 3), (700, 64, 136, 3, 1), (7, 76, 20, 6, 2)):
        h = torch.randn(n, width, generator=g)
        up, down = torch.randn(E, ff, width, generator=g) / width ** 0.5, torch.randn(E, width, ff, generator=g) / ff ** 0.5
        ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(n)]).int()
        weights = torch.rand(n, top, generator=g)
        base = torch.randn(n, width, generator=g)
        pos = torch.arange(n, dtype=torch.int32, device=DEV)
        for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2)):
            hd, u, d = h.to(dtype), up.to(dtype), down.to(dtype)
            want = base.double().clone()
            for t in range(n):
                for e, s in zip(ids[t].tolist(), weights[t]):
                    a = P.gelu(hd[t].double() @ u[e].double().T)
                    want[t] += float(s) * ((a.to(dtype) if dtype == torch.bfloat16 else a).double() @ d[e].double().T)
            act = torch.empty(n * top * ff, dtype=dtype, device=DEV)
            res = base.to(DEV).clone()
            ops.moe_experts(hd.to(DEV), u.to(DEV), d.to(DEV), ids.to(DEV), weights.to(DEV), pos, act, res, top,
                            ops.GEMM_ACT_GELU_ERF)
            assert torch.allclose(res.cpu().double(), want, atol=tol, rtol=tol), (n, dtype)
            if dtype == torch.bfloat16 and ops.moe_grouped_takes(width, ff, E):
                tiles = ops.moe_grouped_tiles(n * top, E)
                scratch = lambda shape, t: torch.empty(shape, dtype=t, device=DEV)
                res = base.to(DEV).clone()
                ops.moe_grouped(hd.to(DEV), u.to(DEV), d.to(DEV), ids.to(DEV), weights.to(DEV), scratch(tiles * 64, torch.int32),
                                scratch(n * top, torch.int32), scratch(tiles, torch.int32), scratch((tiles * 64, ff), dtype),
                                scratch((tiles * 64, width), torch.float32), res, top, ops.GEMM_ACT_GELU_ERF)
                assert torch.allclose(res.cpu().double(), want, atol=tol, rtol=tol), (n, "sorted")
                tiles = ops.moe_grouped_tc_tiles(n * top, E)
                res = base.to(DEV).clone()
                ops.moe_grouped_tc(hd.to(DEV), u.to(DEV), d.to(DEV), ids.to(DEV), weights.to(DEV),
                                   scratch(tiles * 128, torch.int32), scratch(n * top, torch.int32), scratch(tiles, torch.int32),
                                   scratch((tiles * 128, width), dtype), scratch((tiles * 128, ff), dtype),
                                   scratch((tiles * 128, width), torch.float32), res, top, ops.GEMM_ACT_GELU_ERF)
                assert torch.allclose(res.cpu().double(), want, atol=tol, rtol=tol), (n, "tcgen05")
                ops.check_status(DEV)


def _plain_attention(q, k, v, window, keep, scale, bias, gate=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv], bias [H, distances]; float64."""
    T, H = q.shape[:2]
    i = torch.arange(T)
    back = i[:, None] - i[None, :]
    visible = (back >= 0) & ((back < window) | (i[None, :] < keep) if window else back >= 0)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for a in range(H):
        g = a // (H // k.shape[1])
        s = (q[:, a] @ k[:, g].T) * scale
        if bias is not None:
            s = s + bias[a][back.clamp(0, bias.shape[1] - 1)]
        out[:, a] = torch.softmax(s.masked_fill(~visible, -math.inf), -1) @ v[:, g]
    out = out.reshape(T, -1)
    return out if gate is None else out * gate.repeat_interleave(v.shape[-1], 1)


ATTENTION_CASES = [(4, 2, 16, 24, 9, 3, 20), (6, 3, 24, 40, 50, 70, 90), (3, 3, 11, 34, 64, 64, 1), (5, 1, 18, 6, 1, 2, 40),
                   (8, 1, 12, 40, 70, 0, 15), (2, 1, 64, 128, 0, 0, 33), (8, 2, 32, 128, 65, 1, 300), (6, 1, 10, 8, 130, 130, 7),
                   (7, 1, 40, 200, 20, 100, 50)]


@pytest.mark.parametrize("H, G, dk, dv, window, keep, distances", ATTENTION_CASES)
def test_attention_with_a_distance_bias_and_kept_tokens_in_every_cut(H, G, dk, dv, window, keep, distances):
    """The any-size kernel over a cache whose pages are scattered: a prompt, a later portion and single
    tokens, with the key range whole and in slices; pages that nothing may read hold other numbers, and the
    table entries of pages that have been given back are -1."""
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 100 + dk)
    S, page, scale = 260, 64, 1.3 / math.sqrt(dk)
    bias = torch.randn(H, distances, generator=g)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        q, k = torch.randn(S, H, dk, generator=g).to(dtype), torch.randn(S, G, dk, generator=g).to(dtype)
        v = torch.randn(S, G, dv, generator=g).to(dtype)
        pages = [5, 2, 9, 0, 7]
        k_cache = torch.full((10, G, page, dk), 50.0, dtype=dtype)
        v_cache = torch.full((10, G, page, dv), -50.0, dtype=dtype)
        for t in range(S):
            k_cache[pages[t // page], :, t % page] = k[t]
            v_cache[pages[t // page], :, t % page] = v[t]
        want = _plain_attention(q.double(), k.double(), v.double(), window, keep, scale, bias.double())
        for a, b, splits in ((0, 130, 1), (130, 190, 1), (190, 191, 1), (191, 192, 3), (192, 200, 2), (0, 200, 4),
                             (255, 260, 5), (259, 260, 1)):
            n = b - a
            held = [p if not window or (i + 1) * page > a - window + 1 or i * page < keep else -1
                    for i, p in enumerate(pages)]
            table = i32([[3] * 5, held])  # the sequence is row 1 of the batch
            out = torch.full((n, H * dv), 9.0, dtype=dtype, device=DEV)
            partial = torch.empty(n * H * splits * (dv + 2), device=DEV) if splits > 1 else None
            ops.attention_sink(q[a:b].reshape(n, -1).to(DEV), k_cache.to(DEV), v_cache.to(DEV), i32(list(range(a, b))),
                               torch.ones(n, dtype=torch.int32, device=DEV), table, None, None, out, H, G, window, 0,
                               scale, 0.0, splits, partial, keep, bias.to(DEV))
            assert torch.allclose(out.cpu().double(), want[a:b], atol=tol, rtol=tol), (dtype, a, b, splits)
        # without a bias, and a padding row that is left alone
        other = _plain_attention(q.double(), k.double(), v.double(), window, keep, scale, None)
        out = torch.full((3, H * dv), 9.0, dtype=dtype, device=DEV)
        ops.attention_sink(q[[150, 0, 151]].reshape(3, -1).to(DEV), k_cache.to(DEV), v_cache.to(DEV), i32([150, -1, 151]),
                           torch.ones(3, dtype=torch.int32, device=DEV), i32([[3] * 5, pages]), None, None, out, H, G,
                           window, 0, scale, 0.0, 1, None, keep, None)
        assert (out[1] == 9.0).all()
        assert torch.allclose(out[[0, 2]].cpu().double(), other[[150, 151]], atol=tol, rtol=tol)


@pytest.mark.parametrize("H, G, dk, dv, window, keep, distances, gated", [
    (4, 2, 64, 64, 100, 3, 90, False), (2, 1, 128, 128, 70, 65, 33, False), (6, 2, 48, 48, 33, 64, 200, True),
    (3, 3, 64, 128, 64, 0, 17, False), (2, 1, 128, 40, 129, 130, 128, False), (4, 1, 8, 16, 1, 1, 5, True),
    (4, 4, 72, 96, 65, 20, 1, False), (2, 2, 24, 104, 0, 0, 60, False), (2, 1, 64, 64, 20, 300, 64, False)])
def test_prompt_attention_on_the_tensor_cores(H, G, dk, dv, window, keep, distances, gated):
    """The tensor-core prompt form against plain float64 and against the any-size kernel: two sequences in
    one step, one of them a later portion that starts inside a page (the pages between the kept ones and its
    window given back), tiles that end inside a page; padded and whole heads."""
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 1000 + dk + dv)
    scale = 1.2 / math.sqrt(dk)
    bias = torch.randn(H, distances, generator=g)
    lens, starts = [230, 420], [0, 275]
    counts = [n - s for n, s in zip(lens, starts)]
    pages = [[3, 0, 6, 1], [2, 7, 5, 9, 4, 10, 8]]
    k_cache = torch.full((12, G, 64, dk), 50.0, dtype=torch.bfloat16)
    v_cache = torch.full((12, G, 64, dv), -50.0, dtype=torch.bfloat16)
    qs, want, gates = [], {True: [], False: []}, []
    for i, n in enumerate(lens):
        q, k = torch.randn(n, H, dk, generator=g).bfloat16(), torch.randn(n, G, dk, generator=g).bfloat16()
        v = torch.randn(n, G, dv, generator=g).bfloat16()
        gate = torch.rand(n, H, generator=g)
        for t in range(n):
            k_cache[pages[i][t // 64], :, t % 64] = k[t]
            v_cache[pages[i][t // 64], :, t % 64] = v[t]
        for with_bias in (True, False):
            full = _plain_attention(q.double(), k.double(), v.double(), window, keep, scale,
                                    bias.double() if with_bias else None, gate.double() if gated else None)
            want[with_bias].append(full[starts[i]:])
        qs.append(q[starts[i]:].reshape(counts[i], -1))
        gates.append(gate[starts[i]:])
    q, gate = torch.cat(qs).to(DEV), torch.cat(gates).to(DEV) if gated else None
    held = [p if not window or (j + 1) * 64 > starts[1] - window + 1 or j * 64 < keep else -1 for j, p in enumerate(pages[1])]
    table = i32([pages[0] + [-1] * 3, held])
    tiles = i32([(i, q0) for i, c in enumerate(counts) for q0 in range(0, c, 64)])
    pos = i32(list(range(lens[0])) + list(range(starts[1], lens[1])))
    seq = i32([0] * counts[0] + [1] * counts[1])
    assert ops.attention_sink_mma_takes(dk, dv, 64) and not ops.attention_sink_mma_takes(dk + 1, dv, 64)
    for with_bias in (True, False):
        b = bias.to(DEV) if with_bias else None
        out = torch.full((sum(counts), H * dv), 9.0, dtype=torch.bfloat16, device=DEV)
        ops.attention_sink_mma(q, k_cache.to(DEV), v_cache.to(DEV), tiles, i32([0, counts[0]]), i32(starts), i32(counts),
                               table, None, gate, out, H, G, window, 0, scale, 0.0, keep, b)
        assert torch.allclose(out.cpu().double(), torch.cat(want[with_bias]), atol=3e-2, rtol=3e-2), with_bias
        other = torch.empty_like(out)
        ops.attention_sink(q, k_cache.to(DEV), v_cache.to(DEV), pos, seq, table, None, gate, other, H, G, window, 0, scale,
                           0.0, 1, None, keep, b)
        assert torch.allclose(out.float(), other.float(), atol=3e-2, rtol=3e-2), with_bias


def test_head_norms_with_weights_before_the_cache():
    """qkv_prep with a weight per value of a head: q and k heads normed by themselves, before a rotation if
    there is one, values as they are."""
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(8)
    for H, G, dk, dv, dims in ((4, 2, 16, 24, 0), (3, 1, 11, 6, 0), (2, 2, 32, 40, 8), (5, 5, 6, 34, 6), (2, 1, 200, 8, 0)):
        n = 70
        f = torch.tensor([100.0 ** (-2.0 * i / max(dims, 1)) for i in range(dims // 2)])
        a = torch.randn(n, H * dk + G * (dk + dv), generator=g) * 3
        wq, wk = torch.rand(dk, generator=g) + 0.5, torch.rand(dk, generator=g) - 0.5
        pos = torch.arange(3, 3 + n, dtype=torch.int32)
        q = torch.empty(n, H * dk, device=DEV)
        kc, vc = torch.zeros(2, G, 64, dk, device=DEV), torch.zeros(2, G, 64, dv, device=DEV)
        ops.qkv_prep(a.to(DEV), None, None, torch.cat([f, torch.zeros(1)]).to(DEV), pos.to(DEV),
                     torch.zeros(n, dtype=torch.int32, device=DEV), i32([[1, 0]]), q, kc, vc, None, H, G, dk, dv, dims, 1e-5,
                     pairing="half", head_weights=(wq.to(DEV), wk.to(DEV)))

        def normed(x, heads, w):
            y = P.plain_norm(x.double().view(n, heads, dk), w, 1e-5)
            ang = pos.double()[:, None] * f.double()
            c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
            u, v_ = y[..., :dims // 2], y[..., dims // 2:dims]
            return torch.cat([u * c - v_ * s, v_ * c + u * s, y[..., dims:]], -1)
        assert torch.allclose(q.cpu().double(), normed(a[:, :H * dk], H, wq).reshape(n, -1), atol=2e-4, rtol=1e-5)
        want_k = normed(a[:, H * dk:(H + G) * dk], G, wk)
        for t in range(n):
            p = int(pos[t])
            assert torch.allclose(kc[[1, 0][p // 64], :, p % 64].cpu().double(), want_k[t], atol=2e-4, rtol=1e-5)
            assert torch.equal(vc[[1, 0][p // 64], :, p % 64].cpu().reshape(-1), a[t, (H + G) * dk:])


@pytest.mark.parametrize("pairing", ["neighbours", "half"])
def test_the_latents_rows_with_queries_straight_from_the_input(pairing):
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(4)
    for H, dim, rot, dims, rank, pad in ((3, 20, 8, 8, 48, 4), (5, 12, 12, 6, 32, 0), (2, 9, 6, 6, 27, 3), (4, 7, 0, 0, 20, 0),
                                         (1, 64, 32, 32, 300, 8), (40, 8, 4, 2, 16, 0)):
        n = 70
        a = torch.randn(n, H * (dim + rot) + rank + rot + H + pad, generator=g) * 2
        w = torch.rand(rank, generator=g) + 0.5
        pos = torch.arange(5, 5 + n, dtype=torch.int32)
        pos[9] = -1
        f = torch.tensor([50.0 ** (-2.0 * i / max(dims, 1)) for i in range(dims // 2)] + [0.0])
        for gated in (True, False):
            q = torch.full((n, H * dim), 9.0, device=DEV)
            rows = torch.full((n, H * (rank + rot)), 9.0, device=DEV)
            cache = torch.zeros(2, 1, 64, rank + rot, device=DEV)
            gate = torch.empty(n, H, device=DEV) if gated else None
            ops.latent_prep_direct(a.to(DEV), w.to(DEV), f.to(DEV), pos.to(DEV), torch.zeros(n, dtype=torch.int32, device=DEV),
                                   i32([[1, 0]]), q, rows, cache, gate, H, dim, rank, rot, dims, 1e-5, pairing=pairing)

            def turned(x):  # [n, heads, rot]
                y = x.double().clone()
                for i in range(dims // 2):
                    i0, i1 = (2 * i, 2 * i + 1) if pairing == "neighbours" else (i, i + dims // 2)
                    c, s = torch.cos(pos.double() * f[i].double())[:, None], torch.sin(pos.double() * f[i].double())[:, None]
                    y[..., i0], y[..., i1] = x[..., i0] * c - x[..., i1] * s, x[..., i1] * c + x[..., i0] * s
                return y
            qa = a[:, :H * (dim + rot)].view(n, H, dim + rot)
            down = a[:, H * (dim + rot):]
            live = [t for t in range(n) if t != 9]
            assert torch.equal(q.cpu().view(n, H, dim)[live], qa[live][..., :dim]) and (q[9] == 9.0).all()
            got = rows.cpu().view(n, H, rank + rot)
            assert (got[..., :rank] == 9.0).all() and (got[9] == 9.0).all()
            assert torch.allclose(got[live][..., rank:].double(), turned(qa[..., dim:])[live], atol=3e-4)
            want_c = P.plain_norm(down[:, :rank].double(), w, 1e-5)
            want_k = turned(down[:, None, rank:rank + rot])[:, 0]
            for t in live:
                line = cache[[1, 0][int(pos[t]) // 64], 0, int(pos[t]) % 64].cpu().double()
                assert torch.allclose(line, torch.cat([want_c[t], want_k[t]]), atol=3e-4)
            if gated:
                assert torch.allclose(gate.cpu()[live], torch.sigmoid(down[:, rank + rot:rank + rot + H])[live], atol=1e-6)


def test_parts_turned_by_neighbours():
    """The rotation of a part of every head and the latent step with its own query latent know both pairings."""
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(14)
    n, H, length, dims = 9, 3, 10, 6
    src = torch.randn(n, H * 14, generator=g)
    pos = torch.arange(20, 20 + n, dtype=torch.int32)
    f = torch.tensor([1.0, 0.3, 0.05, 0.0])
    dst = torch.zeros(n, H * 12, device=DEV)
    ops.rope_part(src.to(DEV), 14, 3, dst, 12, 2, pos.to(DEV), f.to(DEV), H, length, dims, pairing="neighbours")
    got, x = dst.cpu().view(n, H, 12), src.view(n, H, 14)[..., 3:13]
    want = x.clone()
    for i in range(3):
        c, s = torch.cos(pos.double() * f[i])[:, None].float(), torch.sin(pos.double() * f[i])[:, None].float()
        want[..., 2 * i], want[..., 2 * i + 1] = x[..., 2 * i] * c - x[..., 2 * i + 1] * s, x[..., 2 * i + 1] * c + x[..., 2 * i] * s
    assert torch.allclose(got[..., 2:], want, atol=1e-5) and (got[..., :2] == 0).all()
    a = torch.randn(n, 8 + 12 + 6, generator=g)
    cq, cache = torch.empty(n, 8, device=DEV), torch.zeros(1, 1, 64, 18, device=DEV)
    ones = torch.ones(12, device=DEV)
    ops.latent_prep(a.to(DEV), ones[:8].contiguous(), ones, f.to(DEV), pos.to(DEV), torch.zeros(n, dtype=torch.int32, device=DEV),
                    i32([[0]]), cq, cache, 8, 12, 6, 6, 1e-5, pairing="neighbours")
    x = a[:, 20:].clone()
    for i in range(3):
        c, s = torch.cos(pos.double() * f[i]).float(), torch.sin(pos.double() * f[i]).float()
        x[:, 2 * i], x[:, 2 * i + 1] = a[:, 20 + 2 * i] * c - a[:, 21 + 2 * i] * s, a[:, 21 + 2 * i] * c + a[:, 20 + 2 * i] * s
    assert torch.allclose(cache[0, 0, 20:20 + n, 12:].cpu(), x, atol=1e-5)


@pytest.mark.parametrize("H, dk, dv, window", [(3, 56, 48, 33), (8, 33, 27, 1), (16, 144, 128, 65), (5, 40, 16, 64), (64, 96, 64, 100),
                                               (4, 304, 272, 150), (2, 544, 512, 130), (6, 112, 96, 0), (130, 24, 16, 7)])
def test_latent_attention_with_a_window_and_a_gate_in_every_cut(H, dk, dv, window):
    """Both kernels over scattered pages, pages that have left the window given back: whole prompts, later
    portions, single tokens, slices of the key range."""
    from nnis_b200.csrc import ops
    g = torch.Generator().manual_seed(H + dk)
    S, scale = 260, 1.1 / math.sqrt(dk)
    pages = [5, 2, 9, 0, 7]
    rows = torch.randn(S, 1, dk, generator=g)
    q = torch.randn(S, H, dk, generator=g)
    gate = torch.rand(S, H, generator=g)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        r, qd = rows.to(dtype), q.to(dtype)
        cache = torch.full((10, 1, 64, dk), 50.0, dtype=dtype)
        for t in range(S):
            cache[pages[t // 64], :, t % 64] = r[t]
        want = _plain_attention(qd.double(), r.double(), r[..., :dv].double(), window, 0, scale, None, gate.double())
        for a, b, splits in ((0, 130, 1), (130, 190, 1), (190, 191, 1), (191, 192, 3), (192, 200, 2), (0, 200, 4), (259, 260, 2)):
            n = b - a
            held = [p if not window or (i + 1) * 64 > a - window + 1 else -1 for i, p in enumerate(pages)]
            table = i32([[3] * 5, held])
            pos, seq = i32(list(range(a, b))), torch.ones(n, dtype=torch.int32, device=DEV)
            out = torch.full((n, H * dv), 9.0, dtype=dtype, device=DEV)
            partial = torch.empty(n * H * splits * (dv + 2), device=DEV) if splits > 1 else None
            args = (qd[a:b].reshape(n, -1).to(DEV), cache.to(DEV))
            ops.attention_latent(*args, pos, seq, table, out, H, dv, scale, splits, partial, window=window,
                                 gate=gate[a:b].to(DEV))
            assert torch.allclose(out.cpu().double(), want[a:b], atol=tol, rtol=tol), (dtype, a, b, splits)
            if dtype == torch.bfloat16 and ops.attention_latent_mma_takes(dk, dv, 64):
                out.fill_(9.0)
                if n == 1:  # a decode step: every row a token of its own
                    ops.attention_latent_mma(*args, None, None, None, None, pos, seq, table, out, H, dv, scale, splits,
                                             partial, window=window, gate=gate[a:b].to(DEV))
                else:
                    tiles = torch.from_numpy(ops.latent_tiles([1, n], [0, a], H, ops.latent_tile_rows(dv)))
                    tiles = tiles[tiles[:, 0] == 1].contiguous().to(DEV)
                    ops.attention_latent_mma(*args, tiles, i32([0, 0]), i32([0, a]), i32([1, n]), pos, seq, table, out, H,
                                             dv, scale, splits, partial, window=window, gate=gate[a:b].to(DEV))
                assert torch.allclose(out.cpu().double(), want[a:b], atol=tol, rtol=tol), ("mma", a, b, splits)


# ---- whole models against the plain implementation -----------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "loop_all", "loop_once", "heads64"])
def test_each_configuration_alone(models, name, dtype, tmp_path):
    rng = random.Random(11)
    vocab = read_config(models[name])["vocab"]
    sequences, trace = {}, TraceBuilder()
    # the first tokens, a page's border, windows' edges
    for i, n in enumerate((1, 2, 3, 50, 63, 64, 65, 131, 300)):
        sequences[f"w{i}"] = random_tokens(rng, n, vocab)
        trace.step([(f"w{i}", sequences[f"w{i}"], range(n))], end=[f"w{i}"])
    toks = sequences["d"] = random_tokens(rng, 75, vocab)  # decoding from the second token on
    trace.step([("d", toks[:1], [0])])
    for t in range(1, 75):
        trace.step([("d", toks[t:t + 1], [0])], end=["d"] if t == 74 else [])
    replay_and_check(models, name, dtype, trace, sequences, tmp_path, "alone")


@pytest.mark.parametrize("name", ["mixed", "odd", "heads64"])
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
    assert len(got) == len(want) == len(P.run_order(cfg))
    for i, (a, b) in enumerate(zip(got, want)):
        assert torch.allclose(a.double(), b, atol=1e-4 * float(b.abs().max())), i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "heads64"])
def test_whole_last_tokens_and_unequal_batches(models, name, dtype, tmp_path):
    vocab = read_config(models[name])["vocab"]
    trace, sequences = three_cuts(random.Random(3), vocab)
    replay_and_check(models, name, dtype, trace, sequences, tmp_path, "three cuts")


@pytest.mark.parametrize("name", ["mixed", "odd", "loop_all"])
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
        check_logits(a, plain_of(models[name], "float32", p)[0], "float32", "alone")
    # portions of several sizes, down to two tokens and one
    for cuts in ([2, 2, 60, 1, 64, 71], [64, 64, 64, 8], [199, 1], [1, 199], [39, 2, 7, 152], [3, 17, 16, 164],
                 [1, 1, 1, 2, 130, 65]):
        slot = engine.acquire_slot()
        rows, at = [], 0
        for c in cuts:
            rows.append(engine.step([SequenceStep(slot, prompts[0][at:at + c], list(range(c)))]).cpu().numpy())
            at += c
        engine.release_slot(slot)
        assert at == 200 and np.abs(np.concatenate(rows) - alone[0]).max() < 3e-5 * scale, cuts
    # one batch of all four, then the same again in slots and pages that were used before
    for _ in range(2):
        slots = [engine.acquire_slot() for _ in prompts]
        heads = [max(1, len(p) - 20) for p in prompts]
        got = engine.step([SequenceStep(s, p[:h], list(range(h))) for s, p, h in zip(slots, prompts, heads)]).cpu().numpy()
        at = 0
        for i, h in enumerate(heads):
            assert np.abs(got[at:at + h] - alone[i][:h]).max() < 3e-5 * scale
            at += h
        live = list(range(len(prompts)))
        step = 0
        while live:  # decoded together; the shorter ones end earlier
            batch = [SequenceStep(slots[i], prompts[i][heads[i] + step:heads[i] + step + 1], [0]) for i in live]
            got = engine.step(batch).cpu().numpy()
            for r, i in enumerate(live):
                assert np.abs(got[r] - alone[i][heads[i] + step]).max() < 3e-5 * scale, (i, step)
            step += 1
            for i in list(live):
                if heads[i] + step == len(prompts[i]):
                    engine.release_slot(slots[i])
                    live.remove(i)
    assert engine.cache.usage()["slots_held"] == 0
    engine.cache.check()


def test_pages_that_left_a_window_are_used_by_others_and_the_first_ones_are_not(models):
    """Two sequences grow in turn through a cache with few pages to spare: the pages that one gives back are
    taken by the other at once, while the kept first pages of both must stay as they are."""
    from nnis_b200.engine import Engine, SequenceStep
    name = "mixed"  # a window of nine that keeps 70 tokens, one of 50 that keeps five
    vocab = read_config(models[name])["vocab"]
    rng = random.Random(31)
    a, b = random_tokens(rng, 400, vocab), random_tokens(rng, 400, vocab)
    want_a, want_b = plain_of(models[name], "float32", a)[0], plain_of(models[name], "float32", b)[0]
    engine = Engine.from_dir(models[name], dtype="float32", max_tokens=64 * 12, max_slots=2)
    sa, sb = engine.acquire_slot(), engine.acquire_slot()
    seen = [set() for _ in engine.cache.groups]
    for at in range(0, 384, 32):
        for slot, toks, want in ((sa, a, want_a), (sb, b, want_b)):
            got = engine.step([SequenceStep(slot, toks[at:at + 32], list(range(32)))]).cpu().numpy()
            check_logits(got, want[at:at + 32], "float32", f"turns {at}")
        for g in range(len(engine.cache.groups)):
            seen[g] |= {(s, p) for s in (sa, sb) for p in engine.cache.page_table(g, s) if p >= 0}
    keeps = [g for g, grp in enumerate(engine.cache.groups) if grp.keep_first == 70]
    assert len(keeps) == 1
    pages_of = lambda s: {p for t, p in seen[keeps[0]] if t == s}
    assert pages_of(sa) & pages_of(sb)  # pages really changed hands
    for s in (sa, sb):
        table = engine.cache.page_table(keeps[0], s)
        assert table[0] >= 0 and table[1] >= 0 and table[2] < 0 and table[3] < 0
        engine.release_slot(s)
    engine.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_prompt_shape_that_recurs_is_captured_and_replayed(models, dtype):
    """A large prompt step whose shape comes a second time is recorded as a CUDA graph and replayed from
    the third time on.  Other tokens every time, the same shape."""
    from nnis_b200.engine import Engine, SequenceStep
    engine = Engine.from_dir(models["mixed"], dtype=dtype, max_tokens=64 * 64)
    vocab = read_config(models["mixed"])["vocab"]
    rng = random.Random(77)
    graphs = []
    for round_ in range(4):
        a, b = random_tokens(rng, 300, vocab), random_tokens(rng, 40, vocab)
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
@pytest.mark.parametrize("name", ["mixed", "sharp"])
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
    ``query_pos`` against the key at ``key_pos``.  One row of W_q (the last plain value of every head) lies
    along the normed embedding of the query's token, one of the keys' along the key's token's."""
    from safetensors.torch import load_file, save_file
    os.makedirs(out_dir, exist_ok=True)
    w = load_file(os.path.join(model_dir, "model.safetensors"))
    plain = {k: v.double() for k, v in w.items()}
    h = P.centred_norm(P.embedding(tokens, plain, cfg), plain["l0.norm1"], cfg["norm"]["eps"])
    hq, hk = h[query_pos] / h[query_pos].norm(), h[key_pos] / h[key_pos].norm()
    m = cfg["layers"][0]["mixer"]
    d = m["dim"]
    q = plain["l0.mix.q"].clone()
    if cfg["layers"][0]["type"] == "attention":
        k = plain["l0.mix.k"].clone()
        for a in range(m["heads"]):
            q[a * d + d - 1] = hq
        for a in range(m["kv_heads"]):
            k[a * d + d - 1] = hk
        w["l0.mix.k"] = k.to(torch.bfloat16)
        w["l0.mix.rel"] = (plain["l0.mix.rel"] * 0.3).to(torch.bfloat16)
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
    cfg_rows = config(97, 64, 1e-5, [(first, moe(4, 2, 24, 2, 1)), (latent(2, 8, 4, 16, 16, 1, 0.5), None)], scale=2.0)
    base = make_model(str(tmp_path / "base"), cfg_rows, seed)
    cfg = read_config(base)
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
        if dtype == "float32":
            check_rows(d, dtype, rows, f"{what} {dtype}")
            slot = engine.acquire_slot()
            changed = engine.step([SequenceStep(slot, other, [qp])]).cpu().numpy()
            engine.release_slot(slot)
            seen = float(np.abs(changed[0] - want[qp].numpy()).max()) > 1e-3
            assert seen == visible
        else:
            logits, gaps = plain_of(d, dtype, toks)
            clear = [r for r in rows if float(gaps[r[1]]) >= CLOSE_CALL]
            if clear:  # (the same two positions in every cut: a router's close call may take either out)
                check_logits(np.stack([r for _, _, r in clear]), torch.stack([logits[p] for _, p, _ in clear]), dtype, what)


@pytest.mark.parametrize("kind", ["attention", "latent"])
@pytest.mark.parametrize("window, distance", [(40, 39), (40, 40), (64, 63), (64, 64), (65, 64), (65, 65), (129, 128),
                                              (129, 129), (250, 249), (7, 6), (7, 7)])
def test_a_key_just_inside_and_just_outside_the_window(kind, window, distance, tmp_path):
    n = 270
    qp = n - 3
    first = attention(4, 2, 16, 24, window, 3, 3.0, 50, 10) if kind == "attention" \
        else latent(4, 16, 8, 24, 16, window, 0.5, 100.0)
    _edge(tmp_path, first, qp - distance, qp, n, distance < window, 31, f"{kind} window {window} distance {distance}")


@pytest.mark.parametrize("keep, key", [(0, 0), (1, 0), (1, 1), (5, 4), (5, 5), (64, 63), (64, 64), (65, 64), (65, 65), (130, 129),
                                       (130, 130)])
def test_the_first_tokens_stay_visible_and_the_next_ones_do_not(keep, key, tmp_path):
    """A window of 30 that keeps ``keep`` tokens, a query 200 positions in."""
    _edge(tmp_path, attention(4, 2, 16, 24, 30, keep, 3.0, 50, 10), key, 200, 206, key < keep, 41, f"keep {keep} key {key}")


@pytest.mark.parametrize("rows, far, distance", [(10, 50, 4), (10, 50, 5), (10, 50, 49), (10, 50, 50), (10, 50, 200), (16, 128, 15),
                                                 (16, 128, 16), (16, 128, 63), (16, 128, 64), (2, 3, 0), (2, 3, 1)])
def test_one_bucket_of_distances_decides(rows, far, distance, tmp_path):
    """The bucket that holds ``distance`` gets a bias that outweighs everything else: the query's weight lies on
    the keys at that bucket's distances, in a prompt, in a portion and decoded alone."""
    from nnis_b200.engine import Engine, SequenceStep
    from safetensors.torch import load_file, save_file
    cfg_rows = config(83, 56, 1e-5, [(attention(4, 2, 16, 24, 300, 0, 0.3, far, rows), None)], scale=2.0)
    d = make_model(str(tmp_path / "m"), cfg_rows, 5)
    w = load_file(os.path.join(d, "model.safetensors"))
    b = P.bucket_of(distance, rows, far)
    w["l0.mix.rel"] = torch.zeros(rows, 4, dtype=torch.bfloat16)
    w["l0.mix.rel"][b] = 12.0
    save_file(w, os.path.join(d, "model.safetensors"))
    toks = random_tokens(random.Random(distance), 230, 83)
    probe = {}
    P.forward(toks, load_weights(d, False), read_config(d), probe=probe)
    weights = probe["weights"][0][225]
    inside = [j for j in range(226) if P.bucket_of(225 - j, rows, far) == b]
    assert float(weights[inside].sum()) > 0.9
    for dtype in DTYPES:
        engine = Engine.from_dir(d, dtype=dtype, max_tokens=1024)
        slot = engine.acquire_slot()
        got = engine.step([SequenceStep(slot, toks[:150], list(range(150)))]).cpu().numpy()
        got = np.concatenate([got, engine.step([SequenceStep(slot, toks[150:220], list(range(70)))]).cpu().numpy()])
        for t in range(220, 230):
            got = np.concatenate([got, engine.step([SequenceStep(slot, toks[t:t + 1], [0])]).cpu().numpy()])
        engine.release_slot(slot)
        check_rows(d, dtype, [(toks, i, got[i]) for i in range(230)], f"bucket {rows} {far} {distance} {dtype}")


def test_far_keys_and_page_borders_with_sharp_attention(models, tmp_path):
    """Random sharp heads put most of a query's weight on single keys anywhere in their windows (300,
    129 and 64 tokens and the first ones): prompts that end on both sides of page borders, portions that start
    there, and tokens decoded across them."""
    from nnis_b200.engine import SequenceStep
    vocab = read_config(models["sharp"])["vocab"]
    rng = random.Random(5)
    probe = {}
    toks = random_tokens(rng, 450, vocab)
    P.forward(toks, load_weights(models["sharp"], False), read_config(models["sharp"]), probe=probe)
    peak = torch.stack([m.max(-1).values for m in probe["weights"]])[:, 100:]
    assert float(peak.mean()) > 0.4  # sharp: much of a query's weight on one key, on average
    far = torch.stack([(m.argmax(-1) - torch.arange(450)).abs() for m in probe["weights"]])
    assert int(far.max()) > 120      # and some of those keys lie far back
    kept = [m[200:].argmax(-1) < 66 for m in probe["weights"][-2:]]
    assert any(bool(k.any()) for k in kept)  # some of them among the kept first tokens
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


def _random_config(rng):
    width = rng.choice([40, 64, 76, 96, 128])
    layers = []
    n_layers = rng.randint(1, 4)
    for _ in range(n_layers):
        if rng.random() < 0.5:
            kv = rng.randint(1, 3)
            dim = rng.choice([1, 5, 6, 8, 16, 24, 32, 40, 64])
            rows = rng.choice([2, 3, 5, 8, 16, 31])
            mixer = attention(kv * rng.randint(1, 4), kv, dim, rng.choice([1, 4, 6, 16, 24, 34, 64, 72, 130]),
                              rng.choice([1, 2, 17, 63, 64, 65, 100, 1000]), rng.choice([0, 1, 4, 63, 64, 65, 500]),
                              rng.choice([0.2, 0.5, 1.0]) / math.sqrt(dim), rows // 2 + rng.choice([1, 2, 10, 100, 5000]), rows)
        else:
            rot = rng.choice([0, 1, 2, 4, 8, 16])
            dims = rng.choice([0, rot // 2 * 2, rot // 4 * 2])
            dim = rng.choice([1, 5, 8, 16, 24, 40])
            mixer = latent(rng.randint(1, 6), dim, rot, rng.choice([1, 4, 8, 13, 24, 64]), rng.choice([1, 6, 16, 24, 48, 80, 130]),
                           rng.choice([1, 2, 17, 63, 64, 65, 100, 1000]), rng.choice([0.2, 0.5, 1.0]) / math.sqrt(dim + rot),
                           rng.choice([10.0, 10000.0, 500000.0]), dims)
        mlp = None
        if rng.random() < 0.75:
            count = rng.choice([1, 1, 2, 3, 4])
            size = rng.randint(1, 4)
            keep = rng.randint(1, count)
            mlp = moe(count * size, rng.randint(1, keep * size), rng.choice([1, 8, 12, 24, 40]), count, keep)
        layers.append((mixer, mlp))
    loop = None
    if rng.random() < 0.7:
        start = rng.randint(0, n_layers - 1)
        loop = (start, rng.randint(start + 1, n_layers), rng.randint(1, 3))
    return config(rng.choice([50, 131, 256, 577]), width, rng.choice([1e-5, 1e-6]), layers, loop=loop,
                  scale=rng.choice([1.0, 0.5, 12.0]))


@pytest.mark.parametrize("trial", range(14))
def test_configurations_drawn_at_random(trial, tmp_path):
    """A prompt in one step, a second portion and six tokens one by one, both dtypes, on a model
    whose sizes, layer order, loop and constants are drawn at random: whatever kernels the sizes select."""
    from nnis_b200.engine import Engine, SequenceStep
    rng = random.Random(5100 + trial)
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
        check_rows(d, dtype, [(toks, i, got[i]) for i in range(150)], f"random configuration {trial} {dtype}: {json.dumps(cfg)}")


def _middle_config(rng):
    """Sizes of a small real model: the shapes at which the tensor-core products, the decode projections over
    tiles of rows and the tensor-core attention take over from the any-size kernels."""
    width = rng.choice([192, 256, 384, 512])
    layers = []
    n_layers = rng.randint(2, 4)
    for i in range(n_layers):
        if (i + rng.randint(0, 1)) % 2:
            kv = rng.choice([1, 2, 4])
            dim = rng.choice([32, 64, 80, 128])
            mixer = attention(kv * rng.choice([1, 2, 3, 4]), kv, dim, rng.choice([64, 128, 32, 96]), rng.choice([64, 100, 200, 4096]),
                              rng.choice([0, 4, 64, 100]), 2 / dim, rng.choice([64, 128, 1000]), rng.choice([16, 32]))
        else:
            dim = rng.choice([32, 64])
            mixer = latent(rng.choice([4, 8, 16]), dim, dim // 2, rng.choice([32, 64]), rng.choice([64, 128, 256]),
                           rng.choice([64, 100, 200, 4096]), 1 / math.sqrt(dim))
        mlp = rng.choice([None, moe(8, 2, rng.choice([64, 128]), 4, 2), moe(6, 3, 96, 2, 1)])
        layers.append((mixer, mlp))
    loop = rng.choice([None, (0, n_layers, 2), (1, n_layers, 2), (0, 1, 3)])
    return config(rng.choice([1000, 2048, 4099]), width, 1e-6, layers, loop=loop, scale=rng.choice([1.0, 8.0]))


@pytest.mark.parametrize("trial", range(6))
def test_middle_sizes_drawn_at_random(trial, tmp_path):
    """A batch of two prompts (one of them in two portions) and eight tokens decoded together, both
    dtypes, at sizes of a small real model."""
    from nnis_b200.engine import Engine, SequenceStep
    rng = random.Random(6200 + trial)
    cfg = _middle_config(rng)
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
        check_rows(d, dtype, rows, f"middle size {trial} {dtype}: {json.dumps(cfg)}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_point(models, dtype):
    from nnis_b200 import LLM
    d = models["mixed"]
    cfg = read_config(d)
    bf = dtype == "bfloat16"
    w = load_weights(d, bf)
    llm = LLM(d, dtype=dtype, max_tokens=64 * 32, max_batch=3)
    rng = random.Random(17)
    # (the long ones: pages between the kept first ones and the windows have gone back before decoding)
    prompts = [[5, 9, 1, 200, 33], [7], random_tokens(rng, 260, 307), [250, 3], random_tokens(rng, 135, 307)]
    results = llm.generate(prompts, max_new_tokens=10, stop_token_ids=())
    for p, r in zip(prompts, results):
        assert r.ok and r.finish_reason == "length"
        if not bf:
            assert r.token_ids == P.greedy_generate(cfg, w, p, 10), (dtype, p)
        else:  # a bfloat16 near-tie or a router's close call may go either way: nearly every pick is nearly the best
            seq, far_off = list(p), 0
            for t in r.token_ids:
                logits = P.forward(seq, w, cfg, emulate_bf16=True)[-1]
                far_off += float(logits.max() - logits[t]) > 0.05 * max(1.0, float(logits.abs().max()))
                seq.append(t)
            assert far_off <= 2, p
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
    pools, and the kept first pages stay in the tables that the device holds."""
    from nnis_b200 import LLM
    d = models["mixed"]
    llm = LLM(d, dtype="float32", max_tokens=64 * 20, max_batch=2)
    prompts = [random_tokens(random.Random(3), 20, 307), random_tokens(random.Random(4), 90, 307)]
    results = llm.generate(prompts, max_new_tokens=200, stop_token_ids=())
    w, cfg = load_weights(d, False), read_config(d)
    for p, r in zip(prompts, results):
        logits = P.forward(p + r.token_ids, w, cfg)
        for i, t in enumerate(r.token_ids):
            row = logits[len(p) + i - 1]
            assert float(row.max() - row[t]) <= 1e-4 * float(row.abs().max()), i


def test_sampled_generation_and_the_command_line(models, tmp_path):
    """Sampling with a seed repeats itself, and the command line's generate runs the design."""
    import sys
    from nnis_b200 import LLM
    from nnis_b200.sampling import SamplingConfig
    llm = LLM(models["odd"], dtype="bfloat16", max_tokens=2048, max_batch=2)
    policy = SamplingConfig.seeded(5).with_temperature(0.9).with_top_k(40)
    a = llm.generate([[1, 2, 3], [9, 8]], max_new_tokens=12, sampling=policy, stop_token_ids=())
    b = llm.generate([[1, 2, 3], [9, 8]], max_new_tokens=12, sampling=policy, stop_token_ids=())
    assert [r.token_ids for r in a] == [r.token_ids for r in b] and all(len(r.token_ids) == 12 for r in a)
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "nnis"), "generate", "--model", models["loop_all"],
                        "--prompt-ids", "4,5,6", "--max-new-tokens", "5", "--dtype", "float32"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    want = P.greedy_generate(read_config(models["loop_all"]), load_weights(models["loop_all"], False), [4, 5, 6], 5)
    assert r.stdout.split() == [str(t) for t in want]


def test_replay_program_runs_a_model_folder(models, tmp_path):
    cfg = read_config(models["loop_all"])
    toks = random_tokens(random.Random(4), 40, cfg["vocab"])
    trace = TraceBuilder()
    trace.step([("a", toks[:30], [0, 29]), ("b", toks[:7], [6])])
    trace.step([("a", toks[30:31], [0]), ("b", toks[7:8], [0])], end=["b"])
    trace.step([("a", toks[31:32], [])], end=["a"])
    out = str(tmp_path / "out")
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", models["loop_all"], "--dtype", "float32",
                        "--out", out, "--max-tokens", "256"], input="\n".join(trace.lines) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not os.path.exists(os.path.join(out, "2.f32"))
    want = plain_of(models["loop_all"], "float32", toks)[0]
    check_logits(read_step(out, 0, cfg["vocab"]), torch.stack([want[0], want[29], want[6]]), "float32", "program")
    check_logits(read_step(out, 1, cfg["vocab"]), torch.stack([want[30], want[7]]), "float32", "program")
