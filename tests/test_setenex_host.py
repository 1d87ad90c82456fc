"""Setenex without a GPU: configuration round trip and errors by key, tensor names, the run order
of a looped model, buckets of distances, what the design asks of the cache and pages that a window keeps,
and the plain mechanisms against closed forms."""
import copy
import math

import pytest
import torch

import plain_setenex as P
from setenex_models import (CONFIGS, HEADS_64, LOOP_ALL, LOOP_ONCE, MIXED, ODD, load_weights, make_model, read_config,
                            written)

F = torch.float64


def test_configuration_round_trip_and_spec():
    from nnis_b200.config import config_from_dict, known_architectures
    assert "Setenex" in known_architectures()
    for cfg in CONFIGS.values():
        typed = config_from_dict(written(cfg))
        assert config_from_dict(typed.to_dict()).to_dict() == typed.to_dict()
        spec = typed.to_spec()
        assert [l.block for l in spec.layers] == ["parallel"] * len(cfg["layers"])
        for i, layer in enumerate(cfg["layers"]):
            parts = spec.layers[i].parts
            assert ("ffn" in parts) == (layer["mlp"] is not None) and "ffn_norm" not in parts  # one norm for both
            assert parts["mixer"].kind == {"attention": "sink_attention"}.get(layer["type"], layer["type"])
            assert parts["norm"]["offset"] == 1.0
        assert spec.final_norm["offset"] == 1.0 and spec.head.get("tied_to") is None
    spec = config_from_dict(written(MIXED)).to_spec()
    a = spec.layers[0].part("mixer")
    assert (a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["window"], a["keep_first"]) == (4, 2, 24, 40, 50, 5)
    assert a["distance_bias"]["far"] == 100 and a["qk_norm"] == "head_weight" and a["position"]["dims"] == 0
    b = spec.layers[3].part("mixer")
    assert (b["heads"], b["dim"], b["rot_dim"], b["vdim"], b["kv_rank"], b["window"]) == (5, 12, 12, 8, 32, 200)
    assert b["q_rank"] == 0 and b["gate"] == "head"
    assert (b["position"]["dims"], b["position"]["base"], b["position"]["pairing"]) == (6, 50.0, "neighbours")
    m = spec.layers[1].part("ffn")
    assert (m["experts"], m["top"], m["ff"], m["groups"], m["keep"], m["group_top"]) == (8, 3, 16, 4, 2, 2)
    assert m["scores"] == "sigmoid_all" and m["renormalise"] and m["activation"] == "gelu" and m["weight_on"] == "output"
    assert spec.embedding["scale"] == 3.0


def test_a_loop_is_a_schedule_that_names_its_layers_once_per_pass():
    from nnis_b200.config import config_from_dict
    from nnis_b200.config.spec import StreamEnter
    sched = config_from_dict(written(MIXED)).to_spec().schedule
    assert [e.layer for e in sched] == [0, 1, 2, 1, 2, 1, 2, 3]
    # before every pass, the first too, its row; the embedding does not come back
    assert {i: e.enter for i, e in enumerate(sched) if e.enter is not None} == {
        1: StreamEnter(False, "loop.step", 3, 0), 3: StreamEnter(False, "loop.step", 3, 1),
        5: StreamEnter(False, "loop.step", 3, 2)}
    assert all(e.cache_of is None for e in sched)  # a cache per pass
    sched = config_from_dict(written(LOOP_ALL)).to_spec().schedule
    assert [e.layer for e in sched] == [0, 1, 0, 1] and sched[0].enter == StreamEnter(False, "loop.step", 2, 0)
    sched = config_from_dict(written(LOOP_ONCE)).to_spec().schedule
    assert [e.layer for e in sched] == [0, 1] and sched[1].enter == StreamEnter(False, "loop.step", 1, 0)
    assert all(e.enter is None for e in config_from_dict(written(ODD)).to_spec().schedule)
    assert [(i, t) for i, t, first in P.run_order(MIXED) if first] == [(1, 0), (1, 1), (1, 2)]


@pytest.mark.parametrize("change, word", [
    (lambda c: c.update(architecture="Other"), "architecture"),
    (lambda c: c["layers"][0].update(type="conv"), "not a mixer"),
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("bias_max"), "bias_max"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["mask"].pop("keep_first"), "keep_first"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "moe"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(layers=[]), "at least one layer"),
])
def test_configuration_errors_name_the_key(change, word):
    from nnis_b200.config import ConfigError, config_from_dict
    cfg = copy.deepcopy(written(MIXED))
    change(cfg)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    assert word in str(e.value)


def test_tensor_names_and_shapes(tmp_path):
    from nnis_b200.config import config_from_dict
    from nnis_b200.engine.model import DecoderModel
    specs = DecoderModel.weight_specs_of(config_from_dict(written(MIXED)).to_spec())
    shapes = {n: tuple(s.shape) for n, s in specs.items()}
    assert shapes["embed"] == shapes["head"] == (307, 96)
    assert shapes["loop.step"] == (3, 96) and shapes["final.norm"] == shapes["l0.norm1"] == (96,)
    assert shapes["l0.mix.q"] == (96, 96) and shapes["l0.mix.k"] == (48, 96) and shapes["l0.mix.v"] == (80, 96)
    assert shapes["l0.mix.q.norm"] == shapes["l0.mix.k.norm"] == (24,) and shapes["l0.mix.o"] == (96, 160)
    assert shapes["l0.mix.rel"] == (-1, 4)  # its rows are the stored tensor's
    assert shapes["l1.mix.q"] == (3 * 28, 96) and shapes["l1.mix.dkv"] == (56, 96) and shapes["l1.mix.dkv.norm"] == (48,)
    assert shapes["l1.mix.uk"] == (60, 48) and shapes["l1.mix.uv"] == (72, 48)
    assert shapes["l1.mix.g"] == (3, 96) and shapes["l1.mix.o"] == (96, 72)
    assert shapes["l1.mlp.router"] == (8, 96) and shapes["l1.mlp.correction"] == (8,)
    assert shapes["l1.mlp.e7.up"] == (16, 96) and shapes["l1.mlp.e7.down"] == (96, 16) and "l1.mlp.e8.up" not in shapes
    assert "l2.mlp.router" not in shapes and "l0.norm2" not in shapes and "l1.mlp.e0.gate" not in shapes
    d = make_model(str(tmp_path / "m"), MIXED, 3)
    w = load_weights(d, False)
    assert set(w) == set(shapes) and tuple(w["l0.mix.rel"].shape) == (12, 4) and tuple(w["l2.mix.rel"].shape) == (9, 6)
    from nnis_b200.weights import load_weights as product_load
    got = product_load(d, specs, torch.float32, torch.device("cpu"))
    model = DecoderModel(config_from_dict(read_config(d)).to_spec(), torch.float32, torch.device("cpu"))
    model.load(got)
    assert "loop.step" not in DecoderModel.weight_specs_of(config_from_dict(written(ODD)).to_spec())


@pytest.mark.parametrize("rows, far", [(16, 128), (32, 128), (2, 2), (2, 3), (3, 9), (7, 100), (64, 4096), (12, 100), (33, 300), (9, 33)])
def test_buckets_of_distances(rows, far):
    from nnis_b200.parts.sink_attention import distance_buckets
    got = distance_buckets(rows, far)
    half = rows // 2
    for n in range(len(got) + 40):
        b = got[min(n, len(got) - 1)]
        assert b == P.bucket_of(n, rows, far)
        if n < half:
            assert b == n
        else:  # the logarithmic rule itself, where floating point leaves no doubt
            x = math.log(n / half) / math.log(far / half) * (rows - half)
            if abs(x - round(x)) > 1e-9:
                assert b == min(rows - 1, half + math.floor(x))
    assert got[-1] == rows - 1 and got[-2] < rows - 1 and got == sorted(got)
    # a border that is a whole number opens its bucket
    if (rows, far) == (16, 128):
        assert (got[16], got[15], got[32], got[31], got[64], got[63]) == (10, 9, 12, 11, 14, 13)


def test_a_distance_table_needs_a_far_end_beyond_half_its_rows():
    from nnis_b200.parts.sink_attention import distance_buckets
    for rows, far in ((16, 8), (1, 5), (0, 5)):
        with pytest.raises(ValueError):
            distance_buckets(rows, far)


def test_the_bias_is_laid_out_by_distance(tmp_path):
    from nnis_b200.config import config_from_dict
    from nnis_b200.engine.model import DecoderModel
    from nnis_b200.weights import load_weights as product_load
    d = make_model(str(tmp_path / "m"), ODD, 8)
    spec = config_from_dict(read_config(d)).to_spec()
    model = DecoderModel(spec, torch.float32, torch.device("cpu"))
    model.load(product_load(d, DecoderModel.weight_specs_of(spec), torch.float32, torch.device("cpu")))
    w = load_weights(d, False)
    for i in (0, 2, 4):
        want = P.bias_of_distances(120, w[f"l{i}.mix.rel"], ODD["layers"][i]["mixer"]["bias_max"])
        bias = model.blocks[i].mixer.bias
        for n in (0, 1, 2, 3, 7, 20, 33, 64, 119):
            assert torch.equal(bias[:, min(n, bias.shape[1] - 1)].double(), want[119, 119 - n])


def test_what_the_design_asks_of_the_cache():
    from nnis_b200.cache import CacheManager, KVRequest
    from nnis_b200.config import config_from_dict
    from nnis_b200.engine.model import DecoderModel
    model = DecoderModel(config_from_dict(written(MIXED)).to_spec(), torch.float32, torch.device("cpu"))
    requests = model.cache_requests()
    assert len(requests) == 8 + 1 and requests[-1] is None
    assert requests[0] == KVRequest(2, 24, 50, True, 40, keep_first=5)
    assert requests[1] == requests[3] == requests[5] == KVRequest(1, 56, 33, values=False)
    assert requests[2] == requests[4] == requests[6] == KVRequest(2, 16, 9, True, 16, keep_first=70)
    cache = CacheManager(requests, torch.float32, torch.device("cpu"), 64 * 8, 4, 1 << 20)
    # the three passes of a looped layer have storage of their own within one group
    views = [cache.view(i) for i in (2, 4, 6)]
    assert len({v.k.data_ptr() for v in views}) == 3 and len({v.group for v in views}) == 1
    assert views[0].keep_first == 70 and cache.view(1).v is None and cache.view(1).window == 33
    per = 4 * (2 * (24 + 40) * 55 + 3 * 2 * 32 * 79 + 3 * 56 * 33 + 44 * 100)  # (the last window holds all 100)
    assert cache.kv_bytes_read(100) == per


def test_a_window_that_keeps_the_first_tokens_keeps_their_pages():
    from nnis_b200.cache import PAGE_SIZE, CacheManager, KVRequest
    for keep, kept in ((0, 0), (1, 1), (64, 1), (65, 2), (130, 3)):
        cache = CacheManager([KVRequest(1, 4, 70, keep_first=keep), KVRequest(1, 4, 70)], torch.float32,
                             torch.device("cpu"), PAGE_SIZE * 12, 2, 1 << 20)
        assert (len(cache.groups) == 1) == (keep == 0)  # a group of its own where pages stay
        slot = cache.acquire()
        for n in (1, 63, 64, 65, 130, 200, 201, 500, 640):
            cache.reserve([slot], [n])
            cache.commit([slot], [n])
            table = cache.page_table(0, slot)
            # the next token, at position n, sees keys above n - 70 and the first ones
            needed = {j // PAGE_SIZE for j in range(n) if j > n - 70 or j < keep}
            assert all(table[p] >= 0 for p in needed), (keep, n)
            held = {p for p, page in enumerate(table) if page >= 0}
            assert held == needed | {p for p in held if p < kept or p == (n - 1) // PAGE_SIZE}, (keep, n)
            cache.check()
        # going back within what is still held; the kept pages are there, the ones between are not
        cache.truncate(slot, 639)
        with pytest.raises(Exception):
            cache.truncate(slot, 400)
        cache.check()
        cache.release(slot)
        assert not any(cache.usage()["pages_held"])
        assert cache.page_table(0, cache.acquire()) == []


# ---- the plain mechanisms against closed forms ---------------------------------------------------
def _mixer(cfg, index, tmp_path, seed=5, T=12, **changes):
    cfg = copy.deepcopy(cfg)
    m = cfg["layers"][index]["mixer"]
    for key, value in changes.items():
        if key in ("size", "keep_first"):
            m["mask"][key] = value
        else:
            m[key] = value
    d = make_model(str(tmp_path / f"m{index}_{len(str(changes))}_{hash(str(changes)) % 10**6}"), cfg, seed)
    w = load_weights(d, False)
    h = torch.randn(T, cfg["width"], dtype=F, generator=torch.Generator().manual_seed(1))
    probe = {}
    out = P.MIXERS[cfg["layers"][index]["type"]](h, w, f"l{index}.mix", m, 1e-5, False, probe)
    return m, w, h, out, probe


@pytest.mark.parametrize("size, keep", [(1, 0), (3, 0), (3, 2), (5, 4), (1, 12), (100, 3)])
def test_plain_attention_sees_a_window_and_the_first_tokens(size, keep, tmp_path):
    _, _, _, _, probe = _mixer(MIXED, 0, tmp_path, size=size, keep_first=keep)
    for a in probe["weights"]:
        for i in range(12):
            seen = [j for j in range(12) if a[i, j] > 0]
            assert seen == [j for j in range(i + 1) if i - j < size or j < keep]
            assert abs(a[i].sum() - 1) < 1e-12
    _, _, _, _, probe = _mixer(MIXED, 1, tmp_path, size=size)
    for a in probe["weights"]:
        for i in range(12):
            assert [j for j in range(12) if a[i, j] > 0] == list(range(max(0, i - size + 1), i + 1))


def test_plain_attention_norms_heads_and_adds_the_bias_unscaled(tmp_path):
    m, w, h, out, probe = _mixer(MIXED, 0, tmp_path, size=100, keep_first=0)
    q = (h @ w["l0.mix.q"].T).view(12, 4, 24)
    k = (h @ w["l0.mix.k"].T).view(12, 2, 24)
    v = (h @ w["l0.mix.v"].T).view(12, 2, 40)
    heads = []
    for a in range(4):
        g = a // 2
        rows = torch.zeros(12, 12, dtype=F)
        for i in range(12):
            qi = q[i, a] / torch.sqrt((q[i, a] ** 2).mean() + 1e-5) * w["l0.mix.q.norm"]
            for j in range(i + 1):
                kj = k[j, g] / torch.sqrt((k[j, g] ** 2).mean() + 1e-5) * w["l0.mix.k.norm"]
                rows[i, j] = math.exp(float(qi @ kj) * m["scale"] + float(w["l0.mix.rel"][P.bucket_of(i - j, 12, 100), a]))
        rows = rows / rows.sum(-1, keepdim=True)
        assert torch.allclose(rows, probe["weights"][a], atol=1e-12)
        heads.append(rows @ v[:, g])
    assert torch.allclose(out, torch.cat(heads, -1) @ w["l0.mix.o"].T, atol=1e-12)


def test_plain_rotation_turns_neighbouring_pairs():
    x = torch.arange(1, 19, dtype=F).view(3, 1, 6)
    y = P.rotate_neighbours(x, 4, 100.0)
    assert torch.equal(y[..., 4:], x[..., 4:]) and torch.equal(y[0], x[0])
    for p in range(3):
        for i in range(2):
            a, b = x[p, 0, 2 * i], x[p, 0, 2 * i + 1]
            c, s = math.cos(p * 100.0 ** (-i / 2)), math.sin(p * 100.0 ** (-i / 2))
            assert abs(y[p, 0, 2 * i] - (a * c - b * s)) < 1e-12 and abs(y[p, 0, 2 * i + 1] - (b * c + a * s)) < 1e-12


def test_plain_latent_attention_is_attention_over_what_the_latent_gives(tmp_path):
    m, w, h, out, probe = _mixer(MIXED, 3, tmp_path)
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    down = h @ w["l3.mix.dkv"].T
    c = down[:, :rank] / torch.sqrt((down[:, :rank] ** 2).mean(-1, keepdim=True) + 1e-5) * w["l3.mix.dkv.norm"]
    q = (h @ w["l3.mix.q"].T).view(12, H, d + r)
    kr = P.rotate_neighbours(down[:, None, rank:], m["rot"]["dims"], m["rot"]["base"])[:, 0]
    gate = torch.sigmoid(h @ w["l3.mix.g"].T)
    heads = []
    for a in range(H):
        k = c @ w["l3.mix.uk"][a * d:(a + 1) * d].T
        v = c @ w["l3.mix.uv"][a * dv:(a + 1) * dv].T
        qr = P.rotate_neighbours(q[:, a:a + 1, d:], m["rot"]["dims"], m["rot"]["base"])[:, 0]
        s = (q[:, a, :d] @ k.T + qr @ kr.T) * m["scale"]
        p = torch.softmax(s.masked_fill(torch.ones(12, 12).triu(1).bool(), -math.inf), -1)
        assert torch.allclose(p, probe["weights"][a], atol=1e-12)
        heads.append((p @ v) * gate[:, a:a + 1])
    assert torch.allclose(out, torch.cat(heads, -1) @ w["l3.mix.o"].T, atol=1e-12)


def test_plain_router_ranks_groups_by_their_two_best_and_divides_by_the_sum():
    g = torch.Generator().manual_seed(3)
    h = torch.randn(40, 16, dtype=F, generator=g)
    w = {"r.router": torch.randn(12, 16, dtype=F, generator=g), "r.correction": torch.randn(12, dtype=F, generator=g) * 0.2 - 0.8}
    r = {"experts": 12, "top": 3, "groups": {"count": 4, "keep": 2}}
    ids, weights = P.route(h, w, "r", r)
    s = torch.sigmoid(h @ w["r.router"].T)
    c = s + w["r.correction"]
    assert float(c.min()) < 0  # (a group left out is out, not worth zero)
    by_best = 0
    for t in range(40):
        two = lambda k: float(c[t, 3 * k:3 * k + 3].sort(descending=True).values[:2].sum())
        best = sorted(range(4), key=lambda k: -two(k))[:2]
        by_best += set(best) != set(sorted(range(4), key=lambda k: -float(c[t, 3 * k:3 * k + 3].max()))[:2])
        allowed = [e for k in best for e in range(3 * k, 3 * k + 3)]
        want = sorted(allowed, key=lambda e: -float(c[t, e]))[:3]
        assert ids[t].tolist() == want
        assert torch.allclose(weights[t], s[t, want] / s[t, want].sum(), atol=1e-15)
    assert by_best > 0  # the two rules differ somewhere
    # groups of one expert: the group's rank is that expert's
    ids, _ = P.route(h, w, "r", {"experts": 12, "top": 2, "groups": {"count": 12, "keep": 5}})
    assert all(ids[t].tolist() == c[t].topk(2).indices.tolist() for t in range(40))


def test_plain_experts_are_gelu_layers_weighed_on_their_outputs():
    g = torch.Generator().manual_seed(1)
    w = {"f.router": torch.randn(4, 5, dtype=F, generator=g), "f.correction": torch.zeros(4, dtype=F)}
    for e in range(4):
        w[f"f.e{e}.up"] = torch.randn(8, 5, dtype=F, generator=g)
        w[f"f.e{e}.down"] = torch.randn(5, 8, dtype=F, generator=g)
    h = torch.randn(6, 5, dtype=F, generator=g)
    mlp = {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 4, "top": 2, "groups": {"count": 1, "keep": 1}}}
    out = P.experts_ff(h, w, "f", mlp, False)
    ids, weights = P.route(h, w, "f", mlp["router"])
    for t in range(6):
        want = sum(s * (torch.nn.functional.gelu(h[t] @ w[f"f.e{e}.up"].T) @ w[f"f.e{e}.down"].T)
                   for e, s in zip(ids[t].tolist(), weights[t]))
        assert torch.allclose(out[t], want, atol=1e-12)


def test_plain_forward_runs_every_configuration_and_prefixes_agree(tmp_path):
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        d = make_model(str(tmp_path / name), cfg, 20 + i)
        w = load_weights(d, False)
        n = 40 if cfg is not HEADS_64 else 20
        toks = [(7 * t + 3) % cfg["vocab"] for t in range(n)]
        layers = []
        full = P.forward(toks, w, read_config(d), layers_out=layers)
        assert full.shape == (n, cfg["vocab"]) and torch.isfinite(full).all()
        assert len(layers) == len(P.run_order(cfg))
        part = P.forward(toks[:17], w, cfg)
        assert torch.allclose(full[:17], part, atol=1e-9)  # causal throughout
        both = P.forward(toks, w, cfg, emulate_bf16=True)
        assert 1e-6 < float((both - full).abs().max())
