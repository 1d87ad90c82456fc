"""Zadurax without a GPU: configuration round trip and errors by key, layers that use another's
weights, tensor names, what the design asks of the cache, the chunks of a matrix memory's prompt, and
the plain mechanisms against closed forms."""
import copy
import math

import pytest
import torch

import plain_zadurax as P
from zadurax_models import (CONFIGS, HEADS_64, MIXED, ODD, SHARED, attention, config, dense, latent, load_weights,
                            make_model, memory, read_config)

F = torch.float64
KINDS = {"attention": "sink_attention", "latent_attention": "latent_attention", "mlstm": "matrix_memory"}


def test_configuration_round_trip_and_spec():
    from nnis_b200.config import config_from_dict, known_architectures
    assert "Zadurax" in known_architectures()
    for cfg in CONFIGS.values():
        typed = config_from_dict(cfg)
        assert typed.to_dict() == cfg and config_from_dict(typed.to_dict()).to_dict() == cfg
        spec = typed.to_spec()
        own = [i for i, l in enumerate(cfg["layers"]) if "weights_of" not in l]
        assert [l.prefix for l in spec.layers] == [f"l{i}" for i in own]
        for i, layer in zip(own, spec.layers):
            assert layer.block == "sandwich" and layer.part("mixer").kind == KINDS[cfg["layers"][i]["type"]]
            assert ("ffn" in layer.parts) == (cfg["layers"][i]["mlp"] is not None)
        assert spec.head.get("tied_to") is None
    spec = config_from_dict(MIXED).to_spec()
    a = spec.layers[0].part("mixer")
    assert (a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["window"], a["scale"]) == (4, 2, 24, 24, 50, 0.3)
    assert a["values"] == "keys" and a["gate"] == "value" and a["qk_norm"] == "head_weight" and a.get("sink") is None
    assert (a["position"]["dims"], a["position"]["base"], a["position"]["pairing"]) == (10, 500.0, "neighbours")
    b = spec.layers[2].part("mixer")
    assert (b["heads"], b["dim"], b["rot_dim"], b["vdim"], b["kv_rank"], b["scale"]) == (5, 12, 8, 16, 32, 0.3)
    assert b["sink"] and b["gate"] == "value" and not b.get("window") and b["q_rank"] == 0
    assert b["position"]["scaling"] == {"ramp": "index", "factor": 5.0, "original": 60, "fast": 6.0, "slow": 0.7}
    m = spec.layers[1].part("mixer")
    assert (m["heads"], m["dim"], m["vdim"], m["gate_cap"], m["eps"]) == (3, 20, 28, 6.0, 1e-5)
    f = spec.layers[1].part("ffn")
    assert (f["intermediate_size"], f["activation"]) == (72, "gelu_tanh")


def test_layers_that_use_anothers_weights_are_entries_of_the_schedule():
    from nnis_b200.config import config_from_dict
    spec = config_from_dict(MIXED).to_spec()
    assert [l.prefix for l in spec.layers] == ["l0", "l1", "l2", "l4"]
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 1, 3, 1, 2]
    assert all(e.cache_of is None and e.enter is None for e in spec.schedule)  # a cache per run
    assert [e.layer for e in config_from_dict(SHARED).to_spec().schedule] == [0, 1, 0, 1, 0, 1]
    # a layer may also use the weights of a later one
    cfg = config(50, 32, 1e-5, [(memory(2, 8, 8, 5.0), None), (attention(2, 1, 8, 5, 0.3), dense(16)),
                                (memory(2, 8, 8, 5.0), None)])
    cfg["layers"][0]["weights_of"] = 2
    spec = config_from_dict(cfg).to_spec()
    assert [l.prefix for l in spec.layers] == ["l1", "l2"] and [e.layer for e in spec.schedule] == [1, 0, 1]
    assert [P.owner(MIXED, i) for i in range(7)] == [0, 1, 2, 1, 4, 1, 2] and P.owner(cfg, 0) == 2


@pytest.mark.parametrize("change, word", [
    (lambda c: c.update(architecture="Other"), "architecture"),
    (lambda c: c["layers"][0].update(type="conv"), "not a mixer"),
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "multiple"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=20), "vdim"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][4]["mixer"].pop("kv_heads"), "kv_heads"),
    (lambda c: c["layers"][2]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(base=1.0), "base"),
    (lambda c: c["layers"][1]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].update(dim=0), "dim"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "dense"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][3].update(weights_of=9), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=3), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=0), "differs"),
    (lambda c: c["layers"][1].update(weights_of=5), "each other"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(layers=[]), "at least one layer"),
])
def test_configuration_errors_name_the_key(change, word):
    from nnis_b200.config import ConfigError, config_from_dict
    cfg = copy.deepcopy(MIXED)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    assert word in str(e.value)


def test_tensor_names_and_shapes(tmp_path):
    from nnis_b200.config import config_from_dict
    from nnis_b200.engine.model import DecoderModel
    from nnis_b200.weights import load_weights as product_load
    specs = DecoderModel.weight_specs_of(config_from_dict(MIXED).to_spec())
    shapes = {n: tuple(s.shape) for n, s in specs.items() if s.role != "unused"}
    assert shapes["embed"] == shapes["head"] == (307, 96)
    assert shapes["embed.norm"] == shapes["final.norm"] == shapes["l0.norm1"] == shapes["l2.norm2b"] == (96,)
    assert shapes["l0.mix.q"] == shapes["l0.mix.g"] == (96, 96) and shapes["l0.mix.k"] == (48, 96)
    assert shapes["l0.mix.q.norm"] == shapes["l0.mix.k.norm"] == (24,) and shapes["l0.mix.o"] == (96, 96)
    assert "l0.mix.v" not in shapes and "l0.mix.sink" not in shapes
    assert shapes["l1.mix.q"] == shapes["l1.mix.k"] == (60, 96) and shapes["l1.mix.v"] == shapes["l1.mix.g"] == (84, 96)
    assert shapes["l1.mix.i"] == shapes["l1.mix.f"] == (3, 96) and shapes["l1.mix.i.b"] == shapes["l1.mix.f.b"] == (3,)
    assert shapes["l1.mix.norm"] == (84,) and shapes["l1.mix.o"] == (96, 84)
    assert shapes["l2.mix.q"] == (100, 96) and shapes["l2.mix.dkv"] == (40, 96) and shapes["l2.mix.dkv.norm"] == (32,)
    assert shapes["l2.mix.uk"] == (60, 32) and shapes["l2.mix.uv"] == (80, 32) and shapes["l2.mix.sink"] == (5,)
    assert shapes["l2.mix.g"] == (80, 96) and shapes["l2.mix.o"] == (96, 80)
    assert shapes["l1.mlp.gate"] == shapes["l1.mlp.up"] == (72, 96) and shapes["l1.mlp.down"] == (96, 72)
    # no feed-forward: no norms around it (a folder may hold them all the same); no tensors under a sharing layer's name
    assert "l4.mlp.gate" not in shapes and "l4.norm2" not in shapes and specs["l4.norm2b"].role == "unused"
    assert not any(n.startswith(("l3.", "l5.", "l6.")) for n in specs)
    d = make_model(str(tmp_path / "m"), MIXED, 3)
    assert set(load_weights(d, False)) == set(shapes)
    model = DecoderModel(config_from_dict(read_config(d)).to_spec(), torch.float32, torch.device("cpu"))
    model.load(product_load(d, specs, torch.float32, torch.device("cpu")))
    # the memory's input product: q, k, v, g and both gates, rows up to a multiple of eight
    m = model.blocks[1].mixer
    assert m.w_in.shape == (2 * 60 + 2 * 84 + 6 + 2, 96) and (m.w_in[-2:] == 0).all() and m.gate_off == 120 + 84


def test_what_the_design_asks_of_the_cache():
    from nnis_b200.cache import CacheManager, KVRequest, SlotError, StateRequest
    from nnis_b200.config import config_from_dict
    from nnis_b200.engine.model import DecoderModel
    model = DecoderModel(config_from_dict(MIXED).to_spec(), torch.float32, torch.device("cpu"))
    requests = model.cache_requests()
    assert len(requests) == 7 + 1 and requests[-1] is None
    assert requests[0] == KVRequest(2, 24, 50, True, 24) and requests[4] == KVRequest(1, 16, 9, True, 16)
    assert requests[2] == requests[6] == KVRequest(1, 40, 0, values=False)
    assert requests[1] == requests[3] == requests[5] == StateRequest(
        (3, 20, 28), torch.float32, extra=(((2, 3, 20), torch.float32), ((2, 3), torch.float32)))
    cache = CacheManager(requests, torch.bfloat16, torch.device("cpu"), 64 * 8, 4, 1 << 20)
    views = [cache.view(i) for i in (1, 3, 5)]
    assert len({v.state.data_ptr() for v in views}) == 3  # a state per run of the layer
    assert all(t.dtype == torch.float32 for v in views for t in (v.state, *v.extra))
    slot = cache.acquire()
    for v in views:
        for t in (v.state, *v.extra):
            t[slot].fill_(3.0)
    cache.reserve([slot], [5])
    cache.commit([slot], [5])
    kept = cache.snapshot(slot)
    views[0].extra[1][slot].fill_(9.0)
    cache.reserve([slot], [7])
    cache.commit([slot], [7])
    with pytest.raises(SlotError):  # a state has no earlier value ...
        cache.truncate(slot, 5)
    cache.restore(kept)             # ... but a snapshot has
    assert (views[0].extra[1][slot] == 3.0).all() and cache.length(slot) == 5
    cache.release(slot)
    assert cache.acquire() == slot
    assert all((t[slot] == 0).all() for v in views for t in (v.state, *v.extra))  # a slot used again starts from nothing


# ---- the plain mechanisms against closed forms ---------------------------------------------------
def _mixer(cfg, index, tmp_path, seed=5, T=12, **changes):
    cfg = copy.deepcopy(cfg)
    m = cfg["layers"][index]["mixer"]
    m.update(changes)
    d = make_model(str(tmp_path / "m"), config(50, cfg["width"], 1e-5, [((cfg["layers"][index]["type"], m), None)]), seed)
    w = load_weights(d, False)
    h = torch.randn(T, cfg["width"], dtype=F, generator=torch.Generator().manual_seed(1))
    probe = {}
    return m, w, h, P.MIXERS[cfg["layers"][index]["type"]](h, w, "l0.mix", m, 1e-5, False, probe), probe


@pytest.mark.parametrize("size", [1, 3, 11, 12, 100])
def test_plain_attention_sees_a_window(size, tmp_path):
    _, _, _, _, probe = _mixer(MIXED, 0, tmp_path, mask={"size": size})
    for a in probe["weights"]:
        for i in range(12):
            assert [j for j in range(12) if a[i, j] > 0] == list(range(max(0, i - size + 1), i + 1))
            assert abs(a[i].sum() - 1) < 1e-12


def test_plain_attention_takes_the_raw_keys_as_values_and_gates_every_value(tmp_path):
    m, w, h, out, probe = _mixer(MIXED, 0, tmp_path, mask={"size": 5})
    q = (h @ w["l0.mix.q"].T).view(12, 4, 24)
    k = (h @ w["l0.mix.k"].T).view(12, 2, 24)

    def turned(x, weight, p):  # one head at position p
        x = x / torch.sqrt((x ** 2).mean() + 1e-5) * weight
        y = x.clone()
        for i in range(5):
            a = p * 500.0 ** (-2 * i / 10)
            y[2 * i] = x[2 * i] * math.cos(a) - x[2 * i + 1] * math.sin(a)
            y[2 * i + 1] = x[2 * i + 1] * math.cos(a) + x[2 * i] * math.sin(a)
        return y
    heads = []
    for a in range(4):
        rows = torch.zeros(12, 12, dtype=F)
        for i in range(12):
            for j in range(max(0, i - 4), i + 1):
                rows[i, j] = math.exp(float(turned(q[i, a], w["l0.mix.q.norm"], i)
                                            @ turned(k[j, a // 2], w["l0.mix.k.norm"], j)) * 0.3)
        rows = rows / rows.sum(-1, keepdim=True)
        assert torch.allclose(rows, probe["weights"][a], atol=1e-12)
        heads.append(rows @ k[:, a // 2])
    gated = torch.cat(heads, -1) / (1.0 + torch.exp(-h @ w["l0.mix.g"].T))
    assert torch.allclose(out, gated @ w["l0.mix.o"].T, atol=1e-12)


def test_plain_frequencies_blend_by_index():
    rot = {"base": 300.0, "dims": 16, "scaling": {"factor": 5.0, "original": 60, "fast": 6.0, "slow": 0.7}}
    freq, size = P.turning_rates(rot)
    assert abs(size - (1.0 + 0.1 * math.log(5.0))) < 1e-15
    at = lambda turns: 16 * math.log(60 / (turns * 2 * math.pi)) / (2 * math.log(300.0))
    lo, hi = max(math.floor(at(6.0)), 0), min(math.ceil(at(0.7)), 15)
    assert (lo, hi) == (0, 4)
    for i, f in enumerate(freq):
        plain = 300.0 ** (-i / 8)
        share = min(1.0, i / 4)
        assert abs(f - (plain * (1 - share) + plain / 5.0 * share)) < 1e-15
    assert freq[0] == 1.0 and P.turning_rates({"base": 300.0, "dims": 16}) == ([300.0 ** (-2.0 * i / 16) for i in range(8)], 1.0)
    # both ends of the ramp at one index: a step
    freq, _ = P.turning_rates({"base": 300.0, "dims": 16, "scaling": {"factor": 5.0, "original": 60, "fast": 1e6, "slow": 1e5}})
    assert abs(freq[0] - 1.0) < 1e-15 and abs(freq[1] - 300.0 ** (-1 / 8) / 5.0) < 1e-15


def test_the_product_makes_the_same_frequencies():
    from nnis_b200.parts import POSITIONS
    from nnis_b200.config.zadurax import ZaduraxConfig
    for rot in (MIXED["layers"][2]["mixer"]["rot"], HEADS_64["layers"][1]["mixer"]["rot"], HEADS_64["layers"][4]["mixer"]["rot"],
                {"base": 300.0, "dims": 16, "scaling": {"factor": 5.0, "original": 60, "fast": 1e6, "slow": 1e5}}):
        spec = ZaduraxConfig._position(rot)
        part = POSITIONS.build(spec.kind, spec.params, "", torch.float32, torch.device("cpu"))
        want, size = P.turning_rates(rot)
        assert torch.allclose(part.frequencies()[:len(want)].double(), torch.tensor(want, dtype=F), rtol=2e-7)
        assert abs(part.magnitude - size) < 1e-12


def test_plain_latent_attention_is_attention_over_what_the_latent_gives(tmp_path):
    m, w, h, out, probe = _mixer(MIXED, 2, tmp_path)
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    down = h @ w["l0.mix.dkv"].T
    c = down[:, :rank] / torch.sqrt((down[:, :rank] ** 2).mean(-1, keepdim=True) + 1e-5) * w["l0.mix.dkv.norm"]
    q = (h @ w["l0.mix.q"].T).view(12, H, d + r)
    kr = P.rotate(down[:, None, rank:], m["rot"])[:, 0]
    heads = []
    for a in range(H):
        k, v = c @ w["l0.mix.uk"][a * d:(a + 1) * d].T, c @ w["l0.mix.uv"][a * dv:(a + 1) * dv].T
        s = (q[:, a, :d] @ k.T + P.rotate(q[:, a:a + 1, d:], m["rot"])[:, 0] @ kr.T) * m["scale"]
        e = torch.exp(s) * torch.ones(12, 12, dtype=F).tril()
        p = e / (e.sum(-1, keepdim=True) + math.exp(float(w["l0.mix.sink"][a])))
        assert torch.allclose(p, probe["weights"][a], atol=1e-12)
        assert float(p.sum(-1).max()) < 0.9995  # the sink takes its part
        heads.append(p @ v)
    gated = torch.cat(heads, -1) / (1.0 + torch.exp(-h @ w["l0.mix.g"].T))
    assert torch.allclose(out, gated @ w["l0.mix.o"].T, atol=1e-12)
    # a turned vector is longer by the magnitude, the plain part is not
    x = torch.randn(6, 1, r, dtype=F)
    assert torch.allclose(P.rotate(x, m["rot"]).norm(dim=-1), x.norm(dim=-1) * (0.1 * math.log(5.0) + 1.0))


def test_plain_memory_is_a_weighted_sum_over_the_tokens_so_far():
    """Without the running maximum: token s counts exp(i_s + f_s+1 + .. + f_t) at token t, and the
    denominator is max(|n . q|, 1) in those terms plus 1e-6 times exp(m)."""
    g = torch.Generator().manual_seed(2)
    T, H, d, dv = 30, 3, 5, 4
    q, k = torch.randn(T, H, d, dtype=F, generator=g), torch.randn(T, H, d, dtype=F, generator=g)
    v = torch.randn(T, H, dv, dtype=F, generator=g)
    i = torch.randn(T, H, dtype=F, generator=g) * 3
    f = torch.nn.functional.logsigmoid(torch.randn(T, H, dtype=F, generator=g) * 3)
    out = P.matrix_memory(q, k, v, i, f)
    below_one = 0
    for h in range(H):
        m = 0.0
        for t in range(T):
            m = max(float(f[t, h]) + m, float(i[t, h]))
            c = torch.stack([torch.exp(i[s, h] + f[s + 1:t + 1, h].sum()) for s in range(t + 1)])
            dots = k[:t + 1, h] @ q[t, h]
            n = float((c * dots).sum())
            below_one += abs(n) < 1
            bottom = max(abs(n), 1.0) + 1e-6 * math.exp(m)
            assert torch.allclose(out[t, h], ((c * dots)[:, None] * v[:t + 1, h]).sum(0) / bottom, atol=1e-10)
    assert 0 < below_one < T * H  # both sides of the maximum were met


def test_plain_memory_mixer_caps_its_gates_and_norms_its_heads(tmp_path):
    m, w, h, out, _ = _mixer(MIXED, 1, tmp_path)
    H, d, dv, cap = 3, 20, 28, 6.0
    q, k = (h @ w["l0.mix.q"].T).view(12, H, d) / math.sqrt(d), (h @ w["l0.mix.k"].T).view(12, H, d)
    v = (h @ w["l0.mix.v"].T).view(12, H, dv)
    i = cap * torch.tanh((h @ w["l0.mix.i"].T + w["l0.mix.i.b"]) / cap)
    f = -torch.log1p(torch.exp(-cap * torch.tanh((h @ w["l0.mix.f"].T + w["l0.mix.f.b"]) / cap)))
    assert float(i.abs().max()) < cap and float(f.max()) < 0
    o = P.matrix_memory(q, k, v, i, f)
    o = (o / torch.sqrt((o ** 2).mean(-1, keepdim=True) + 1e-5)).reshape(12, -1) * w["l0.mix.norm"]
    assert torch.allclose(out, (o / (1.0 + torch.exp(-h @ w["l0.mix.g"].T))) @ w["l0.mix.o"].T, atol=1e-12)


def test_plain_feed_forward_is_a_gated_gelu():
    g = torch.Generator().manual_seed(1)
    w = {f"f.{n}": torch.randn(s, dtype=F, generator=g) for n, s in (("gate", (8, 5)), ("up", (8, 5)), ("down", (5, 8)))}
    h = torch.randn(6, 5, dtype=F, generator=g)
    want = (torch.nn.functional.gelu(h @ w["f.gate"].T, approximate="tanh") * (h @ w["f.up"].T)) @ w["f.down"].T
    assert torch.allclose(P.dense(h, w, "f", False), want, atol=1e-12)


def test_chunks_cover_every_sequence_once():
    from nnis_b200.csrc import ops
    chunks, first = ops.scan_segments([64, 1, 130, 63], 64)
    assert chunks.tolist() == [[0, 0], [1, 0], [2, 0], [2, 64], [2, 128], [3, 0]] and first.tolist() == [0, 1, 2, 5, 6]


def test_plain_forward_runs_every_configuration_and_prefixes_agree(tmp_path):
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        d = make_model(str(tmp_path / name), cfg, 20 + i)
        w = load_weights(d, False)
        assert read_config(d) == cfg
        n = 40 if cfg is not HEADS_64 else 20
        toks = [(7 * t + 3) % cfg["vocab"] for t in range(n)]
        layers = []
        full = P.forward(toks, w, cfg, layers_out=layers)
        assert full.shape == (n, cfg["vocab"]) and torch.isfinite(full).all()
        assert len(layers) == len(cfg["layers"])
        assert torch.allclose(full[:17], P.forward(toks[:17], w, cfg), atol=1e-9)  # causal throughout
        assert 1e-6 < float((P.forward(toks, w, cfg, emulate_bf16=True) - full).abs().max())
    assert ODD["layers"][6]["weights_of"] == 2
