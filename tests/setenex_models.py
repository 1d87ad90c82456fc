"""Small Setenex configurations and model folders for the tests.  The sizes differ between them in
everything, none is a power-of-two family throughout, and each choice of the design appears in several
values: one and several key/value heads, one to eight query heads a key/value head, keys and values of
unequal sizes, distance tables of two rows to many with near and far ends, windows of one token, shorter than a
page, of a page and a token, and longer than the prompts, no first tokens kept, a few, a page of them and
more than a page, latents with and without a rotated part, rotations over a part of it, layers with and
without experts, routers with one group, with groups of one expert, and with some groups left out; loops
over the first layers, the middle, all of them, one pass, and none."""
from __future__ import annotations

import json
import os
from typing import Dict

import torch


def attention(heads, kv_heads, dim, vdim, window, keep, scale, bias_max, rows):
    """A mixer of type "attention"; ``rows`` of its distance table is no configuration key (the stored
    tensor has it) and is taken out by ``config``."""
    return ("attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                          "bias_max": bias_max, "mask": {"size": window, "keep_first": keep}, "rows": rows})


def latent(heads, dim, rot_dim, vdim, kv_rank, window, scale, base=10000.0, dims=None):
    return ("latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                 "scale": scale, "mask": {"size": window},
                                 "rot": {"base": base, "dims": rot_dim if dims is None else dims}})


def moe(experts, top, ff, count=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def config(vocab, width, eps, layers, loop=None, scale=1.0):
    """``layers``: (mixer, mlp) pairs.  The tables' row numbers stand under "rows" of the result, which
    ``make_model`` takes out of what it writes."""
    entries, rows = [], {}
    for i, ((kind, mixer), mlp) in enumerate(layers):
        mixer = dict(mixer)
        if kind == "attention":
            rows[i] = mixer.pop("rows")
        entries.append({"type": kind, "mixer": mixer, "mlp": mlp})
    cfg = {"architecture": "Setenex", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "embedding": {"scale": scale}, "layers": entries, "rows": rows}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


# both mixers, a loop over the middle layers three times
MIXED = config(307, 96, 1e-5, [
    (attention(4, 2, 24, 40, 50, 5, 0.3, 100, 12), moe(6, 2, 24, 3, 2)),
    (latent(3, 20, 8, 24, 48, 33, 0.25, 500.0), moe(8, 3, 16, 4, 2)),
    (attention(6, 2, 16, 16, 9, 70, 0.4, 33, 9), None),
    (latent(5, 12, 12, 8, 32, 200, 0.3, 50.0, dims=6), moe(5, 2, 40)),
], loop=(1, 3, 3), scale=3.0)
# sizes that are no multiples of eight or four; no loop; a window of one token; a latent without rotation
ODD = config(211, 76, 1e-6, [
    (attention(3, 3, 11, 34, 64, 64, 0.4, 40, 7), moe(3, 1, 20, 3, 2)),
    (latent(2, 9, 6, 10, 27, 1, 0.4), moe(7, 4, 12)),
    (attention(5, 1, 18, 6, 1, 3, 0.2, 2, 2), None),
    (latent(4, 7, 0, 13, 20, 65, 0.5), moe(12, 5, 8, 4, 3)),
    (attention(2, 1, 7, 9, 33, 0, 0.7, 300, 33), moe(4, 4, 28, 2, 2)),
], scale=0.5)
# the whole model is one loop, passed twice
LOOP_ALL = config(150, 64, 1e-5, [
    (attention(8, 1, 12, 24, 30, 2, 0.5, 64, 16), moe(4, 2, 16, 2, 1)),
    (latent(2, 16, 4, 40, 24, 70, 0.3, 100.0), moe(9, 3, 8, 3, 2)),
], loop=(0, 2, 2), scale=2.0)
# a loop of one pass over the last layer (its row is still added)
LOOP_ONCE = config(150, 72, 1e-5, [
    (latent(1, 8, 2, 8, 16, 40, 0.5), moe(2, 1, 48, 2, 1)),
    (attention(2, 2, 20, 12, 100, 130, 0.35, 500, 24), moe(3, 3, 24)),
], loop=(1, 2, 1))
# attention made sharp: large scores, so that most of a query's weight lies on one key (experts in the last
# layer only: a router's close call at one position must not reach others through such keys)
SHARP = config(150, 64, 1e-5, [
    (attention(4, 2, 16, 16, 300, 10, 1.2, 200, 16), None),
    (latent(2, 24, 8, 8, 32, 129, 0.7, 100.0), None),
    (attention(2, 2, 8, 32, 64, 66, 2.0, 30, 6), moe(4, 2, 40, 2, 1))])
# sizes of the tensor-core kernels: heads of 64 and 128, padded ones, latents of more and less than a run
HEADS_64 = config(150, 64, 1e-5, [
    (attention(4, 2, 64, 64, 100, 12, 0.15, 90, 16), moe(4, 2, 64, 2, 1)),
    (latent(4, 32, 16, 64, 128, 70, 0.2), moe(6, 2, 64, 3, 1)),
    (attention(2, 1, 128, 128, 500, 0, 0.1, 128, 32), None),
    (attention(6, 2, 40, 72, 64, 65, 0.2, 1000, 20), None),
    (attention(3, 1, 96, 56, 80, 3, 0.12, 60, 10), None),
    (latent(2, 16, 32, 40, 272, 150, 0.2, 3000.0), None)], loop=(1, 3, 2), scale=4.0)
CONFIGS: Dict[str, dict] = {"mixed": MIXED, "odd": ODD, "loop_all": LOOP_ALL, "loop_once": LOOP_ONCE,
                            "sharp": SHARP, "heads64": HEADS_64}


def written(cfg: dict) -> dict:
    """The configuration as config.json has it."""
    return {k: v for k, v in cfg.items() if k != "rows"}


def make_model(tmp_dir: str, cfg: dict, seed: int) -> str:
    """A model folder with random weights whose activations and scores are of order one.
    Tensors that random numbers around zero would make harmless are moved to where they matter:
    distance tables with clearly different rows (as many as the configuration's "rows" says), the routers'
    corrections large enough to change choices and to make choice scores negative, the loop's rows of the
    size of the embedding, norm weights some way off their centre."""
    from nnis_b200.weights import write_random_model
    from safetensors.torch import load_file, save_file
    write_random_model(written(cfg), seed, tmp_dir, std=1.0, norm_std=0.1, std_by_fan_in=True)
    path = os.path.join(tmp_dir, "model.safetensors")
    w = load_file(path)
    g = torch.Generator().manual_seed(seed + 1)
    for name in sorted(w):
        t = w[name].float()
        if name.endswith(".rel"):
            layer = int(name.split(".")[0][1:])
            t = torch.randn((cfg["rows"][layer], t.shape[1]), generator=g)
        elif name.endswith(".correction"):
            t = torch.empty_like(t).uniform_(-1.1, 0.1, generator=g)
        elif name.endswith(".router"):
            t = torch.randn(t.shape, generator=g) * (2.0 / t.shape[1] ** 0.5)
        elif name.endswith((".q.norm", ".k.norm", ".dkv.norm")):
            t = torch.empty_like(t).uniform_(0.6, 1.5, generator=g)
        elif "norm" in name:
            t = torch.empty_like(t).uniform_(-0.4, 0.4, generator=g)
        elif name == "loop.step":
            t = torch.randn(t.shape, generator=g) * 0.7
        elif name == "embed":
            t = torch.randn(t.shape, generator=g) * 0.5
        w[name] = t.to(torch.bfloat16)
    save_file(w, path)
    return tmp_dir


def load_weights(model_dir: str, as_bf16: bool):
    from safetensors.torch import load_file
    w = load_file(os.path.join(model_dir, "model.safetensors"))
    return {k: (v.to(torch.bfloat16).double() if as_bf16 else v.double()) for k, v in w.items()}


def read_config(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)
