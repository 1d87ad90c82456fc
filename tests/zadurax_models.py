"""Small Zadurax configurations and model folders for the tests.  The sizes differ between them in
everything, none is a power-of-two family throughout, and each choice of the design appears in several
values: one and several key/value heads, windows of one token, shorter than a page, of a page and a
token, and longer than the prompts, rotations over all, a part and none of a head, frequencies with and
without a ramp, latents with and without a rotated part, memories whose keys are smaller and larger than
their values, caps from small to large, layers with and without a feed-forward, layers that use another's
weights (once, twice, by way of a layer that does so too), and none."""
from __future__ import annotations

import json
import os
from typing import Dict

import torch


def attention(heads, kv_heads, dim, window, scale, base=10000.0, dims=None):
    return ("attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                          "mask": {"size": window}, "rot": {"base": base, "dims": dim // 2 * 2 if dims is None else dims}})


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, scaling=None):
    """``scaling``: (factor, original, fast, slow)."""
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return ("latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                 "scale": scale, "rot": rot})


def memory(heads, dim, vdim, cap):
    return ("mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap})


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(vocab, width, eps, layers):
    """``layers``: (mixer, mlp) pairs, or the number of the layer whose weights are used."""
    entries = []
    for layer in layers:
        if isinstance(layer, int):
            entries.append({**entries[layer], "weights_of": layer})
        else:
            (kind, mixer), mlp = layer
            entries.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Zadurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": entries}


# all three mixers; the memory's weights twice more, once by way of the layer that uses them already
MIXED = config(307, 96, 1e-5, [
    (attention(4, 2, 24, 50, 0.3, 500.0, 10), dense(120)),
    (memory(3, 20, 28, 6.0), dense(72)),
    (latent(5, 12, 8, 16, 32, 0.3, 300.0, (5.0, 60, 6.0, 0.7)), dense(136)),
    1,
    (attention(6, 1, 16, 9, 0.5, 50.0), None),
    3,
    2,
])
# sizes that are no multiples of eight or four; windows of one token and of a page and one
ODD = config(211, 76, 1e-6, [
    (memory(5, 9, 13, 20.0), None),
    (attention(3, 3, 11, 65, 0.4, 40.0, 6), dense(50)),
    (latent(2, 9, 6, 10, 27, 0.4, 1000.0), dense(33)),
    (memory(1, 34, 7, 2.5), dense(20)),
    (attention(5, 5, 6, 1, 0.2), dense(41)),
    (latent(4, 7, 0, 13, 20, 0.5), None),
    2,
    (attention(2, 1, 7, 33, 0.7, 100.0, 0), dense(12)),
])
# every later layer runs with the first two layers' weights
SHARED = config(150, 64, 1e-5, [
    (latent(2, 16, 12, 40, 24, 0.3, 100.0, (2.0, 30, 4.0, 1.0)), dense(88)),
    (memory(8, 12, 24, 9.0), dense(64)),
    0, 1, 2, 1,
])
# memories alone: keys longer than values, a cap that flattens most gates, several chunks of state
MEMORIES = config(131, 72, 1e-5, [
    (memory(2, 40, 12, 1.0), dense(40)),
    (memory(3, 16, 68, 15.0), dense(56)),
    0,
])
# attention made sharp: large scores, so that most of a query's weight lies on one key
SHARP = config(150, 64, 1e-5, [
    (attention(4, 2, 16, 300, 1.1, 200.0, 4), dense(64)),
    (latent(2, 24, 8, 8, 32, 0.8, 100.0, (3.0, 50, 5.0, 1.0)), None),
    (attention(2, 2, 8, 64, 1.6, 1000.0, 2), dense(40)),
])
# sizes of the tensor-core kernels: heads of 64 and 128, padded ones, latents of more and less than a run
HEADS_64 = config(150, 64, 1e-5, [
    (attention(4, 2, 64, 100, 0.15, 5000.0, 32), dense(128)),
    (latent(4, 32, 16, 64, 128, 0.2, 3000.0, (8.0, 100, 8.0, 1.0)), dense(64)),
    (memory(2, 64, 128, 12.0), dense(96)),
    (attention(2, 1, 128, 500, 0.1), None),
    (latent(2, 16, 32, 40, 272, 0.2, 3000.0), dense(64)),
    (memory(3, 72, 136, 8.0), None),
    (attention(6, 2, 40, 64, 0.2, 900.0, 20), dense(64)),
    (memory(1, 136, 64, 10.0), dense(64)),
    2,
])
CONFIGS: Dict[str, dict] = {"mixed": MIXED, "odd": ODD, "shared": SHARED, "memories": MEMORIES, "sharp": SHARP,
                            "heads64": HEADS_64}


def make_model(tmp_dir: str, cfg: dict, seed: int) -> str:
    """A model folder with random weights whose activations and scores are of order one.
    Tensors that random numbers around zero would make harmless are moved to where they matter:
    sinks that take a good part of a softmax, forget gates that keep some heads' memory for hundreds
    of tokens and others' for a few, norm weights some way off one.

    A memory's output is divided by max(|n . q|, exp(-m)) and then by its own size, so where n . q passes
    through zero its direction turns round: no rounding however small may be expected to agree there.
    The embeddings therefore share a direction that the memories' q and k respond to alike, which keeps
    n . q well away from zero (the kernels' own tests meet it on both sides)."""
    from nnis_b200.weights import write_random_model
    from safetensors.torch import load_file, save_file
    write_random_model(cfg, seed, tmp_dir, std=1.0, norm_std=0.1, std_by_fan_in=True)
    path = os.path.join(tmp_dir, "model.safetensors")
    w = load_file(path)
    g = torch.Generator().manual_seed(seed + 1)
    shared = torch.randn(cfg["width"], generator=g).sign() * 0.5
    for name in sorted(w):
        t = w[name].float()
        layer = cfg["layers"][int(name[1:].split(".")[0])] if name[0] == "l" else {"type": ""}
        if name.endswith(".sink"):
            t = torch.empty_like(t).uniform_(-1.0, 2.5, generator=g)
        elif name.endswith(".mix.f.b"):
            t = torch.empty_like(t).uniform_(-1.0, 6.0, generator=g)
        elif name.endswith(".mix.i.b"):
            t = torch.empty_like(t).uniform_(-3.0, 3.0, generator=g)
        elif name.endswith((".mix.i", ".mix.f")):
            t = torch.randn(t.shape, generator=g) * (1.5 / t.shape[1] ** 0.5)
        elif name.endswith((".norm1b", ".norm2b")):  # (so that the shared direction is still there in late layers)
            t = torch.empty_like(t).uniform_(0.2, 0.5, generator=g)
        elif "norm" in name:
            t = torch.empty_like(t).uniform_(0.6, 1.5, generator=g)
        elif name == "embed":
            t = torch.randn(t.shape, generator=g) * 0.5 + shared
        elif layer["type"] == "mlstm" and name.endswith((".mix.q", ".mix.k")):
            m = layer["mixer"]
            gq = torch.Generator().manual_seed(seed + int(name[1:].split(".")[0]))  # q's and k's answer is the same
            answer = torch.randn(m["heads"] * m["dim"], generator=gq).sign() * 0.45 * max(1.0, (12 / m["dim"]) ** 0.5)
            t = t + answer[:, None] * shared / shared.norm()
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
