"""Setenex, plainly: whole sequences, no cache, no batches, float64, one function per
mechanism, written from the design's equations.  It reads config.json's keys and the
tensor names by itself and shares no code with the package.

``emulate_bf16`` rounds where the bfloat16 engine rounds (the normed rows that feed the
projections, q and the cached k and v after their norms, the latent and the rotated key part,
the queries carried into the latent's space and the weighted sums there, the heads before the
output projection, the experts' activations); norms, angles, scores, distance biases, softmax,
gates, routers and the residual sum stay exact.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def bf(x: torch.Tensor, on: bool) -> torch.Tensor:
    return x.to(torch.bfloat16).to(F) if on else x


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The stored weight lies around zero: the multiplier is 1 + w."""
    return rms(x, eps) * (1.0 + w.to(F))


def plain_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * w.to(F)


# ---- attention with a learned bias per distance -------------------------------------------
def bucket_of(n: int, buckets: int, far: float) -> int:
    """Distances below half the buckets have one each; the others share the second half
    logarithmically up to ``far``.  The edges are compared in whole numbers: n lies at or beyond
    the k-th edge if (n / half)^m >= (far / half)^k, m buckets in the second half."""
    half = buckets // 2
    if n < half:
        return n
    m = buckets - half
    k = 0
    while k < m - 1 and n ** m * half ** (k + 1) >= int(far) ** (k + 1) * half ** m:
        k += 1
    return half + k


def bias_of_distances(T: int, table: torch.Tensor, far: float) -> torch.Tensor:
    """[T, T, heads]: the bias of query i and key j (0 where j > i)."""
    rows = [bucket_of(n, table.shape[0], far) for n in range(T)]
    i = torch.arange(T)
    distance = (i[:, None] - i[None, :]).clamp(min=0)
    return table.to(F)[torch.tensor(rows)[distance]]


def kept_window(T: int, size: int, keep_first: int) -> torch.Tensor:
    i = torch.arange(T)
    back = i[:, None] - i[None, :]
    return (back >= 0) & ((back < size) | (i[None, :] < keep_first))


def attention(h, w, p, m, eps, e16, probe=None):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = bf(plain_norm((h @ w[p + ".q"].to(F).T).view(T, H, d), w[p + ".q.norm"], eps), e16)
    k = bf(plain_norm((h @ w[p + ".k"].to(F).T).view(T, G, d), w[p + ".k.norm"], eps), e16)
    v = bf((h @ w[p + ".v"].to(F).T).view(T, G, dv), e16)
    bias = bias_of_distances(T, w[p + ".rel"], m["bias_max"])
    visible = kept_window(T, int(m["mask"]["size"]), int(m["mask"]["keep_first"]))
    out = torch.zeros(T, H, dv, dtype=F)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * float(m["scale"]) + bias[:, :, a]
        weights = torch.softmax(s.masked_fill(~visible, -math.inf), dim=-1)
        if probe is not None:
            probe.setdefault("weights", []).append(weights)
        out[:, a] = weights @ v[:, g]
    return bf(out.reshape(T, H * dv), e16) @ w[p + ".o"].to(F).T


# ---- attention over a latent --------------------------------------------------------------
def rotate_neighbours(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, d], rows at positions 0 ..: value 2i turns with value 2i + 1 by the angle
    position * base^(-2i/dims), for the first ``dims`` values."""
    T = x.shape[0]
    y = x.clone()
    for i in range(dims // 2):
        a = torch.arange(T, dtype=F) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


def latent_attention(h, w, p, m, eps, e16, probe=None):
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m["rot"]
    q = (h @ w[p + ".q"].to(F).T).view(T, H, d + r)
    q_plain = bf(q[..., :d], e16)
    q_rot = bf(rotate_neighbours(q[..., d:], int(rot["dims"]), rot["base"]), e16)
    down = h @ w[p + ".dkv"].to(F).T
    c = bf(plain_norm(down[:, :rank], w[p + ".dkv.norm"], eps), e16)
    k_rot = bf(rotate_neighbours(down[:, rank:].view(T, 1, r), int(rot["dims"]), rot["base"]), e16)[:, 0]
    uk = w[p + ".uk"].to(F).view(H, d, rank)
    uv = w[p + ".uv"].to(F).view(H, dv, rank)
    gates = torch.sigmoid(h @ w[p + ".g"].to(F).T)
    i = torch.arange(T)
    back = i[:, None] - i[None, :]
    visible = (back >= 0) & (back < int(m["mask"]["size"]))
    out = torch.zeros(T, H, dv, dtype=F)
    for a in range(H):
        if e16:  # (the engine scores and sums in the latent's space, with a rounding at each border)
            plain = bf(q_plain[:, a] @ uk[a], e16) @ c.T
        else:
            plain = q_plain[:, a] @ (c @ uk[a].T).T
        s = (plain + q_rot[:, a] @ k_rot.T) * float(m["scale"])
        weights = torch.softmax(s.masked_fill(~visible, -math.inf), dim=-1)
        if probe is not None:
            probe.setdefault("weights", []).append(weights)
        if e16:
            out[:, a] = bf((weights @ c) * gates[:, a:a + 1], e16) @ uv[a].T
        else:
            out[:, a] = (weights @ (c @ uv[a].T)) * gates[:, a:a + 1]
    return bf(out.reshape(T, H * dv), e16) @ w[p + ".o"].to(F).T


# ---- experts ------------------------------------------------------------------------------
def gelu(x):
    return 0.5 * x * (1.0 + torch.erf(x / math.sqrt(2.0)))


def expert(h, w, p, e16):
    return bf(gelu(h @ w[p + ".up"].to(F).T), e16) @ w[p + ".down"].to(F).T


def route(h, w, p, r, probe=None):
    """ids [T, top] and the weights of the chosen (their scores, summing to one)."""
    E, top = int(r["experts"]), int(r["top"])
    s = torch.sigmoid(h @ w[p + ".router"].to(F).T)
    choice = s + w[p + ".correction"].to(F)
    count, keep = int(r["groups"]["count"]), int(r["groups"]["keep"])
    size = E // count
    ids = torch.zeros(h.shape[0], top, dtype=torch.long)
    gaps = []
    for t in range(h.shape[0]):
        value = [float(x) for x in choice[t]]
        strength = [sum(sorted(value[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(count)]
        order = sorted(range(count), key=lambda g: (-strength[g], g))
        kept = set(order[:keep])
        allowed = sorted((e for e in range(E) if e // size in kept), key=lambda e: (-value[e], e))
        ids[t] = torch.tensor(allowed[:top])
        gap = value[allowed[top - 1]] - value[allowed[top]] if len(allowed) > top else math.inf
        if keep < count:
            gap = min(gap, strength[order[keep - 1]] - strength[order[keep]])
        gaps.append(gap)
    if probe is not None:
        # how clearly the choice was made: the last expert chosen against the first one left out, and the groups
        probe.setdefault("gaps", []).append(torch.tensor(gaps, dtype=F))
    chosen = s.gather(1, ids)
    return ids, chosen / (chosen.sum(-1, keepdim=True) + 1e-20)


def experts_ff(h, w, p, mlp, e16, probe=None):
    ids, weights = route(h, w, p, mlp["router"], probe)
    out = torch.zeros(h.shape[0], w[p + ".e0.down"].shape[0], dtype=F)
    for e in range(int(mlp["router"]["experts"])):
        t, s = torch.nonzero(ids == e, as_tuple=True)
        if t.numel():
            out[t] += weights[t, s][:, None] * expert(h[t], w, f"{p}.e{e}", e16)
    return out


# ---- the model ----------------------------------------------------------------------------
MIXERS = {"attention": attention, "latent_attention": latent_attention}


def run_order(cfg: dict) -> List[tuple]:
    """(layer, pass number or None, first of its pass) in the order the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    order = [(i, None, False) for i in range(start)]
    for t in range(times):
        order += [(i, t, i == start) for i in range(start, stop)]
    return order + [(i, None, False) for i in range(stop, n)]


def embedding(tokens: List[int], w: Dict[str, torch.Tensor], cfg: dict) -> torch.Tensor:
    return w["embed"].to(F)[tokens] * float(cfg["embedding"]["scale"])


def forward(tokens: List[int], w: Dict[str, torch.Tensor], cfg: dict, emulate_bf16: bool = False,
            probe: Optional[dict] = None, layers_out: Optional[list] = None) -> torch.Tensor:
    eps = float(cfg["norm"]["eps"])
    e16 = emulate_bf16
    x = embedding(tokens, w, cfg)
    for i, t, first in run_order(cfg):
        layer = cfg["layers"][i]
        p = f"l{i}"
        if first:
            x = x + w["loop.step"].to(F)[t]
        h = bf(centred_norm(x, w[p + ".norm1"], eps), e16)
        y = MIXERS[layer["type"]](h, w, p + ".mix", layer["mixer"], eps, e16, probe)
        if layer.get("mlp") is not None:
            y = y + experts_ff(h, w, p + ".mlp", layer["mlp"], e16, probe)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return bf(centred_norm(x, w["final.norm"], eps), e16) @ w["head"].to(F).T


def greedy_generate(cfg: dict, w: Dict[str, torch.Tensor], prompt: List[int], n: int) -> List[int]:
    """n tokens, each the largest logit after everything so far (ties to the lower id)."""
    seq, out = list(prompt), []
    for _ in range(n):
        logits = forward(seq, w, cfg)[-1]
        t = int(torch.nonzero(logits == logits.max())[0])
        out.append(t)
        seq.append(t)
    return out
