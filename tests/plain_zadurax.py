"""Zadurax, plainly: whole sequences, no cache, no batches, float64, one function per
mechanism, written from the design's equations.  It reads config.json's keys and the
tensor names by itself and shares no code with the package.

``emulate_bf16`` rounds where the bfloat16 engine rounds (the normed rows that feed the
projections, q and the cached keys and values, the latent and the rotated key part, the
queries carried into the latent's space and the weighted sums there, the gated heads before
the output projection, the feed-forward's activations); norms, angles, scores, softmax, sinks,
gates, the matrix memory with everything that enters it, and the residual sum stay exact.
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


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * w.to(F)


def project(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return h @ w.to(F).T


# ---- rotation -----------------------------------------------------------------------------
def turning_rates(rot: dict):
    """(frequency of every pair, the number that multiplies every cosine and sine)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def at(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(at(float(sc["fast"]))), 0)
    hi = min(math.ceil(at(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, d], rows at positions 0 ..: value 2i turns with value 2i + 1, for the first
    ``dims`` values of a head."""
    freq, size = turning_rates(rot)
    t = torch.arange(x.shape[0], dtype=F)
    y = x.clone()
    for i, fi in enumerate(freq):
        c, s = (torch.cos(t * fi) * size)[:, None], (torch.sin(t * fi) * size)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


# ---- attention whose values are its keys --------------------------------------------------
def window_mask(T: int, size: int) -> torch.Tensor:
    i = torch.arange(T)
    back = i[:, None] - i[None, :]
    return (back >= 0) & (back < size)


def attention(h, w, p, m, eps, e16, probe=None):
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = project(h, w[p + ".q"]).view(T, H, d)
    raw = project(h, w[p + ".k"]).view(T, G, d)
    q = bf(rotate(norm(q, w[p + ".q.norm"], eps), m["rot"]), e16)
    k = bf(rotate(norm(raw, w[p + ".k.norm"], eps), m["rot"]), e16)
    v = bf(raw, e16)  # as projected: before norm and rotation
    visible = window_mask(T, int(m["mask"]["size"]))
    out = torch.zeros(T, H, d, dtype=F)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * float(m["scale"])
        weights = torch.softmax(s.masked_fill(~visible, -math.inf), dim=-1)
        if probe is not None:
            probe.setdefault("weights", []).append(weights)
        out[:, a] = weights @ v[:, g]
    gated = out.reshape(T, H * d) * torch.sigmoid(project(h, w[p + ".g"]))
    return project(bf(gated, e16), w[p + ".o"])


# ---- attention over a latent --------------------------------------------------------------
def softmax_with_sink(s: torch.Tensor, sink: float) -> torch.Tensor:
    """One more term exp(sink) in the denominator, with no key and no value."""
    top = torch.clamp(s.max(dim=-1, keepdim=True).values, min=sink)
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def latent_attention(h, w, p, m, eps, e16, probe=None):
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = project(h, w[p + ".q"]).view(T, H, d + r)
    q_plain = bf(q[..., :d], e16)
    q_rot = bf(rotate(q[..., d:], m["rot"]), e16)
    down = project(h, w[p + ".dkv"])
    c = bf(norm(down[:, :rank], w[p + ".dkv.norm"], eps), e16)
    k_rot = bf(rotate(down[:, rank:].view(T, 1, r), m["rot"]), e16)[:, 0]
    uk, uv = w[p + ".uk"].to(F).view(H, d, rank), w[p + ".uv"].to(F).view(H, dv, rank)
    visible = window_mask(T, T)
    out = torch.zeros(T, H, dv, dtype=F)
    for a in range(H):
        if e16:  # (the engine scores and sums in the latent's space, with a rounding at each border)
            plain = bf(q_plain[:, a] @ uk[a], e16) @ c.T
        else:
            plain = q_plain[:, a] @ (c @ uk[a].T).T
        s = (plain + q_rot[:, a] @ k_rot.T) * float(m["scale"])
        weights = softmax_with_sink(s.masked_fill(~visible, -math.inf), float(w[p + ".sink"][a]))
        if probe is not None:
            probe.setdefault("weights", []).append(weights)
        out[:, a] = bf(weights @ c, e16) @ uv[a].T if e16 else weights @ (c @ uv[a].T)
    gated = out.reshape(T, H * dv) * torch.sigmoid(project(h, w[p + ".g"]))
    return project(bf(gated, e16), w[p + ".o"])


# ---- matrix memory ------------------------------------------------------------------------
def matrix_memory(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, dv], log gates i, f [T, H] -> [T, H, dv]: token by token."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F)
    n = torch.zeros(H, d, dtype=F)
    m = torch.zeros(H, dtype=F)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        m = m_new
        bottom = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(1) / bottom[:, None]
    return out


def mlstm(h, w, p, m, eps, e16, probe=None):
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    q = project(h, w[p + ".q"]).view(T, H, d) * d ** -0.5
    k = project(h, w[p + ".k"]).view(T, H, d)
    v = project(h, w[p + ".v"]).view(T, H, dv)
    i = cap * torch.tanh((project(h, w[p + ".i"]) + w[p + ".i.b"].to(F)) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((project(h, w[p + ".f"]) + w[p + ".f.b"].to(F)) / cap))
    o = matrix_memory(q, k, v, i, f)
    y = rms(o, eps).reshape(T, H * dv) * w[p + ".norm"].to(F) * torch.sigmoid(project(h, w[p + ".g"]))
    return project(bf(y, e16), w[p + ".o"])


# ---- feed-forward -------------------------------------------------------------------------
def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def dense(h, w, p, e16):
    return project(bf(gelu_tanh(project(h, w[p + ".gate"])) * project(h, w[p + ".up"]), e16), w[p + ".down"])


# ---- the model ----------------------------------------------------------------------------
MIXERS = {"attention": attention, "latent_attention": latent_attention, "mlstm": mlstm}


def owner(cfg: dict, i: int) -> int:
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(tokens: List[int], w: Dict[str, torch.Tensor], cfg: dict, emulate_bf16: bool = False,
            probe: Optional[dict] = None, layers_out: Optional[list] = None) -> torch.Tensor:
    eps = float(cfg["norm"]["eps"])
    e16 = emulate_bf16
    x = norm(w["embed"].to(F)[tokens], w["embed.norm"], eps)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}"
        y = MIXERS[layer["type"]](bf(norm(x, w[p + ".norm1"], eps), e16), w, p + ".mix", layer["mixer"], eps, e16, probe)
        x = x + norm(y, w[p + ".norm1b"], eps)
        if layer.get("mlp") is not None:
            y = dense(bf(norm(x, w[p + ".norm2"], eps), e16), w, p + ".mlp", e16)
            x = x + norm(y, w[p + ".norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return project(bf(norm(x, w["final.norm"], eps), e16), w["head"])


def greedy_generate(cfg: dict, w: Dict[str, torch.Tensor], prompt: List[int], n: int) -> List[int]:
    """n tokens, each the largest logit after everything so far (ties to the lower id)."""
    seq, out = list(prompt), []
    for _ in range(n):
        logits = forward(seq, w, cfg)[-1]
        t = int(torch.nonzero(logits == logits.max())[0])
        out.append(t)
        seq.append(t)
    return out
