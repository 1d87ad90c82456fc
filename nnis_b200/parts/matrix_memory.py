"""Matrix memory with exponential gates: the mLSTM of xLSTM.

Per head, with q = W_q h * dim^-1/2, k = W_k h, v = W_v h and the log gates
i = cap tanh((W_i h + b_i) / cap), f = logsigmoid(cap tanh((W_f h + b_f) / cap)):

    m_t = max(f + m_t-1, i)                                    m_0 = 0
    S_t = exp(f + m_t-1 - m_t) S_t-1 + exp(i - m_t) k v^T      n_t likewise with k in k v^T's place
    o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + floor)

Each head's o is divided by its root mean square, the joined heads are multiplied by a weight per
value and by sigmoid(W_g h), and W_o adds the result into the residual stream.

S [heads, dim, vdim], n [heads, dim] and m [heads] are float32 in the cache's state area and zero when
a slot is taken, so a later portion of a prompt or a single token goes on from what the tokens
before left.  n and m are kept twice, for even and for odd positions: position p reads one and leaves
the other, so CTAs that share a head need no order among themselves.

One product makes q, k, v and all gates' logits in float32; everything after it is float32 in every
dtype.  Single tokens update the memory in one kernel.  Prompts go in chunks of 64 tokens that are
worked side by side: what a chunk adds by itself, then the states between the chunks in order, then
the outputs of every chunk from the state before it and its own tokens.

params: hidden_size, heads, dim, vdim, gate_cap, floor, eps, names {q, k, v, g, i, i_bias, f, f_bias,
norm, o}.
"""
from __future__ import annotations

from typing import Dict, Mapping

import torch

from ..cache import StateRequest, StateView
from ..csrc import ops
from ..weights.loader import WeightSpec
from .base import MIXERS, Part
from .linear import ADD_F32, STORE_F32, linear


class MatrixMemory(Part):
    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["heads"])
        self.dim = int(params["dim"])
        self.vdim = int(params["vdim"])
        self.cap = float(params["gate_cap"])
        self.floor = float(params.get("floor", 1e-6))
        self.eps = float(params["eps"])
        self.names = params["names"]
        if min(self.heads, self.dim, self.vdim) <= 0 or not self.cap > 0:
            raise ValueError("matrix memory: heads, dim, vdim and gate_cap must be positive")
        if self.dim > 2048:
            raise ValueError("matrix memory kernels take key sizes up to 2048")
        self.gate_off = self.heads * (2 * self.dim + self.vdim)  # g's first column of the input product
        self.w_in = self.w_o = self.i_bias = self.f_bias = self.norm = None

    def _name(self, key: str) -> str:
        return self.tensor_name(self.names[key])

    def _projections(self):
        H = self.heads
        return (("q", H * self.dim), ("k", H * self.dim), ("v", H * self.vdim), ("g", H * self.vdim), ("i", H), ("f", H))

    def weight_specs(self) -> Dict[str, WeightSpec]:
        W, H = self.hidden, self.heads
        specs = {self._name(p): WeightSpec((rows, W), "matrix", fan_in=W) for p, rows in self._projections()}
        specs[self._name("i_bias")] = WeightSpec((H,), "vector")
        specs[self._name("f_bias")] = WeightSpec((H,), "vector")
        specs[self._name("norm")] = WeightSpec((H * self.vdim,), "vector", init="ones")
        specs[self._name("o")] = WeightSpec((W, H * self.vdim), "matrix", fan_in=H * self.vdim)
        return specs

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        rows = [tensors[self._name(p)] for p, _ in self._projections()]
        # (zero rows up to a multiple of eight, as the decode projection kernels take them)
        rows.append(rows[0].new_zeros((-sum(r.shape[0] for r in rows) % 8, self.hidden)))
        self.w_in = torch.cat(rows, 0).contiguous()
        self.w_o = tensors[self._name("o")]
        self.i_bias, self.f_bias = tensors[self._name("i_bias")], tensors[self._name("f_bias")]
        self.norm = tensors[self._name("norm")]

    def parameter_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_o))

    # -- cache ------------------------------------------------------------
    def cache_request(self) -> StateRequest:
        H = self.heads
        return StateRequest((H, self.dim, self.vdim), torch.float32,
                            extra=(((2, H, self.dim), torch.float32), ((2, H), torch.float32)))

    def check_shared_cache(self, view) -> None:
        raise ValueError("a matrix memory keeps a state of its own")

    def step_flops(self, counts, starts) -> float:
        W, H = self.hidden, self.heads
        return 2.0 * sum(counts) * (W * self.w_in.shape[0] + H * self.vdim * W + 2 * H * self.dim * self.vdim)

    # -- work lists ---------------------------------------------------------
    CHUNKS, FIRST_CHUNK = "matrix_memory/chunks", "matrix_memory/first_chunk"

    def step_tables(self, counts, starts, have=()):
        """The chunks of every sequence of a prompt step (the same list for every layer)."""
        if self.CHUNKS in have:
            return {}
        chunks, first = ops.scan_segments(counts, ops.memory_chunk_tokens())
        return {self.CHUNKS: chunks, self.FIRST_CHUNK: first}

    # -- run --------------------------------------------------------------
    def forward(self, x: torch.Tensor, ctx, residual: torch.Tensor, cache: StateView) -> None:
        n = residual.shape[0]
        H, ws = self.heads, ctx.workspace
        rows = ws.get("memory_in", (n, self.w_in.shape[0]), torch.float32)
        linear(x, self.w_in, None, rows, STORE_F32, decode=ctx.decode)
        o_raw = ws.get("memory_o", (n, H * self.vdim), torch.float32)
        sizes = (H, self.dim, self.vdim, self.cap, self.dim ** -0.5, self.floor)
        norm_state, max_state = cache.extra
        if ctx.decode:
            ops.memory_step(rows, self.i_bias, self.f_bias, cache.state, norm_state, max_state, ctx.token_pos,
                            ctx.token_seq, ctx.seq_slots, o_raw, *sizes)
        else:
            chunks = ctx.tables[self.CHUNKS]
            c = chunks.shape[0]
            ops.memory_prompt(rows, self.i_bias, self.f_bias, cache.state, norm_state, max_state, chunks,
                              ctx.tables[self.FIRST_CHUNK], ctx.seq_slots, ctx.seq_first_row, ctx.seq_start,
                              ctx.seq_count, ws.get("memory_gates", (3, n, H), torch.float64),
                              ws.get("memory_chunk_gates", (4, c, H), torch.float64),
                              ws.get("memory_chunk_state", (c, H, self.dim, self.vdim), torch.float32),
                              ws.get("memory_chunk_norm", (c, H, self.dim), torch.float32), o_raw, *sizes)
        gated = ws.get("memory_gated", (n, H * self.vdim), self.dtype)
        ops.memory_finish(o_raw, rows, self.gate_off, self.norm, ctx.token_pos, gated, H, self.vdim, self.eps)
        linear(gated, self.w_o, None, residual, ADD_F32, ws, decode=ctx.decode)


MIXERS.register("matrix_memory", MatrixMemory)
