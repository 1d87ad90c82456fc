"""Causal attention whose keys and values come from one small latent per position.

The layer's input h goes down to two latents: ``cq = rms(W_dq h) * w_q`` for the
queries and ``c = rms((W_dkv h)[:kv_rank]) * w_kv`` for keys and values; the last
``rot_dim`` rows of ``W_dkv h`` are a key part that every head shares and that is
rotated by position.  Per head, ``q = W_uq cq`` is ``dim`` plain and ``rot_dim``
rotated values, the plain key is ``W_uk c`` and the value ``W_uv c``; a score is
``(q_plain . k_plain + q_rot . k_rot) * scale`` and the weights an ordinary softmax
over the positions up to the query's (``window`` > 0: over the last ``window`` of them).

With ``q_rank`` 0 there is no latent for the queries: ``q = W_q h``.  Then the queries, the
latent and, with ``gate`` "head", the logits of a gate per head (head i's output is multiplied
by ``sigmoid(W_g h)_i``) come from one product of stacked matrices, and one kernel
(``latent_prep_direct``) packs, turns, norms, stores and takes the sigmoid; the gate multiplies
the weighted sum of latents, which is the head's output before its linear ``W_uv``.  With
``gate`` "value" W_g has a row per output value and the joined heads are multiplied value by value
by ``sigmoid(W_g h)``, in the epilogue of the product with ``W_uv``.  With ``sink`` the softmax's
denominator also holds ``exp(sink_h)``, a learned number per head (names["sink"]) with no key and no
value.  A position encoding with a ``magnitude`` multiplies every cosine and sine by it (q_rank 0).

Only ``[c | k_rot]`` is cached, one row per position for all heads, in a cache
group without storage for values.  Because ``q_plain . (W_uk c) = (W_uk^T q_plain) . c``,
the queries are carried into the latent's space (one small product per head,
``W_uk`` transposed per head at load) and attention runs there: a score is one dot
product with the cached row, the output is a weighted sum of the rows' ``c`` part,
and the heads' values are made from that sum (``W_uv`` per head) before ``W_o`` adds
into the residual stream.  Prompts, later chunks and single tokens take the same way.

params: hidden_size, heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, eps, window, gate, sink,
position (a ``rope_frequencies`` PartSpec, either pairing), names {dq, dq_norm, uq (or q), dkv,
dkv_norm, uk, uv, o, gate, sink}.
"""
from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..cache import PAGE_SIZE, KVRequest, KVView
from ..csrc import ops
from ..weights.loader import WeightSpec
from .base import MIXERS, POSITIONS, Part
from .linear import ADD_F32, STORE, STORE_F32, linear


class LatentAttention(Part):
    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["heads"])
        self.dim = int(params["dim"])
        self.rot = int(params["rot_dim"])
        self.vdim = int(params["vdim"])
        self.q_rank = int(params.get("q_rank") or 0)  # 0: queries straight from h
        self.kv_rank = int(params["kv_rank"])
        self.scale = float(params["scale"])
        self.eps = float(params["eps"])
        self.window = int(params.get("window") or 0)
        gate = params.get("gate", False)
        if gate not in (False, None, "head", "value"):
            raise ValueError(f"latent attention: gate {gate!r} is not known (head, value)")
        self.has_gate = bool(gate)
        self.gate_by_value = gate == "value"
        self.gate_cols = (self.heads * self.vdim if self.gate_by_value else self.heads) if self.has_gate else 0
        self.has_sink = bool(params.get("sink", False))
        if self.has_gate and self.q_rank:
            raise ValueError("latent attention: a gate goes with queries straight from the input (q_rank 0)")
        self.names = params["names"]
        pos = params["position"]
        self.position = POSITIONS.build(pos.kind, pos.params, prefix, dtype, device)
        if not hasattr(self.position, "frequencies"):
            raise ValueError("latent attention rotates by a table of frequencies (rope_frequencies)")
        if self.position.dims > self.rot:
            raise ValueError(f"rotation over {self.position.dims} dimensions, the rotated part has {self.rot}")
        self.pairing = getattr(self.position, "pairing", "half")
        self.magnitude = float(getattr(self.position, "magnitude", 1.0))
        if self.magnitude != 1.0 and self.q_rank:
            raise ValueError("latent attention: a rotation with a magnitude goes with queries straight from the input "
                             "(q_rank 0)")
        for what in ("heads", "dim", "vdim", "kv_rank"):
            if getattr(self, what) <= 0:
                raise ValueError(f"latent attention: {what} must be positive")
        if self.kv_rank > 512:
            raise ValueError("latent attention kernels take latents of up to 512 values")
        self.row = self.kv_rank + self.rot  # a cached row, and a query in the latent's space
        self.q_cols = self.heads * (self.dim + self.rot)
        self.w_down = self.w_uq = self.w_ukt = self.w_uv = self.w_o = None
        self.norm_q = self.norm_kv = self.sink = None

    # -- weights ----------------------------------------------------------
    def _name(self, key: str) -> str:
        return self.tensor_name(self.names[key])

    def weight_specs(self) -> Dict[str, WeightSpec]:
        W, H = self.hidden, self.heads
        if self.q_rank:
            specs = {
                self._name("dq"): WeightSpec((self.q_rank, W), "matrix", fan_in=W),
                self._name("dq_norm"): WeightSpec((self.q_rank,), "vector", init="ones"),
                self._name("uq"): WeightSpec((self.q_cols, self.q_rank), "matrix", fan_in=self.q_rank),
            }
        else:
            specs = {self._name("q"): WeightSpec((self.q_cols, W), "matrix", fan_in=W)}
        if self.has_gate:
            specs[self._name("gate")] = WeightSpec((self.gate_cols, W), "matrix", fan_in=W)
        if self.has_sink:
            specs[self._name("sink")] = WeightSpec((H,), "vector")
        specs.update({
            self._name("dkv"): WeightSpec((self.kv_rank + self.rot, W), "matrix", fan_in=W),
            self._name("dkv_norm"): WeightSpec((self.kv_rank,), "vector", init="ones"),
            self._name("uk"): WeightSpec((H * self.dim, self.kv_rank), "matrix", fan_in=self.kv_rank),
            self._name("uv"): WeightSpec((H * self.vdim, self.kv_rank), "matrix", fan_in=self.kv_rank),
            self._name("o"): WeightSpec((W, H * self.vdim), "matrix", fan_in=H * self.vdim),
        })
        return specs

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        H = self.heads
        # what reads h is one product: [q latent | c raw | k_rot raw], or [q | c raw | k_rot raw | gate]
        keys = ["dq" if self.q_rank else "q", "dkv"] + (["gate"] if self.has_gate else [])
        rows = [tensors[self._name(k)] for k in keys]
        if not self.q_rank:  # zero rows up to a multiple of eight, as the decode projection kernels take them
            rows.append(rows[0].new_zeros((-sum(r.shape[0] for r in rows) % 8, self.hidden)))
        self.w_down = torch.cat(rows, 0).contiguous()
        if self.q_rank:
            self.norm_q = tensors[self._name("dq_norm")]
            self.w_uq = tensors[self._name("uq")]
        self.norm_kv = tensors[self._name("dkv_norm")]
        if self.has_sink:
            self.sink = tensors[self._name("sink")]
        # per head [kv_rank, dim]: the product that carries q_plain into the latent's space
        self.w_ukt = tensors[self._name("uk")].view(H, self.dim, self.kv_rank).transpose(1, 2).contiguous()
        self.w_uv = tensors[self._name("uv")].view(H, self.vdim, self.kv_rank).contiguous()
        self.w_o = tensors[self._name("o")]

    def parameter_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in
                   (self.w_down, self.w_uq, self.w_ukt, self.w_uv, self.w_o, self.norm_q, self.norm_kv)
                   if t is not None)

    # -- cache ------------------------------------------------------------
    def cache_request(self) -> Optional[KVRequest]:
        return KVRequest(1, self.row, self.window, values=False)

    def check_shared_cache(self, view: KVView) -> None:
        raise ValueError("latent attention writes a cache of its own")

    def step_flops(self, counts, starts) -> float:
        H, W = self.heads, self.hidden
        tokens = sum(counts)
        into_q = W * self.q_rank + self.q_rank * self.q_cols if self.q_rank else W * (self.q_cols + self.gate_cols)
        per_token = into_q + W * self.row + H * self.dim * self.kv_rank + H * self.vdim * self.kv_rank + H * self.vdim * W
        keys = sum(sum(min(st + q + 1, self.window) for q in range(c)) if self.window
                   else c * st + c * (c + 1) // 2 for c, st in zip(counts, starts))
        return 2.0 * tokens * per_token + 2.0 * H * (self.row + self.kv_rank) * keys

    # -- work lists ---------------------------------------------------------
    def _tiles_name(self) -> str:
        return f"latent_mma/heads{self.heads}/rows{ops.latent_tile_rows(self.kv_rank)}"

    def _tensor_cores(self) -> bool:
        return self.dtype == torch.bfloat16 and ops.attention_latent_mma_takes(self.row, self.kv_rank, PAGE_SIZE)

    def step_tables(self, counts, starts, have=()):
        """The tiles of the tensor-core kernel for a prompt step: 64 or 128 stacked (token,
        head) rows each; the same for every layer with this number of heads and tile."""
        if not self._tensor_cores() or self._tiles_name() in have:
            return {}
        return {self._tiles_name(): ops.latent_tiles(counts, starts, self.heads,
                                                     ops.latent_tile_rows(self.kv_rank))}

    def _decode_splits(self, ctx, n: int) -> int:
        """Slices of the key range in a step of single tokens: enough CTAs for two per SM,
        at least two pages a slice."""
        ctas = n * -(-self.heads // ops.latent_tile_rows(self.kv_rank)) * -(-self.kv_rank // 512)
        keys = ctx.max_context if not self.window else min(ctx.max_context, self.window + PAGE_SIZE - 1)
        pages = max(1, -(-keys // PAGE_SIZE))
        want = -(-2 * ops.sm_count(self.device) // max(1, ctas * max(1, ctx.share)))
        return int(max(1, min(want, pages // 2, 64)))

    # -- run --------------------------------------------------------------
    def forward(self, x: torch.Tensor, ctx, residual: torch.Tensor, cache: KVView) -> None:
        n = residual.shape[0]
        H, ws = self.heads, ctx.workspace
        table = ctx.page_tables[cache.group]
        freq = self.position.frequencies()
        down = ws.get("latent_down", (n, self.w_down.shape[0]), torch.float32)
        linear(x, self.w_down, None, down, STORE_F32, decode=ctx.decode)
        q_lat = ws.get("latent_q_abs", (n, H * self.row), self.dtype)
        # (a gate per head multiplies inside the attention kernel, one per value after W_uv)
        gate = ws.get("latent_gate", (n, H), torch.float32) if self.has_gate and not self.gate_by_value else None
        if self.q_rank:
            self._queries_from_latent(ctx, down, q_lat, freq, table, cache)
        else:
            q = ws.get("latent_q", (n, H * self.dim), self.dtype)
            ops.latent_prep_direct(down, self.norm_kv, freq, ctx.token_pos, ctx.token_seq, table, q, q_lat, cache.k,
                                   gate, H, self.dim, self.kv_rank, self.rot, self.position.dims, self.eps,
                                   pairing=self.pairing, magnitude=self.magnitude)
            ops.batched_linear(q, self.dim, self.w_ukt, q_lat, self.row)
        o_lat = ws.get("latent_o", (n, H * self.kv_rank), self.dtype)
        tiles = ctx.tables.get(self._tiles_name())
        if self._tensor_cores() and (ctx.decode or tiles is not None):
            splits = self._decode_splits(ctx, n) if ctx.decode else 1
            partial = ws.get("attn_partial", (n * H * splits * (self.kv_rank + 2),), torch.float32) \
                if splits > 1 else None
            if ctx.decode:
                ops.attention_latent_mma(q_lat, cache.k, None, None, None, None, ctx.token_pos, ctx.token_seq,
                                         table, o_lat, H, self.kv_rank, self.scale, splits, partial,
                                         window=self.window, gate=gate, sink=self.sink)
            else:
                ops.attention_latent_mma(q_lat, cache.k, tiles, ctx.seq_first_row, ctx.seq_start,
                                         ctx.seq_count, ctx.token_pos, ctx.token_seq, table, o_lat, H,
                                         self.kv_rank, self.scale, window=self.window, gate=gate, sink=self.sink)
        else:
            splits = ctx.attention_splits(n * H)
            if self.window:  # a slice has at least 64 keys of the window
                splits = max(1, min(splits, -(-self.window // 64)))
            partial = ws.get("attn_partial", (n * H * splits * (self.kv_rank + 2),), torch.float32) \
                if splits > 1 else None
            ops.attention_latent(q_lat, cache.k, ctx.token_pos, ctx.token_seq, table, o_lat, H, self.kv_rank,
                                 self.scale, splits, partial, window=self.window, gate=gate, sink=self.sink)
        attn = ws.get("attn", (n, H * self.vdim), self.dtype)
        ops.batched_linear(o_lat, self.kv_rank, self.w_uv, attn, self.vdim, gate=down if self.gate_by_value else None,
                           gate_off=self.q_cols + self.row if self.gate_by_value else 0)
        linear(attn, self.w_o, None, residual, ADD_F32, ws, decode=ctx.decode)

    def _queries_from_latent(self, ctx, down, q_lat, freq, table, cache) -> None:
        """Queries by way of their own latent: norm, up-projection, into the latent's space."""
        n, H, ws = down.shape[0], self.heads, ctx.workspace
        cq = ws.get("latent_cq", (n, self.q_rank), self.dtype)
        ops.latent_prep(down, self.norm_q, self.norm_kv, freq, ctx.token_pos, ctx.token_seq, table, cq,
                        cache.k, self.q_rank, self.kv_rank, self.rot, self.position.dims, self.eps,
                        pairing=self.pairing)
        q = ws.get("latent_q", (n, self.q_cols), self.dtype)
        linear(cq, self.w_uq, None, q, STORE, decode=ctx.decode)
        ops.batched_linear(q, self.dim + self.rot, self.w_ukt, q_lat, self.row)
        if self.rot:
            ops.rope_part(q, self.dim + self.rot, self.dim, q_lat, self.row, self.kv_rank, ctx.token_pos,
                          freq, H, self.rot, self.position.dims, pairing=self.pairing)


MIXERS.register("latent_attention", LatentAttention)
