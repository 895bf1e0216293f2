"""Attention through one cached latent per token (``LatentAttentionSpec``).

Per token the cache holds the normed latent c (``kv_rank``) and one rotated key part (``rot_dim``) shared by all
heads: one key/value head of ``kv_rank + rot_dim`` elements and no value pages.  A head's plain key is W_uk,h c, so
its score q_plain . (W_uk,h c) equals (W_uk,h^T q_plain) . c: the queries are carried into the latent's space
(one batched product per step) and attention runs against the cached rows as they are, all heads sharing them;
the values are the rows' first ``kv_rank`` elements, and W_uv,h is applied to the attention's output (a second
batched product).  Nothing per head is made for a cached token.

That is the way of decode steps and short portions.  A long prompt portion has many queries for every cached token, so
there it pays to make keys and values per head once: the context's rows are gathered from their pages, ONE product makes
every head's [plain key | rotated key part | value] of them (the rotated part through rows of the identity, which copies
it exactly), and the tcgen05 prompt kernel attends with keys of ``head_dim + rot_dim`` and values of ``value_dim``
elements instead of rows of ``kv_rank + rot_dim`` and ``kv_rank`` (PRELUDE_LATENT_EXPAND=0 turns it off).  With a window only
the rows that the portion sees are gathered.

Steps: down projections of queries and of latent + key part; norm of the query latent; up projection of the
queries (or, for queries that come from the input directly, one merged projection [queries | latent + key part | gate]);
one kernel norms the latent, rotates the key part and the queries' rotated part and writes the page;
queries into latent space; attention with the sink and the gate per head; values out of latent space (a gate per element
multiplies them there); output projection.
A layer that reads another layer's cache (``share_cache``) has no down projection of its own and writes nothing.
"""
from __future__ import annotations

import os
from typing import Dict

import torch

from ..config.spec import LatentAttentionSpec
from ..ops import kernels as K
from ..ops.linear import PendingProduct, batched_linear, linear
from ..ops.paged_general import ROWS_MIN_PORTION, attention_general, attention_rows, gather_rows, rows_plan, rows_supported
from ..weights.loader import TensorReq
from .registry import KvPagesNeed, RunContext, make_part, register_part

EXPAND = os.environ.get("PRELUDE_LATENT_EXPAND", "1") != "0"


@register_part("mixer", "latent_attention")
class LatentAttention:
    defer_output = False        # True: the output projection is handed on as a product still to run (``PendingProduct``)

    def __init__(self, spec: LatentAttentionSpec, prefix: str):
        self.spec, self.prefix = spec, prefix
        self.position = make_part("position", spec.position, prefix)
        if getattr(self.position, "rates_host", None) is None:
            raise ValueError("this mixer takes a position encoding given by rates (kind 'rotary_rates')")
        if self.position.rotary_dim > spec.rot_dim:
            raise ValueError(f"a rotation of {self.position.rotary_dim} elements does not fit the rotated part of {spec.rot_dim}")
        if spec.head_gate and spec.element_gate:
            raise ValueError("the output's gate is one per head or one per element, not both")
        self.q_dim = spec.head_dim + spec.rot_dim
        self.g_cols = spec.num_heads * spec.value_dim if spec.element_gate else spec.num_heads if spec.head_gate else 0
        self.row = spec.kv_rank + spec.rot_dim                  # what a token keeps in the cache
        self.w_dq = self.w_uq = self.w_dkv = self.w_uk_t = self.w_uv = self.w_o = None
        self.dq_norm = self.dkv_norm = self.sink = None
        self.w_in = self.w_gate = None         # direct queries: the merged projection; low-rank queries: the gate's own
        self.w_rows = None                     # [heads * (q_dim + value_dim), row]: a cached row to every head's key and value
        self.owns_latent = True

    def share_cache(self) -> None:
        """The layer reads rows that another layer caches: it has no down projection of its own."""
        self.owns_latent = False

    def parts(self):
        return (self.position,)

    def tensors(self) -> Dict[str, TensorReq]:
        s, p = self.spec, self.prefix
        if s.q_rank is None:
            req = {f"{p}.{s.q_name}": TensorReq((s.num_heads * self.q_dim, s.hidden_size))}
        else:
            req = {
                f"{p}.{s.dq_name}": TensorReq((s.q_rank, s.hidden_size)),
                f"{p}.{s.dq_name}{s.norm_suffix}": TensorReq((s.q_rank,), "norm"),
                f"{p}.{s.uq_name}": TensorReq((s.num_heads * self.q_dim, s.q_rank)),
            }
        if self.owns_latent:
            req[f"{p}.{s.dkv_name}"] = TensorReq((self.row, s.hidden_size))
            req[f"{p}.{s.dkv_name}{s.norm_suffix}"] = TensorReq((s.kv_rank,), "norm")
        req.update({
            f"{p}.{s.uk_name}": TensorReq((s.num_heads * s.head_dim, s.kv_rank)),
            f"{p}.{s.uv_name}": TensorReq((s.num_heads * s.value_dim, s.kv_rank)),
            f"{p}.{s.o_name}": TensorReq((s.hidden_size, s.num_heads * s.value_dim)),
        })
        if self.g_cols:
            req[f"{p}.{s.gate_name}"] = TensorReq((self.g_cols, s.hidden_size))
        if s.sink:
            req[f"{p}.{s.sink_name}"] = TensorReq((s.num_heads,), "bias")
        return req

    def load(self, get, ctx: RunContext) -> None:
        s, p = self.spec, self.prefix

        def mat(name):
            return get(f"{p}.{name}").to(device=ctx.device, dtype=ctx.dtype).contiguous()

        def vec(name):
            return get(f"{p}.{name}").to(device=ctx.device, dtype=torch.float32).contiguous()

        self.w_o = mat(s.o_name)
        if s.q_rank is None:
            mats = [mat(s.q_name)] + ([mat(s.dkv_name)] if self.owns_latent else []) + ([mat(s.gate_name)] if self.g_cols else [])
            pad = (-sum(m.shape[0] for m in mats)) % 8         # rows of the merged projection stay 16-byte aligned
            if pad:
                mats.append(torch.zeros((pad, s.hidden_size), dtype=ctx.dtype, device=ctx.device))
            self.w_in = torch.cat(mats, dim=0).contiguous()
        else:
            self.w_dq, self.w_uq = mat(s.dq_name), mat(s.uq_name)
            self.dq_norm = vec(s.dq_name + s.norm_suffix)
            if self.owns_latent:
                self.w_dkv = mat(s.dkv_name)
            if self.g_cols:
                self.w_gate = mat(s.gate_name)
        if self.owns_latent:
            self.dkv_norm = vec(s.dkv_name + s.norm_suffix)
        # head h's rows of W_uk, transposed: [heads, kv_rank, head_dim], the weight of "queries into latent space"
        self.w_uk_t = mat(s.uk_name).view(s.num_heads, s.head_dim, s.kv_rank).transpose(1, 2).contiguous()
        self.w_uv = mat(s.uv_name).view(s.num_heads, s.value_dim, s.kv_rank)
        if s.sink:
            self.sink = vec(s.sink_name)
        self.position.load(get, ctx)
        if EXPAND and ctx.dtype == torch.bfloat16 and rows_supported(self.q_dim, s.value_dim, self.row):
            w = torch.zeros((s.num_heads, self.q_dim + s.value_dim, self.row), dtype=ctx.dtype, device=ctx.device)
            w[:, :s.head_dim, :s.kv_rank] = self.w_uk_t.transpose(1, 2)
            w[:, s.head_dim:self.q_dim, s.kv_rank:] = torch.eye(s.rot_dim, dtype=ctx.dtype, device=ctx.device)
            w[:, self.q_dim:, :s.kv_rank] = self.w_uv
            self.w_rows = w.view(s.num_heads * (self.q_dim + s.value_dim), self.row)

    def activation_bytes_per_token(self, elem: int) -> int:
        s = self.spec
        rows = 0 if self.w_rows is None else s.num_heads * (2 * self.q_dim + s.value_dim) + self.row
        return ((s.q_rank or 0) * 2 + rows + s.num_heads * (2 * self.q_dim + 2 * self.row + s.value_dim) + self.row + self.g_cols) * elem + s.hidden_size * elem

    def cache_need(self) -> KvPagesNeed:
        return KvPagesNeed(1, self.row, self.spec.window, v_heads=0, v_head_dim=0)

    def _prepare(self, q, ckv, batch, cache, q_out, q_split, q_out2) -> None:
        """Rotated queries (their parts after ``q_split`` to q_out2 behind the latent's place); with ``ckv`` the normed latent and
        the rotated key part into the page."""
        s, pos = self.spec, self.position
        K.qkv_prepare(q, ckv, None, n_heads=s.num_heads, q_dim=self.q_dim, k_weight=self.dkv_norm if ckv is not None else None,
                      k_norm_cols=s.kv_rank, eps=s.norm_eps, rates=pos.rates, rot_dims=pos.rotary_dim, adjacent=pos.adjacent,
                      amplitude=pos.amplitude, q_rot_off=s.head_dim, k_rot_off=s.kv_rank, positions=batch.positions,
                      table_row=batch.table_row_of_token, block_table=batch.block_tables[cache.group], q_out=q_out, q_split=q_split,
                      q_out2=q_out2, q2_off=s.kv_rank, k_pages=cache.k_pages if ckv is not None else None, status=batch.status)

    def _rows_plan(self, batch):
        """The plan of the step's long portions whose keys and values are made per head, or None.  A step that is being recorded
        has the shape of its token count alone and keeps to the latent's space."""
        recorder = batch.extras.get("recorder")
        if self.w_rows is None or batch.decode_only or batch.max_q_len < ROWS_MIN_PORTION or recorder is not None:
            return None
        return rows_plan(batch, self.spec.window)

    def _in_latent_space(self, q, ckv, gate, batch, cache, below, o) -> None:
        """Attention against the cached rows as they are; portions of ``below`` tokens and more are left out."""
        s = self.spec
        T, H = batch.n_tokens, s.num_heads
        q_plain = batch.workspace("latent_q_plain", (T, H, s.head_dim), q.dtype)
        q_lat = batch.workspace("latent_q", (T, H, self.row), q.dtype)
        self._prepare(q, ckv, batch, cache, q_plain, s.head_dim, q_lat)
        # queries into latent space, head by head: q_lat[:, h, :kv_rank] = q_plain[:, h] W_uk,h
        batched_linear(q_plain.transpose(0, 1), self.w_uk_t, q_lat.transpose(0, 1)[:, :, :s.kv_rank])
        o_lat = attention_general(q_lat, cache.k_pages, None, s.kv_rank, batch, cache.group, s.softmax_scale, s.window, self.sink,
                                  out=batch.workspace("latent_o", (T, H, s.kv_rank), q.dtype), gate=gate if s.head_gate else None, below=below)
        # values out of latent space: o[:, h] = o_lat[:, h] W_uv,h^T
        batched_linear(o_lat.transpose(0, 1), self.w_uv, o.transpose(0, 1))
        if s.element_gate:
            K.sigmoid_gate_(o.view(T, H * s.value_dim), gate)

    def forward(self, x: torch.Tensor, batch, cache, write_cache: bool = True) -> torch.Tensor:
        s = self.spec
        T, H = batch.n_tokens, s.num_heads
        gate = None
        if s.q_rank is None:
            proj = linear(x, self.w_in)
            q = proj[:, :H * self.q_dim]                                  # [T, H * (head_dim + rot_dim)]
            c0 = H * self.q_dim + (self.row if self.owns_latent else 0)
            ckv = proj[:, H * self.q_dim:c0] if write_cache else None     # [T, kv_rank + rot_dim]
            if self.g_cols:
                gate = proj[:, c0:c0 + self.g_cols]
        else:
            cq = K.rmsnorm(linear(x, self.w_dq), self.dq_norm, s.norm_eps)
            q = linear(cq, self.w_uq)
            ckv = linear(x, self.w_dkv) if write_cache else None
            if self.g_cols:
                gate = linear(x, self.w_gate)
        o = batch.workspace("latent_values", (T, H, s.value_dim), x.dtype)
        plan = self._rows_plan(batch)
        if plan is None or not plan.all_long:
            self._in_latent_space(q, ckv, gate, batch, cache, None if plan is None else ROWS_MIN_PORTION, o)
            ckv = None                                                    # cached
        if plan is not None:
            q_full = batch.workspace("latent_q_full", (T, H, self.q_dim), x.dtype)
            self._prepare(q, ckv, batch, cache, q_full, self.q_dim, None)
            kv = linear(gather_rows(cache.k_pages, batch, cache.group, plan), self.w_rows)
            attention_rows(q_full, kv, s.value_dim, batch, plan, s.softmax_scale, self.sink, gate, o)
        o = o.view(T, H * s.value_dim)
        return PendingProduct(o, self.w_o) if self.defer_output else linear(o, self.w_o)
