"""General paged attention over a step's batch: keys and values of different sizes, values that are part of the
cached key rows, a window, a sink.  Picks the kernel for the type and shape; which one ran changes the rounding,
never what is computed.

float32 always runs the plain warp-per-row kernel.  bfloat16 runs the tensor-core kernel where it takes the shape
(key size in multiples of 16, value size in multiples of 32 up to 512), prompt portions and single tokens alike; a
step of few rows has its keys dealt to several blocks per row (PRELUDE_GENERAL_ATTN=plain turns it off).  Prompt
portions that fill the tcgen05 prompt kernel's blocks go to that kernel where it takes the shape (keys and values of
one size, 64 or 128, in pages of their own; PRELUDE_GENERAL_PROMPT_ATTN=mma turns it off): it knows the same masks,
cap, sink and gate and reads the same pages, permuting them on their way into shared memory.
"""
from __future__ import annotations

import os
from typing import Optional

import numpy as np
import torch

from . import kernels as K
from . import library as _l
from .attention import TC_MIN_FILL, _prefill_plan, _sm_count
from .library import check

KERNEL = os.environ.get("PRELUDE_GENERAL_ATTN", "auto")
PROMPT_KERNEL = os.environ.get("PRELUDE_GENERAL_PROMPT_ATTN", "auto")
MAX_SPLITS = 32


def tc_takes(q: torch.Tensor, k_pages: torch.Tensor, v_pages: Optional[torch.Tensor], value_dim: int) -> bool:
    if KERNEL == "plain" or q.dtype != torch.bfloat16:
        return False
    H, kd, G = q.shape[1], q.shape[2], k_pages.shape[1]
    if v_pages is not None and v_pages.shape[1] != G:
        return False
    return bool(_l.library().pb_attention_paged_tc_supported(H, G, kd, value_dim, 1 if v_pages is None else 0))


def attention_general(q: torch.Tensor, k_pages: torch.Tensor, v_pages: Optional[torch.Tensor], value_dim: int, batch, group: int,
                      scale: float, window: Optional[int], sink: Optional[torch.Tensor], out: Optional[torch.Tensor] = None,
                      keep_first: int = 0, chunk: Optional[int] = None, softcap: Optional[float] = None,
                      gate: Optional[torch.Tensor] = None, below: Optional[int] = None) -> torch.Tensor:
    """q [T, H, kd] of the batch's tokens against the pages of cache group ``group``; ``v_pages`` None: the values are
    the first ``value_dim`` elements of the key rows.  ``keep_first``, ``chunk``, ``softcap``, ``gate``: as for
    ``kernels.attention_paged``.  ``below``: portions of that many tokens and more are left to the caller (their rows of the
    result hold anything).  While a step is being captured piece by piece, the tensor-core
    kernel is launched between the pieces: its grid follows how the step's tokens are spread over requests."""
    T, H, kd = q.shape
    if out is None:
        out = torch.empty((T, H, value_dim), dtype=q.dtype, device=q.device)
    if not tc_takes(q, k_pages, v_pages, value_dim):
        # one warp per row whatever the step holds: the launch has the shape of the token count alone
        return K.attention_paged(q, k_pages, v_pages, value_dim, batch.positions, batch.table_row_of_token, batch.block_tables[group],
                                 scale, window, sink, status=batch.status, out=out, keep_first=keep_first, chunk=chunk,
                                 softcap=softcap, gate=gate)
    recorder = batch.extras.get("recorder")
    if recorder is not None and recorder.capturing and not batch.decode_only:
        recorder.run_between_pieces(lambda: attention_general(q, k_pages, v_pages, value_dim, batch, group, scale, window, sink, out,
                                                              keep_first, chunk, softcap, gate, below))
        return out
    lib = _l.library()
    table = batch.block_tables[group]
    num_pages, G, page_size, _ = k_pages.shape
    if batch.decode_only:
        tile_seq = tile_tok0 = None
        n_tiles = T
    else:
        # The tcgen05 prompt kernel works on 256 query rows at a time and pays for all of them: it takes the portions
        # that fill at least TC_MIN_FILL of a block's tokens, this kernel the shorter ones and the single tokens.  Both
        # write disjoint rows of `out`.
        long_min, long_tiles = below, 0
        if (PROMPT_KERNEL != "mma" and v_pages is not None and kd == value_dim and v_pages.shape[3] == kd
                and lib.pb_attention_prefill_tc_plain_pages_supported(H, G, kd, page_size)):
            tc_tokens = lib.pb_attention_prefill_tc_tile_tokens(H, G)
            long_min = 1 if PROMPT_KERNEL == "tc" else max(2, int(tc_tokens * TC_MIN_FILL))
            tile_seq, tile_tok0, long_tiles = _prefill_plan(batch, tc_tokens, long_min, None)
            if long_tiles:
                check(lib.pb_attention_prefill_tc_masked_bf16(
                    q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), out.data_ptr(), table.data_ptr(), table.shape[1],
                    batch.positions.data_ptr(), batch.table_row_of_token.data_ptr(), batch.cu_q.data_ptr(), batch.q_start.data_ptr(),
                    tile_seq.data_ptr(), tile_tok0.data_ptr(), long_tiles, page_size, num_pages, T, H, G, kd, float(scale), int(window or 0), 0,
                    int(keep_first or 0), int(chunk or 0), float(softcap or 0.0), K._ptr(sink), K._ptr(gate),
                    0 if gate is None else gate.stride(0), batch.status.data_ptr(), _l.current_stream_ptr(q.device)),
                    "attention_prefill_tc_masked")
        tile_seq, tile_tok0, n_tiles = _prefill_plan(batch, lib.pb_attention_paged_tc_tile_tokens(H, G), 0, long_min)
        if n_tiles == 0:
            return out
    # few rows: deal each row's keys to several blocks, until the device is about twice full
    max_ctx = batch.max_kv_len if batch.max_kv_len else table.shape[1] * page_size
    if window:
        max_ctx = min(max_ctx, window + (keep_first or 0) + batch.max_q_len + 64)
    elif chunk:
        max_ctx = min(max_ctx, chunk + 32)
    blocks = n_tiles * G * (-(-(H // G) // 32))
    splits = 1
    # (putting the parts together writes every row of the step: not beside rows that the prompt kernel wrote)
    if blocks < _sm_count(q.device) and (batch.decode_only or not long_tiles):
        key_tiles = -(-max_ctx // 32)
        splits = max(1, min(MAX_SPLITS, 2 * _sm_count(q.device) // blocks, key_tiles))    # two blocks a multiprocessor: one wave
        splits = -(-key_tiles // -(-key_tiles // splits))               # as many blocks as have tiles to work on
    scratch = None
    if splits > 1:
        scratch = batch.workspace("general_attention_parts", (lib.pb_attention_paged_tc_scratch_floats(T, H, value_dim, splits),), torch.float32)
    vp = k_pages if v_pages is None else v_pages
    check(lib.pb_attention_paged_tc_bf16(
        q.data_ptr(), k_pages.data_ptr(), vp.data_ptr(), out.data_ptr(), K._ptr(sink), batch.positions.data_ptr(),
        batch.table_row_of_token.data_ptr(), table.data_ptr(), table.shape[1], batch.cu_q.data_ptr(), K._ptr(tile_seq), K._ptr(tile_tok0),
        n_tiles, page_size, num_pages, T, H, G, kd, value_dim, vp.shape[3], 1 if v_pages is None else 0, float(scale), int(window or 0),
        int(keep_first or 0), int(chunk or 0), float(softcap or 0.0), K._ptr(gate), 0 if gate is None else gate.stride(0),
        splits, K._ptr(scratch), batch.status.data_ptr(), _l.current_stream_ptr(q.device)), "attention_paged_tc")
    return out


# -- keys and values of every query head's own in dense rows (made of a latent for a long prompt portion) -----------------
ROW_BLOCK = 128                       # rows of a block of the dense rows, keys of a tile of the tcgen05 prompt kernel
ROWS_MIN_PORTION = int(256 * TC_MIN_FILL)         # tokens from which a portion fills that kernel's blocks
# most rows (cached tokens of all long portions of a step) for which keys and values are made per head
ROWS_MAX = int(os.environ.get("PRELUDE_LATENT_ROWS_MAX", str(1 << 16)))


class RowsPlan:
    """Which blocks of 128 dense rows a step's long portions need: block b holds positions ``block_pos0[b]`` .. of request
    ``block_seq[b]``; ``row_blocks`` [requests, stride] lists a request's blocks by position / 128 (0 where it has none, also
    for blocks that the window has passed)."""

    def __init__(self, block_seq, block_pos0, row_blocks, n_blocks: int, all_long: bool, window: Optional[int] = None):
        self.block_seq, self.block_pos0, self.row_blocks, self.n_blocks, self.all_long = block_seq, block_pos0, row_blocks, n_blocks, all_long
        self.window = window


def rows_plan(batch, window: Optional[int] = None) -> Optional[RowsPlan]:
    """The plan of a step's portions of ``ROWS_MIN_PORTION`` tokens and more (made once per step and window), or None where
    there is none or the tokens they see together are more than ``ROWS_MAX``."""
    key = ("rows_plan", window) if window else "rows_plan"
    if key in batch.extras:
        return batch.extras[key]
    plan = None
    lens, ctx = np.asarray(batch.q_lens), np.asarray(batch.kv_len_host)
    long = np.nonzero(lens >= ROWS_MIN_PORTION)[0]
    first = np.zeros(long.size, dtype=np.int64)              # the first block that a token of the portion sees
    if window:
        first = np.maximum(np.asarray(batch.q_start_host)[long] - window + 1, 0) // ROW_BLOCK
    if long.size and int((ctx[long] - first * ROW_BLOCK).sum()) <= ROWS_MAX:
        ends = -(-ctx[long] // ROW_BLOCK)
        n, stride = int((ends - first).sum()), int(ends.max())
        host = np.zeros(2 * n + lens.shape[0] * stride, dtype=np.int32)
        table = host[2 * n:].reshape(lens.shape[0], stride)
        at = 0
        for r, b0, b1 in zip(long.tolist(), first.tolist(), ends.tolist()):
            k = b1 - b0
            host[at:at + k] = r
            host[n + at:n + at + k] = np.arange(b0, b1, dtype=np.int32) * ROW_BLOCK
            table[r, b0:b1] = np.arange(at, at + k, dtype=np.int32)
            at += k
        dev = torch.from_numpy(host).to(batch.token_ids.device, non_blocking=True)
        plan = RowsPlan(dev[:n], dev[n:2 * n], dev[2 * n:].view(lens.shape[0], stride), n, bool((lens >= ROWS_MIN_PORTION).all()), window)
    batch.extras[key] = plan
    return plan


def rows_supported(kd: int, vd: int, row: int) -> bool:
    return row % 8 == 0 and bool(_l.library().pb_attention_prefill_tc_rows_supported(kd, vd))


def gather_rows(pages: torch.Tensor, batch, group: int, plan: RowsPlan) -> torch.Tensor:
    """The cached rows of the plan's blocks out of ``pages`` [num_pages, 1, page_size, width]: [blocks * 128, width], zeros behind
    a request's last token and where the plan's window has passed."""
    num_pages, one, page_size, width = pages.shape
    if one != 1 or pages.dtype != torch.bfloat16:
        raise _l.KernelLibraryError("gather_rows: one head of bfloat16 rows")
    out = batch.workspace("latent_rows", (plan.n_blocks * ROW_BLOCK, width), pages.dtype)
    table = batch.block_tables[group]
    check(_l.library().pb_rows_gather_bf16(
        pages.data_ptr(), out.data_ptr(), plan.block_seq.data_ptr(), plan.block_pos0.data_ptr(), plan.n_blocks, batch.kv_len.data_ptr(),
        batch.cu_q.data_ptr(), batch.table_row_of_token.data_ptr(), table.data_ptr(), table.shape[1], page_size, num_pages, width,
        batch.q_start.data_ptr(), int(plan.window or 0), batch.status.data_ptr(), _l.current_stream_ptr(out.device)), "rows_gather")
    return out


def attention_rows(q: torch.Tensor, kv: torch.Tensor, value_dim: int, batch, plan: RowsPlan, scale: float, sink: Optional[torch.Tensor],
                   gate: Optional[torch.Tensor], out: torch.Tensor) -> torch.Tensor:
    """Causal attention of the plan's long portions over dense rows (inside the plan's window): q [T, H, kd], kv [blocks * 128,
    H * (kd + value_dim)] (a head's key before its value), out [T, H, value_dim] (the other portions' rows are left alone); the
    tcgen05 prompt kernel.  ``gate``: columns [T, H], a number a head, or [T, H * value_dim], one an element, or None."""
    T, H, kd = q.shape
    lib = _l.library()
    if kv.shape != (plan.n_blocks * ROW_BLOCK, H * (kd + value_dim)) or tuple(out.shape) != (T, H, value_dim) or not kv.is_contiguous():
        raise _l.KernelLibraryError(f"attention_rows: q {tuple(q.shape)}, rows {tuple(kv.shape)}, out {tuple(out.shape)}")
    if gate is not None and tuple(gate.shape) not in ((T, H), (T, H * value_dim)):
        raise _l.KernelLibraryError(f"attention_rows: a gate {tuple(gate.shape)} for {T} tokens, {H} heads of {value_dim}")
    tile_seq, tile_tok0, n_tiles = _prefill_plan(batch, 256, ROWS_MIN_PORTION, None)
    check(lib.pb_attention_prefill_tc_rows_bf16(
        q.data_ptr(), kv.data_ptr(), out.data_ptr(), plan.row_blocks.data_ptr(), plan.row_blocks.shape[1], plan.n_blocks,
        batch.positions.data_ptr(), batch.token_seq.data_ptr(), batch.cu_q.data_ptr(), batch.q_start.data_ptr(), tile_seq.data_ptr(),
        tile_tok0.data_ptr(), n_tiles, T, H, kd, value_dim, float(scale), int(plan.window or 0), K._ptr(sink), K._ptr(gate),
        0 if gate is None else gate.stride(0), 0 if gate is None or gate.shape[1] == H else 1,
        batch.status.data_ptr(), _l.current_stream_ptr(q.device)), "attention_prefill_tc (rows)")
    return out
