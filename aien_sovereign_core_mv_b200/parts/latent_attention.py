"""Attention whose keys and values are made from one cached latent per token."""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels as K
from ..registry import register_mixer
from .base import CacheNeed, Mixer, Position, RunBinding, StepContext
from .linear import linear, stack_rows


@register_mixer("latent_attention")
class LatentAttention(Mixer):
    """Queries through a latent: c_q = RMSnorm(W_dq h) (weight ``dq_norm``), q = W_uq c_q, per head ``head_dim``
    unrotated then ``rot_dim`` rotated numbers; without a ``q_rank`` (0) q = W_q h.  Keys and values through a latent: W_dkv h has ``kv_rank`` + ``rot_dim``
    rows; the first kv_rank, RMS-normed (weight ``dkv_norm``), are the latent c, the rest one rotated key part shared by
    all heads.  Per head the unrotated key is W_uk c and the value W_uv c; score = (q_unrot . k_unrot + q_rot . k_rot) *
    ``scale``; causal, optionally only the last ``window`` positions (the token itself included); optionally a learned
    sink per head in the softmax denominator; optionally (``head_gate``) head h's output times sigmoid(W_g h)_h, or (``out_gate``) the concatenated
    heads element by element times sigmoid(W_g h); W_o on the heads.  The rotation turns neighbouring pairs of the first
    ``rotary_dim`` numbers of the rotated part (the position part's table).

    The cache keeps one row [c | k_rot] per token and nothing per head.  Two forms of the same sums read it.  *Absorbed*:
    no head's keys or values are built; W_uk is applied to the query (q_lat = W_uk,h^T q_unrot) and W_uv to the weighted
    sum of latents, so a cached row serves every head as key and as value.  *Expanded* (portions of prompts in a bfloat16
    engine, without a rotated part): the contexts' keys and values are made per head by one product for the length of the
    step, which costs less than carrying every score and sum at the latent's size as soon as a portion has more than
    a few dozen tokens (``kernels.latent_expand_takes``); single tokens beside them take the absorbed form.  ``own_cache`` False: the layer has no W_dkv and attends over the rows
    another layer wrote (its run binding names that layer's planes).  ``cache_window``: how many positions the cache
    must keep, when layers that share it have different windows (default: ``window``)."""

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, rot_dim: int, value_dim: int, kv_rank: int, q_rank: int,
                 position: Position, scale: Optional[float] = None, window: int = 0, cache_window: Optional[int] = None,
                 sink: bool = False, norm_eps: float = 1e-6, own_cache: bool = True, head_gate: bool = False,
                 out_gate: bool = False):
        self.hidden_size, self.num_heads, self.head_dim, self.rot_dim = int(hidden_size), int(num_heads), int(head_dim), int(rot_dim)
        self.value_dim, self.kv_rank, self.q_rank = int(value_dim), int(kv_rank), int(q_rank or 0)
        if min(self.num_heads, self.head_dim, self.value_dim, self.kv_rank) <= 0 or min(self.q_rank, self.rot_dim) < 0:
            raise ValueError("latent attention: heads, head_dim, value_dim and kv_rank must be positive")
        if self.rot_dim and getattr(position, "pairing", "interleaved") != "interleaved":
            raise ValueError("this mixer rotates neighbouring pairs (2i with 2i+1): give it a position part with pairing='interleaved'")
        self.position = position
        self.rotary_dim = int(getattr(position, "rotary_dim", 0) or 0) if self.rot_dim else 0
        if self.rotary_dim > self.rot_dim:
            raise ValueError(f"the position part rotates {self.rotary_dim} numbers, the rotated part has {self.rot_dim}")
        self.scale = float(scale) if scale is not None else (self.head_dim + self.rot_dim) ** -0.5
        self.window = int(window or 0)
        self.cache_window = self.window if cache_window is None else int(cache_window)
        if self.window < 0 or (self.window == 0) != (self.cache_window == 0) or self.cache_window < self.window:
            raise ValueError("cache_window must cover window (0 for both: every earlier position is seen)")
        self.sink, self.norm_eps, self.own_cache = bool(sink), float(norm_eps), bool(own_cache)
        self.head_gate, self.out_gate = bool(head_gate), bool(out_gate)
        if self.head_gate and self.out_gate:
            raise ValueError("latent attention: a gate per head or one per element, not both")
        self.q_head = self.head_dim + self.rot_dim
        self.gate_rows = self.num_heads if self.head_gate else (self.num_heads * self.value_dim if self.out_gate else 0)
        self.q_cols = self.q_rank or self.num_heads * self.q_head        # rows of the first product that belong to the query
        self.side_rows, self.riders = self.gate_rows, 0                  # and those behind them: gates, riders
        self.row = self.kv_rank + self.rot_dim
        # the expanded form of portions (a bfloat16 engine's)
        self._expandable = self.rot_dim == 0 and self.kv_rank % 8 == 0 and self.head_dim % 8 == 0 and self.value_dim % 8 == 0 \
            and max(self.head_dim, self.value_dim) <= 128
        self.w_kv = None
        self.w_down = self.w_uq = self.w_uk_t = self.w_uv = self.w_o = self.dq_norm = self.dkv_norm = self.sinks = None

    # ---- tensors
    def param_shapes(self):
        H, n = self.hidden_size, self.num_heads
        shapes = {"dq_proj": ((self.q_rank, H), "matrix"), "dq_norm": ((self.q_rank,), "norm"),
                  "uq_proj": ((n * self.q_head, self.q_rank), "matrix")} if self.q_rank else {"q_proj": ((n * self.q_head, H), "matrix")}
        shapes = {**shapes, "uk_proj": ((n * self.head_dim, self.kv_rank), "matrix"),
                  "uv_proj": ((n * self.value_dim, self.kv_rank), "matrix"), "o_proj": ((H, n * self.value_dim), "matrix")}
        if self.own_cache:
            shapes.update({"dkv_proj": ((self.row, H), "matrix"), "dkv_norm": ((self.kv_rank,), "norm")})
        if self.sink:
            shapes["sink"] = ((n,), "vector")
        if self.gate_rows:
            shapes["g_proj"] = ((self.gate_rows, H), "matrix")
        return shapes

    takes_riders = True

    def _stack(self, dq, side, dkv):
        """Rows query latent | head gates and riders, filled up to whole vectors | key/value latent | shared key part."""
        head = stack_rows([dq] + side, 8) if side else dq
        self.side_rows = head.shape[0] - self.q_cols
        self.w_down = stack_rows([head] + ([dkv] if dkv is not None else []))

    def set_riders(self, weight):
        w = self.w_down
        gates = [w[self.q_cols:self.q_cols + self.gate_rows]] if self.gate_rows else []
        dkv = w[self.q_cols + self.side_rows:] if self.own_cache else None
        self.riders = weight.shape[0]
        self._stack(w[:self.q_cols], gates + [weight], dkv)

    def bind(self, tensors):
        self._stack(tensors["dq_proj" if self.q_rank else "q_proj"], [tensors["g_proj"]] if self.gate_rows else [],
                    tensors["dkv_proj"] if self.own_cache else None)
        self.w_uq = tensors["uq_proj"].contiguous() if self.q_rank else None
        self.w_o = tensors["o_proj"].contiguous()
        n = self.num_heads
        # per head [kv_rank, head_dim]: the matrix that takes a head's unrotated query to the latent
        self.w_uk_t = tensors["uk_proj"].view(n, self.head_dim, self.kv_rank).transpose(1, 2).contiguous()
        self.w_uv = tensors["uv_proj"].view(n, self.value_dim, self.kv_rank).contiguous()
        if self._expandable and tensors["uk_proj"].dtype == torch.bfloat16 == tensors["uv_proj"].dtype:
            self.w_kv = torch.cat([tensors["uk_proj"], tensors["uv_proj"]], dim=0).contiguous()      # all heads' keys | all heads' values
        self.dq_norm = tensors["dq_norm"].contiguous() if self.q_rank else None
        if self.own_cache:
            self.dkv_norm = tensors["dkv_norm"].contiguous()
            if self.dq_norm is not None:
                self.dkv_norm = self.dkv_norm.to(self.dq_norm.dtype)
        if self.sink:
            self.sinks = tensors["sink"].float().contiguous()           # the softmax is float32

    def cache_need(self):
        planes = (("latent", (self.row,)),)
        return CacheNeed("window", self.cache_window, planes) if self.cache_window > 0 else CacheNeed("full", 0, planes)

    def workspace_bytes(self, lim):
        n = self.num_heads
        per_token = (self.q_cols + self.side_rows + self.row) * 4 + self.q_rank * lim.itemsize + n * self.q_head * 4 + n * self.row * 4 \
            + n * self.kv_rank * lim.itemsize + n * self.value_dim * lim.itemsize + self.hidden_size * 4
        # the partial results of a step with few tiles: tokens * heads * ksplit rows, which latent_attention_tc_ksplit keeps
        # below 296 tiles' worth of 64 rows
        split = 296 * K.LATENT_TC_TILE * (self.kv_rank + 2) * 4
        expand = 0
        if self._expandable and lim.itemsize == 2:
            rows = K.latent_expand_rows(lim.max_context, lim.max_seqs)
            per_row = n * (self.head_dim + self.value_dim) * 2
            rows = min(rows, K.LATENT_EXPAND_MAX_BYTES // per_row + 128)
            expand = rows * (per_row + self.kv_rank * 2) + lim.max_seqs * (lim.max_context // 128 + 2) * 4 + 4096
        return lim.max_tokens * per_token + 16384 + split + K.PARTIALS_MAX_BYTES + expand

    # ---- one step
    def _expanded(self, ctx, q, cache, group, portions, gate, o):
        """The portions' rows of ``o``: keys and values per head for the length of the step."""
        n, ws = self.num_heads, ctx.workspace
        length = K.latent_expand_rows(ctx.max_ctx_len, 1)
        lat = ws.take((portions * length, self.kv_rank), torch.bfloat16)
        table = ws.take((ctx.num_seqs, length // 128), torch.int32)
        K.latent_gather(cache, group, ctx.q_start, ctx.ctx_len, ctx.num_seqs, portions, length, lat, table)
        kv = linear(ctx, lat, self.w_kv)
        k, v = kv[:, :n * self.head_dim], kv[:, n * self.head_dim:]
        by_head = gate if self.head_gate else None
        element = gate if self.out_gate else None
        K.portion_attention(ctx, q, k, v, table, o, n, self.head_dim, self.value_dim, self.window, self.scale, self.sinks, by_head, element)

    def _absorbed(self, ctx, q, cache, group, tc, gate, o, rot, singles, n_single):
        """Rows of ``o`` over the latent itself: all of the step's, or those of ``singles`` (tokens that come alone)."""
        T, n, ws = ctx.num_tokens, self.num_heads, ctx.workspace
        cos, sin, rdims = rot if rot is not None else (None, None, 0)
        qf = ws.take((T, n * self.row), torch.bfloat16 if tc else torch.float32)    # per head: the query in the latent | rotated part
        K.head_project(q, self.q_head, 0, self.w_uk_t, qf, self.row, 0, rows=singles, num_rows=n_single)
        if self.rot_dim:
            K.rotate_pairs_rows(q, self.q_head, self.head_dim, qf, self.row, self.kv_rank, n, self.rot_dim, rdims, cos, sin)
        mixed = ws.take((T, n * self.kv_rank), ctx.dtype)
        if tc:
            alone = ctx.decode_only or singles is not None
            small = K.latent_attention_tc_small_tiles(alone, self.kv_rank)
            count = n_single if singles is not None else T
            ksplit = K.latent_attention_tc_ksplit(count, n_single if singles is not None else ctx.num_seqs, n, ctx.max_ctx_len, self.window, small)
            scratch = ws.take((K.latent_attention_tc_scratch(count, n, self.kv_rank, ksplit),), torch.float32) if ksplit > 1 else None
            K.latent_attention_tc(qf, cache, group.block_table, group.max_blocks, ctx.q_start, ctx.positions, mixed, ctx.num_seqs, n,
                                  self.kv_rank, self.rot_dim, group.page_size, self.window, self.scale, self.sinks, ksplit, scratch, small,
                                  singles, n_single)
        else:
            K.latent_attention(qf, cache, group.block_table, group.max_blocks, ctx.seq_of_token, ctx.positions, mixed, n, self.kv_rank,
                               self.rot_dim, group.page_size, self.window, self.scale, self.sinks)
        K.head_project(mixed, self.kv_rank, 0, self.w_uv, o, self.value_dim, 0, gate=gate, rows=singles, num_rows=n_single)

    def forward(self, ctx: StepContext, h: torch.Tensor, run: RunBinding):
        T, n, ws = ctx.num_tokens, self.num_heads, ctx.workspace
        group = ctx.groups[run.group]
        cache = group.storage["latent"][run.slot]                       # [tokens of the pool, kv_rank + rot_dim]
        writes = run.writes and self.own_cache
        if run.writes and not self.own_cache:
            raise RuntimeError("a latent-attention layer without its own key/value projection was bound to write a cache")
        kv_off = self.q_cols + self.side_rows
        w_down = self.w_down if writes else self.w_down[:kv_off]
        tc = K.latent_attention_tc_supports(cache.dtype, self.kv_rank, self.rot_dim) and ctx.dtype == torch.bfloat16
        # a query latent is normed in float32; without one the rows are an operand of the next product as they are
        d = linear(ctx, h, w_down, out_dtype=torch.float32 if self.q_rank or self.riders or not tc else torch.bfloat16)
        rot = self.position.rotary(ctx) if self.rotary_dim else None
        cos, sin, rdims = rot if rot is not None else (None, None, 0)
        cq = ws.take((T, self.q_rank), ctx.dtype) if self.q_rank else None
        K.latent_prepare(d, self.q_rank, self.dq_norm, self.norm_eps, cq, kv_off, self.kv_rank, self.rot_dim, rdims,
                         self.dkv_norm, cos, sin, group.slot_map if writes else None, cache if writes else None)
        # per head: unrotated | rotated part, before rotation; an operand of the tensor-core products where those run
        q = linear(ctx, cq, self.w_uq, out_dtype=torch.bfloat16 if tc else torch.float32) if self.q_rank else d
        gate = d[:, self.q_cols:self.q_cols + self.gate_rows] if self.gate_rows else None
        o = ws.take((T, n * self.value_dim), ctx.dtype)
        tiles = ctx.prefill_tiles[2] if ctx.prefill_tiles is not None and not ctx.decode_only else 0
        singles, n_single = ctx.single_tokens if ctx.single_tokens is not None else (None, 0)
        portions = ctx.num_seqs - n_single if tiles > 0 else 0
        gate_suits = gate is None or (gate.dtype == torch.float32 if self.head_gate else
                                      gate.dtype == torch.bfloat16 and gate.stride(0) % 8 == 0 and gate.data_ptr() % 16 == 0)
        expand = tc and self.w_kv is not None and q.dtype == torch.bfloat16 and q.stride(0) % 8 == 0 and gate_suits and \
            K.latent_expand_takes(T - n_single, portions, ctx.max_ctx_len, n, self.head_dim, self.value_dim, self.kv_rank)
        if expand:
            self._expanded(ctx, q[:, :n * self.q_head], cache, group, portions, gate, o)
        if not expand or n_single > 0:
            self._absorbed(ctx, q, cache, group, tc, gate, o, rot, singles if expand else None, n_single if expand else 0)
        y = linear(ctx, o, self.w_o, out_dtype=torch.float32, may_defer_sum=True)        # the consumer's norm adds partial products
        if not self.riders:
            return y
        r0 = self.q_cols + self.gate_rows
        return y, d[:, r0:r0 + self.riders]
