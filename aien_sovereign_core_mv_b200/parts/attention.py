"""Grouped-query attention over the paged cache."""
from __future__ import annotations

import math
from typing import Optional

import torch

from .. import kernels as K
from ..registry import register_mixer
from .base import CacheNeed, Mixer, Position, Prenormed, ResidualSink, RunBinding, StepContext
from .linear import linear, linear_into_residual, linear_prenormed


@register_mixer("paged_attention")
class PagedAttention(Mixer):
    """q/k/v projection (one product over the stacked rows q|k|v), optional per-head RMSNorm of
    q and k before rotation, rotation, write of k and v into the token's cache slot, causal
    attention over the request's pages (optionally only the last ``window`` keys), output
    projection.  Formulas: crates/aien-inference-abi/src/transformer_backend.rs:1229-1319 and
    src/backend.rs:311-379; the stacked q|k|v rows follow src/resident.rs:284-288.

    A run that does not write its cache (``run.writes == False``) projects q only and attends
    over the planes another run filled."""

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, position: Position,
                 qk_norm: bool = False, qk_norm_eps: float = 1e-6, window: int = 0, scale: Optional[float] = None):
        if num_heads % num_kv_heads:
            raise ValueError(f"num_heads {num_heads} is not a multiple of num_kv_heads {num_kv_heads}")
        if head_dim % 2 or head_dim > 256:
            raise ValueError(f"head_dim {head_dim}: the attention kernels take even sizes up to 256")
        if getattr(position, "pairing", "halves") != "halves":
            raise ValueError("this mixer rotates halves (i with i + d/2); interleaved pairs belong to 'chunked_sink_attention'")
        self.hidden_size, self.num_heads, self.num_kv_heads, self.head_dim = int(hidden_size), int(num_heads), int(num_kv_heads), int(head_dim)
        self.position = position
        self.qk_norm, self.qk_norm_eps = bool(qk_norm), float(qk_norm_eps)
        self.window = int(window or 0)
        self.scale = float(scale) if scale is not None else 1.0 / math.sqrt(head_dim)
        self.q_dim, self.kv_dim = self.num_heads * self.head_dim, self.num_kv_heads * self.head_dim
        self.w_qkv = self.w_o = self.q_norm_w = self.k_norm_w = None

    # ---- tensors
    def param_shapes(self):
        H = self.hidden_size
        shapes = {
            "q_proj": ((self.q_dim, H), "matrix"), "k_proj": ((self.kv_dim, H), "matrix"),
            "v_proj": ((self.kv_dim, H), "matrix"), "o_proj": ((H, self.q_dim), "matrix"),
        }
        if self.qk_norm:
            shapes["q_norm"] = ((self.head_dim,), "norm")
            shapes["k_norm"] = ((self.head_dim,), "norm")
        return shapes

    def bind(self, tensors):
        q, k, v = tensors["q_proj"], tensors["k_proj"], tensors["v_proj"]
        if not (q.dtype == k.dtype == v.dtype):
            q, k, v = q.float(), k.float(), v.float()
        self.w_qkv = torch.cat([q, k, v], dim=0).contiguous()       # rows q | k | v
        self.w_o = tensors["o_proj"].contiguous()
        if self.qk_norm:
            qn, kn = tensors["q_norm"], tensors["k_norm"]
            if qn.dtype != kn.dtype:
                qn, kn = qn.float(), kn.float()
            self.q_norm_w, self.k_norm_w = qn.contiguous(), kn.contiguous()

    def cache_need(self):
        return CacheNeed.keys_and_values("window" if self.window > 0 else "full", self.window, self.num_kv_heads, self.head_dim)

    def workspace_bytes(self, lim):
        return lim.max_tokens * (2 * self.q_dim + 2 * self.kv_dim + self.q_dim + self.hidden_size) * lim.itemsize + 4096 \
            + 8 * K.GEMV_MAX_ROWS * (self.q_dim + 2 * self.kv_dim + self.hidden_size) * 4 + 2 * K.PARTIALS_MAX_BYTES \
            + K.attention_workspace_bytes(lim, self.num_heads, self.head_dim) + K.FUSED_NORM_SCRATCH_BYTES(self.hidden_size)

    # ---- one step
    takes_prenormed = True
    feeds_residual = True

    def _project(self, ctx: StepContext, h, w: torch.Tensor) -> torch.Tensor:
        if isinstance(h, Prenormed):
            y = linear_prenormed(ctx, h, w)
            if y is not None:
                return y
            h = h.materialise(ctx)
        return linear(ctx, h, w, may_defer_sum=True)

    def forward(self, ctx: StepContext, h, run: RunBinding, sink: Optional[ResidualSink] = None):
        T = ctx.num_tokens
        group = ctx.groups[run.group]
        k_cache, v_cache = group.storage["k"][run.slot], group.storage["v"][run.slot]     # [tokens, nkv, hd] each
        if run.writes:
            qkv = self._project(ctx, h, self.w_qkv)
            q, k, v = qkv[..., :self.q_dim], qkv[..., self.q_dim:self.q_dim + self.kv_dim], qkv[..., self.q_dim + self.kv_dim:]
        else:
            q = self._project(ctx, h, self.w_qkv[:self.q_dim])
            k = v = None
        rot = self.position.rotary(ctx)
        cos, sin, rdim = rot if rot is not None else (None, None, 0)
        if (K._FORCE_ATTN == "fused" and ctx.decode_only and run.writes and q.dim() == 2 and rot is not None
                and K.decode_attention_supports(q, k_cache, self.num_heads, self.num_kv_heads, self.head_dim)):
            # One launch: q/k norm, rotation, cache write and attention.  Opt-in (AIEN_B200_ATTENTION=fused):
            # measured on the Qwen3-8B shape it equals the two launches at batch 1 and loses at batch 8
            # and 64, where every chunk's CTA repeats the q work.
            out = ctx.workspace.take((T, self.q_dim), ctx.dtype)
            K.paged_attention_decode_fused(ctx, q, k, v, self.q_norm_w, self.k_norm_w, self.qk_norm_eps, cos, sin, rdim, group,
                                           k_cache, v_cache, out, self.num_heads, self.num_kv_heads, self.head_dim,
                                           self.window, self.scale)
            return linear(ctx, out, self.w_o, may_defer_sum=True)
        q_out = ctx.workspace.take((T, self.q_dim), ctx.dtype) if q.dim() == 3 else q
        K.qk_norm_rope_kv_write(q, k, v, self.head_dim, self.q_norm_w, self.k_norm_w if k is not None else None,
                                self.qk_norm_eps, cos, sin, rdim,
                                group.slot_map if k is not None else None,
                                k_cache if k is not None else None, v_cache if k is not None else None, q_out=q_out)
        if rot is None:
            self.position.apply(ctx, q_out, group, run)
        out = ctx.workspace.take((T, self.q_dim), ctx.dtype)
        K.paged_attention(ctx, q_out, k_cache, v_cache, group, out, self.num_heads, self.num_kv_heads, self.head_dim,
                          self.window, self.scale)
        return linear_into_residual(ctx, out, self.w_o, sink) or linear(ctx, out, self.w_o, may_defer_sum=True)


from .state_space import BranchMixer            # noqa: E402  (the two-products form this mixer follows)


@register_mixer("gated_capped_attention")
class GatedCappedAttention(BranchMixer):
    """Grouped-query attention with a capped score and an output gate.  q = W_q h (``num_heads`` heads of ``head_dim``),
    k = W_k h, v = W_v h (``num_kv_heads`` heads; values of ``value_dim`` numbers), with ``bias`` one vector each added; q and
    k are rotated over the dimensions the position part names (halves: i with i + d/2; the rest pass unchanged); score =
    q.k * ``scale``, then (``softcap`` c > 0) c * tanh(score / c); causal, optionally only the last ``window`` keys or the
    keys of the token's own chunk of ``chunk`` positions (counted from position 0 of the sequence); ordinary softmax.  The
    concatenated heads are multiplied element by element by sigmoid(W_g h) (``gate``) and projected by W_o.  One product
    makes q | k | v | g.  Rotation, scores, softmax and the gate are float32 in both engine precisions."""

    key_maps = 1                 # attention maps per head, each with queries and keys of its own over the same values

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, position: Position,
                 value_dim: Optional[int] = None, scale: Optional[float] = None, softcap: float = 0.0, window: int = 0, gate: bool = True,
                 chunk: int = 0, bias: bool = False):
        if num_heads % num_kv_heads:
            raise ValueError(f"num_heads {num_heads} is not a multiple of num_kv_heads {num_kv_heads}")
        self.hidden_size, self.num_heads, self.num_kv_heads, self.head_dim = int(hidden_size), int(num_heads), int(num_kv_heads), int(head_dim)
        self.value_dim = int(value_dim if value_dim is not None else head_dim)
        if not (0 < self.head_dim <= 256 and 0 < self.value_dim <= 256):
            raise ValueError(f"head sizes {self.head_dim} / {self.value_dim}: the attention kernels take sizes up to 256")
        if getattr(position, "pairing", "halves") != "halves":
            raise ValueError("this mixer rotates halves (i with i + d/2)")
        self.position = position
        self.scale = float(scale) if scale is not None else self.head_dim ** -0.5
        self.softcap, self.window, self.chunk, self.gate, self.bias = float(softcap or 0.0), int(window or 0), int(chunk or 0), bool(gate), bool(bias)
        if self.softcap < 0.0 or self.window < 0 or self.chunk < 0:
            raise ValueError("softcap, window and chunk must not be negative")
        if self.window and self.chunk:
            raise ValueError("a window or a chunk mask, not both")
        n = self.key_maps
        self.q_dim, self.k_dim, self.v_dim = n * self.num_heads * self.head_dim, n * self.num_kv_heads * self.head_dim, self.num_kv_heads * self.value_dim
        self.out_cols = self.num_heads * self.value_dim
        self.in_rows = self.q_dim + self.k_dim + self.v_dim + (self.out_cols if self.gate else 0)
        self.w_in = self.w_o = self.b_in = None

    def param_shapes(self):
        H = self.hidden_size
        shapes = {"q_proj": ((self.q_dim, H), "matrix"), "k_proj": ((self.k_dim, H), "matrix"), "v_proj": ((self.v_dim, H), "matrix"),
                  "o_proj": ((H, self.out_cols), "matrix")}
        if self.bias:
            shapes.update({"q_bias": ((self.q_dim,), "small"), "k_bias": ((self.k_dim,), "small"), "v_bias": ((self.v_dim,), "small")})
        if self.gate:
            shapes["g_proj"] = ((self.out_cols, H), "matrix")
        return shapes

    def query_rows(self, t: torch.Tensor) -> torch.Tensor:
        """Rows of the query projection (or its bias) in the order the kernels take the query heads."""
        return t

    def bind(self, tensors):
        rows = [self.query_rows(tensors["q_proj"]), tensors["k_proj"], tensors["v_proj"]] + ([tensors["g_proj"]] if self.gate else [])
        if len({t.dtype for t in rows}) > 1:
            rows = [t.float() for t in rows]
        self.w_in = torch.cat(rows, dim=0).contiguous()                 # rows q | k | v | g
        self.w_o = tensors["o_proj"].contiguous()
        if self.bias:
            self.b_in = torch.cat([self.query_rows(tensors["q_bias"]).float(), tensors["k_bias"].float(), tensors["v_bias"].float()]).contiguous()

    def in_weight(self):
        return self.w_in

    def out_weight(self):
        return self.w_o

    def cache_need(self):
        planes = (("k", (self.key_maps * self.num_kv_heads, self.head_dim)), ("v", (self.num_kv_heads, self.value_dim)))
        if self.chunk > 0:
            return CacheNeed("chunk", self.chunk, planes)
        return CacheNeed("window" if self.window > 0 else "full", self.window, planes)

    def store(self, ctx, run):
        group = ctx.groups[run.group]
        return group, group.storage["k"][run.slot], group.storage["v"][run.slot]

    def core_workspace_bytes(self, lim):
        n = self.key_maps
        return lim.max_tokens * (self.q_dim * lim.itemsize + n * self.out_cols * 4) + 1024 \
            + K.capped_attention_workspace_bytes(lim, n * self.num_heads, self.value_dim, self.window, self.chunk)

    def prepare(self, ctx, proj, col0, store):
        """Biases, rotation and cache write of the step's tokens; the queries [T, maps * heads * head_dim]."""
        n = self.key_maps
        group, k_cache, v_cache = store
        if col0 and self.b_in is not None:
            raise ValueError("a mixer with biases does not share its first product")
        rot = self.position.rotary(ctx)
        cos, sin, rdim = rot if rot is not None else (None, None, 0)
        q = ctx.workspace.take((ctx.num_tokens, self.q_dim), ctx.dtype)
        K.rope_halves_value_write(proj, col0, col0 + self.q_dim, col0 + self.q_dim + self.k_dim, n * self.num_heads, n * self.num_kv_heads,
                                  self.head_dim, self.value_dim, cos, sin, rdim, group.slot_map, q, k_cache, v_cache, bias=self.b_in,
                                  nv=self.num_kv_heads)
        return q

    def core(self, ctx, proj, col0, store, out, out_col0, mult):
        T = ctx.num_tokens
        q = self.prepare(ctx, proj, col0, store)
        group, k_cache, v_cache = store
        dst = out[:, out_col0:out_col0 + self.out_cols]
        gated = self.gate or mult != 1.0
        o = ctx.workspace.take((T, self.out_cols), ctx.dtype) if gated else dst
        K.capped_attention(ctx, q, k_cache, v_cache, group, o, self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim,
                           self.window, self.scale, self.softcap, self.chunk)
        if self.gate:
            g0 = col0 + self.q_dim + self.k_dim + self.v_dim
            K.sigmoid_gate(o, proj[:, g0:g0 + self.out_cols], mult, dst)
        elif gated:
            K.scale_rows(o, mult, dst)


class _PlainOutput(GatedCappedAttention):
    """The forms without an output gate: the first product may leave partial products (the rotation's kernel adds them) and
    its rows in the compute dtype; the last one leaves its sum to the next norm."""

    feeds_residual = True

    def __init__(self, *args, **kwargs):
        super().__init__(*args, gate=False, **kwargs)

    def workspace_bytes(self, lim):
        return super().workspace_bytes(lim) + K.PARTIALS_MAX_BYTES + K.FUSED_NORM_SCRATCH_BYTES(self.hidden_size)

    def forward(self, ctx: StepContext, h: torch.Tensor, run: RunBinding, sink: Optional[ResidualSink] = None):
        proj = linear(ctx, h, self.w_in, may_defer_sum=True)
        y = ctx.workspace.take((ctx.num_tokens, self.out_cols), ctx.dtype)
        self.core(ctx, proj, 0, self.store(ctx, run), y, 0, 1.0)
        return linear_into_residual(ctx, y, self.w_o, sink) or linear(ctx, y, self.w_o, may_defer_sum=True)


@register_mixer("value_attention")
class ValueAttention(_PlainOutput):
    """Grouped-query attention with values of their own size, rotated halves, an optional chunk mask or window, an optional
    cap on the score and optional biases (see :class:`GatedCappedAttention`), without an output gate."""


@register_mixer("differential_attention")
class DifferentialAttention(_PlainOutput):
    """Two attention maps per head over the same values, combined by their difference.  W_q h holds per query head and W_k h
    per key/value head the numbers of map 1 and then those of map 2 (``head_dim`` each); each map is an attention of its own
    (rotation, scale, cap, mask, softmax).  With a1, a2 the maps' outputs of a head and the layer's one number
    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + ``diff``: o = a1 - lambda * a2, divided by sqrt(mean(o^2) + ``norm_eps``) over
    the head's values and multiplied by 1 - ``diff``; then W_o.

    The query rows are stored group by group, map 1 of the group's heads before map 2, so that to the attention kernels the
    maps are key heads of their own, two of which share a value head.  The maps' outputs, their difference and its norm
    are float32 in both engine precisions."""

    key_maps = 2

    def __init__(self, *args, diff: float = 0.0, norm_eps: float = 1e-6, **kwargs):
        super().__init__(*args, **kwargs)
        self.diff, self.norm_eps = float(diff), float(norm_eps)
        self.lam = 0.0

    def param_shapes(self):
        shapes = dict(super().param_shapes())
        for n in ("lq1", "lk1", "lq2", "lk2"):
            shapes[n] = ((self.head_dim,), "small")
        return shapes

    def query_rows(self, t):
        per, g, d = self.num_heads // self.num_kv_heads, self.num_kv_heads, self.head_dim
        return t.reshape(g, per, 2, d, *t.shape[1:]).transpose(1, 2).reshape(t.shape)

    def bind(self, tensors):
        super().bind(tensors)
        dot = lambda a, b: float((tensors[a].double() * tensors[b].double()).sum())
        self.lam = math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + self.diff

    def core(self, ctx, proj, col0, store, out, out_col0, mult):
        q = self.prepare(ctx, proj, col0, store)
        group, k_cache, v_cache = store
        K.difference_attention(ctx, q, k_cache, v_cache, group, out[:, out_col0:out_col0 + self.out_cols], self.num_heads, self.num_kv_heads,
                               self.head_dim, self.value_dim, self.window, self.scale, self.softcap, self.chunk, self.lam, self.norm_eps,
                               (1.0 - self.diff) * mult)
