"""Dense gated feed-forward."""
from __future__ import annotations

import torch

from .. import kernels as K
from ..registry import register_feed_forward
from typing import Optional

from .base import FeedForward, Prenormed, ResidualSink, StepContext
from .linear import linear, linear_into_residual, linear_prenormed, _FORCE


@register_feed_forward("swiglu")
class SwiGLU(FeedForward):
    """y = (act(h Wg^T) * (h Wu^T)) Wd^T with ``act`` "silu" (or "gelu_tanh", the tanh form of the gelu), no bias (crates/aien-inference-abi/src/
    transformer_backend.rs:1322-1362, silu in src/backend.rs:572-579).  gate and up are one
    product over the stacked rows gate | up (src/resident.rs:284-288)."""

    def __init__(self, hidden_size: int, intermediate_size: int, act: str = "silu"):
        self.hidden_size, self.intermediate_size = int(hidden_size), int(intermediate_size)
        if act not in K.GATED_ACTS:
            raise ValueError(f"activation {act!r}: known are {sorted(K.GATED_ACTS)}")
        self.act, self.epilogue = act, K.GATED_ACTS[act]
        self.w_gate_up = self.w_down = None

    def param_shapes(self):
        H, I = self.hidden_size, self.intermediate_size
        return {"gate_proj": ((I, H), "matrix"), "up_proj": ((I, H), "matrix"), "down_proj": ((H, I), "matrix")}

    GROUP = 8      # gate and up rows interleaved in runs of 8: one decode-kernel tile holds both

    def bind(self, tensors):
        g, u = tensors["gate_proj"], tensors["up_proj"]
        if g.dtype != u.dtype:
            g, u = g.float(), u.float()
        I, H = self.intermediate_size, self.hidden_size
        self.group = self.GROUP if (g.dtype == torch.bfloat16 and I % self.GROUP == 0) else 0
        if self.group:
            n = I // self.group
            self.w_gate_up = torch.stack([g.view(n, self.group, H), u.view(n, self.group, H)], dim=1).reshape(2 * I, H).contiguous()
        else:
            self.w_gate_up = torch.cat([g, u], dim=0).contiguous()
        self.w_down = tensors["down_proj"].contiguous()

    def workspace_bytes(self, lim):
        return lim.max_tokens * (3 * self.intermediate_size + self.hidden_size) * lim.itemsize + 4096 \
            + 8 * K.GEMV_MAX_ROWS * self.hidden_size * 4 + K.PARTIALS_MAX_BYTES + K.FUSED_NORM_SCRATCH_BYTES(self.hidden_size)

    takes_prenormed = True
    feeds_residual = True

    def hidden(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        """act(h Wg^T) * (h Wu^T)."""
        act = ctx.workspace.take((ctx.num_tokens, self.intermediate_size), ctx.dtype)
        if self.group == 8 and h.shape[0] <= K.GEMV_ROUTE_ROWS and K.gemv_supports(h, self.w_gate_up, act):
            K.gemv(h, self.w_gate_up, act, epilogue=self.epilogue)      # act(gate)*up inside the product
        elif self.group == 8 and K.gemm_tc_supports(h, self.w_gate_up, act) and not _FORCE:
            K.gemm_tc(h, self.w_gate_up, act, epilogue=self.epilogue)   # the same, in the tensor-core epilogue
        else:
            gu = linear(ctx, h, self.w_gate_up)
            K.swiglu(gu, act, self.group, self.act)
        return act

    def forward(self, ctx: StepContext, h, sink: Optional[ResidualSink] = None):
        if isinstance(h, Prenormed):
            act = linear_prenormed(ctx, h, self.w_gate_up, epilogue=1) if self.group == 8 and self.act == "silu" else None
            if act is not None:
                return linear_into_residual(ctx, act, self.w_down, sink) or linear(ctx, act, self.w_down, may_defer_sum=True)
            h = h.materialise(ctx)
        act = self.hidden(ctx, h)
        return linear_into_residual(ctx, act, self.w_down, sink) or linear(ctx, act, self.w_down, may_defer_sum=True)


@register_feed_forward("mlp_act")
class ActMLP(FeedForward):
    """y = W_down act(W_up h), no gate and no bias; ``act``: "gelu_tanh", "gelu" (the erf form) or "relu2" (the square of
    relu).  The activation runs in the first product's epilogue where the kernel has one."""

    def __init__(self, hidden_size: int, intermediate_size: int, act: str = "gelu_tanh"):
        self.hidden_size, self.intermediate_size = int(hidden_size), int(intermediate_size)
        if act not in K.ACT_KINDS:
            raise ValueError(f"activation {act!r}: known are {sorted(K.ACT_KINDS)}")
        self.act = K.ACT_KINDS[act]
        self.w_up = self.w_down = None

    def param_shapes(self):
        H, I = self.hidden_size, self.intermediate_size
        return {"up": ((I, H), "matrix"), "down": ((H, I), "matrix")}

    def bind(self, tensors):
        self.w_up, self.w_down = tensors["up"].contiguous(), tensors["down"].contiguous()

    def workspace_bytes(self, lim):
        return lim.max_tokens * (self.intermediate_size * lim.itemsize + self.hidden_size * 4) + 4096 + K.PARTIALS_MAX_BYTES

    def forward(self, ctx: StepContext, h: torch.Tensor):
        a = linear(ctx, h, self.w_up, act=self.act)
        return linear(ctx, a, self.w_down, out_dtype=torch.float32, may_defer_sum=True)    # the branch norm adds partial products


@register_feed_forward("clamped_glu")
class ClampedGLU(FeedForward):
    """g = min(W_gate h + b_gate, ``limit``), u = clamp(W_up h + b_up, -limit, limit); y = W_down (g * sigmoid(``alpha`` g)
    * (u + 1)) + b_down.  One product makes gate | up; its float32 result, the biases and the activation meet in one
    kernel.  The last bias is handed to the consumer of the branch (``pending_bias``), which adds it with the sum."""

    def __init__(self, hidden_size: int, intermediate_size: int, limit: float, alpha: float = 1.702, bias: bool = True):
        self.hidden_size, self.intermediate_size = int(hidden_size), int(intermediate_size)
        self.limit, self.alpha, self.bias = float(limit), float(alpha), bool(bias)
        if not self.limit > 0.0:
            raise ValueError(f"limit {limit!r} must be positive")
        self.w_gate_up = self.w_down = self.b_gate = self.b_up = self.b_down = None

    def param_shapes(self):
        H, I = self.hidden_size, self.intermediate_size
        shapes = {"gate": ((I, H), "matrix"), "up": ((I, H), "matrix"), "down": ((H, I), "matrix")}
        if self.bias:
            shapes.update({"gate_bias": ((I,), "small"), "up_bias": ((I,), "small"), "down_bias": ((H,), "small")})
        return shapes

    def bind(self, tensors):
        g, u = tensors["gate"], tensors["up"]
        if g.dtype != u.dtype:
            g, u = g.float(), u.float()
        self.w_gate_up = torch.cat([g, u], dim=0).contiguous()           # rows gate | up
        self.w_down = tensors["down"].contiguous()
        if self.bias:
            self.b_gate, self.b_up = tensors["gate_bias"].float().contiguous(), tensors["up_bias"].float().contiguous()
            self.b_down = tensors["down_bias"].float().contiguous()

    def workspace_bytes(self, lim):
        I = self.intermediate_size
        return lim.max_tokens * (2 * I * 4 + I * lim.itemsize + self.hidden_size * 4) + 8192 + K.PARTIALS_MAX_BYTES

    def pending_bias(self):
        return self.b_down

    def forward(self, ctx: StepContext, h: torch.Tensor):
        I = self.intermediate_size
        gu = linear(ctx, h, self.w_gate_up, out_dtype=torch.float32)
        act = ctx.workspace.take((ctx.num_tokens, I), ctx.dtype)
        K.clamped_glu(gu, 0, I, I, self.b_gate, self.b_up, self.limit, self.alpha, act)
        return linear(ctx, act, self.w_down, out_dtype=torch.float32, may_defer_sum=True)
