"""Parts that mix along the time axis in front of a mixer and along the depth axis behind a layer.

``CausalInputConv``: a short causal convolution added to what a mixer reads.  ``DepthAverage``: what a
layer hands on is a weighted sum of the embedding's output and of every layer's result so far.
"""

from __future__ import annotations

import torch

from ..csrc import ops
from .base import (BranchSum, InputPart, ParamDecl, PendingBranch, StateNeed, StreamCopy, StreamPart,
                   register_input_part, register_stream_part)
from .builtin import BranchLayerNorm, fp32_stream


class CausalInputConv(InputPart):
    """``h'_t = h_t + sum_j w[:, j] h_(t - taps + 1 + j)`` per channel, zeros before the sequence's start; the
    last ``taps - 1`` inputs are per-request state (fp32, oldest first).  The sum is fp32.

    params: ``hidden_size``, ``taps``.  tensors: ``weight [hidden_size, taps]``.
    """

    def __init__(self, spec):
        super().__init__(spec)
        self.hidden, self.taps = int(self.param("hidden_size")), int(self.param("taps"))
        if not 1 <= self.taps <= ops.INPUT_CONV_MAX_TAPS:
            raise ValueError(f"{self.taps} convolution taps (1 to {ops.INPUT_CONV_MAX_TAPS} are taken)")

    def param_decls(self):
        return {"weight": ParamDecl((self.hidden, self.taps), "table")}

    def state_need(self):
        return StateNeed((self.taps - 1, self.hidden), torch.float32) if self.taps > 1 else None

    def bind(self, tensors, dtype, device):
        self.weight_t = tensors["weight"].to(torch.float32).t().contiguous()     # [taps, hidden]: a tap's channels lie together
        self.dtype = dtype

    def forward(self, h, ctx, cache):
        return ops.input_conv(h, self.weight_t, cache.input_state, ctx, self.dtype)


class DepthAverage(StreamPart):
    """Behind layer ``index``: with ``X_0`` the embedding's output and ``X_(j+1)`` the result of layer ``j`` (the
    stream it hands on, before this part), the stream becomes ``sum_(j <= index + 1) weights[j] X_j``, all of it
    fp32.  The results are kept for the step, one tensor for all layers.

    The layer's last norm and sum run in the same kernel (``finishes_branch``); in steps of single tokens so
    does the next layer's input convolution (``prepares_input``).

    params: ``hidden_size``, ``index``, ``layers`` (of the model; behind the last one nothing is kept).
    tensors: ``weights [index + 2]``.
    """

    needs_embedding = True
    finishes_branch = True
    prepares_input = True

    def __init__(self, spec):
        super().__init__(spec)
        self.hidden = int(self.param("hidden_size"))
        self.index, self.layers = int(self.spec.params["index"]), int(self.param("layers"))
        if not 0 <= self.index < self.layers:
            raise ValueError(f"layer {self.index} of {self.layers}")

    def param_decls(self):
        return {"weights": ParamDecl((self.index + 2,), "table")}

    def bind(self, tensors, dtype, device):
        self.weights = tensors["weights"].to(torch.float32).contiguous()
        self.dtype = dtype

    def forward(self, x, residual, ctx, embedded, following=None):
        if embedded is None or embedded.dtype != torch.float32:
            raise ValueError("a depth average needs an fp32 embedding output")
        history = ctx.scratch.get("depth_results")
        if history is None:
            if self.index:
                raise ValueError("depth averages stand behind every layer, in order")
            kept = self.layers - 1
            history = torch.empty((kept, *embedded.shape), dtype=torch.float32, device=embedded.device)
            ctx.scratch["depth_results"] = history
        branch = norm = None
        if isinstance(x, PendingBranch):
            branch, norm = x.branch, x.norm
            if isinstance(branch, BranchSum):
                branch = branch.total()
            if not isinstance(norm, BranchLayerNorm):       # a norm this part's kernel does not know
                residual, _ = norm.add_branch(residual, branch, keep=residual is embedded)
                branch = norm = None
        else:
            residual = fp32_stream(x, residual)
        conv = None
        if following is not None and ctx.decode_only and isinstance(following[0], CausalInputConv):
            conv = (following[0].weight_t, following[1].input_state)
        out, prepared = ops.branch_depth_average(
            residual, branch, (norm.weight, norm.bias, norm.eps) if norm is not None else None, embedded, history,
            self.index, self.weights, self.dtype, ctx, conv)
        return StreamCopy.of(out if self.dtype == torch.float32 else None, prepared), out


register_input_part("causal_input_conv", CausalInputConv, replace=True)
register_stream_part("depth_average", DepthAverage, replace=True)
