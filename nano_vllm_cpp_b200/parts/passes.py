"""Layers that run several times: what stands before each pass over them.

A model's ``order`` may name a layer in several calls (each with a cache entry of its own), so a stretch of layers that is run
t times in a row with the same weights is t runs of calls.  A call that opens a pass may carry the pass's number
(``LayerCall.pass_index``); the model then hands its residual stream through its *pass input* before that call.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import Part, RowMix, BranchSum, StreamRows, NormedBranch, TensorSpec
from .linear import linear
from .registry import register_part


class RecallInput(Part):
    """``x <- A x + B x0 + s_t``: the stream projected, the embedding rows ``x0`` recalled through a projection of their own,
    and a learned vector for pass t.  Tensors: ``in`` [width, 2 width] = [A | B], ``step`` [passes, width].

    ``B x0`` is the same for every pass: it is made once per step (``recall``).  A pass is then two launches: the stream takes
    in what is pending and its rows are written for the product, and the product with ``A`` makes the new stream with ``s_t``
    as its bias; ``B x0`` goes on as the pending branch, which the next norm adds."""

    def __init__(self, size: int, passes: int, in_name: str = "in", step_name: str = "step"):
        if passes < 1:
            raise ValueError("a stretch of layers runs at least once")
        self.size, self.passes, self.in_name, self.step_name = int(size), int(passes), in_name, step_name

    def tensor_specs(self, available=None):
        return {self.in_name: TensorSpec((self.size, 2 * self.size)),
                self.step_name: TensorSpec((self.passes, self.size), kind="vector")}

    def load(self, fetch, ctx):
        self.ctx = ctx
        w = fetch(self.in_name)
        self.w_stream, self.w_recall = w[:, :self.size].contiguous(), w[:, self.size:].contiguous()
        self.steps = fetch(self.step_name).float().contiguous()

    def _rows(self, x, pending):
        """The stream with what is pending taken in (in place), and its rows for a product."""
        branch = mix = None
        if isinstance(pending, NormedBranch):
            pending.add_to(x)
        elif isinstance(pending, BranchSum):
            branch = pending.sum()
        elif isinstance(pending, RowMix):
            if pending.gate_logit is None and pending.index.shape[1] <= ops.STREAM_MAX_MIX:
                mix = pending.as_tuple()
            else:
                branch = pending.sum()
        elif not isinstance(pending, StreamRows):
            branch = pending
        rows = x if self.ctx.act_dtype == torch.float32 else torch.empty(x.shape, dtype=self.ctx.act_dtype, device=x.device)
        if branch is not None or mix is not None or rows is not x:
            ops.stream_mix_norm(x, 1, branch=branch, mix=mix, out=None if rows is x else rows)
        return rows

    def recall(self, x0):
        """``B x0`` for the embedding rows ``x0`` (float32)."""
        return linear(self.ctx, self._rows(x0, None), self.w_recall, torch.float32)

    def forward(self, x, pending, recalled, t: int):
        """Returns the stream that pass t starts from and what is pending on it."""
        return linear(self.ctx, self._rows(x, pending), self.w_stream, torch.float32, bias=self.steps[t]), recalled


register_part("pass_input", "recall", RecallInput)
