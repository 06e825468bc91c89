"""Several residual streams beside one another, and the shift of a row towards the row of the token before.

``hyper_connection``: with X_1 .. X_s the streams, a sublayer f reads ``u = sum_s a[s] X_s`` (through its norm) and its
output y goes back as ``X_t <- sum_s M[s, t] X_s + b[t] y``, all streams at once from the old ones.  The coefficients are
a sublayer's own.  :class:`ResidualStreams` is what such blocks pass on in place of the single residual stream: it keeps
the last sublayer's output beside the streams it still has to enter, so that the update, the next sublayer's weighted
sum, its norm, the token shift and the cast are one kernel.

``token_shift``: ``h_t + (h_(t-1) - h_t) * mu`` on normed rows, zeros in front of a request's first token.  The last row
(before its shift) belongs to the request (:class:`~hfee_b200.cache.FixedState`), so a prompt may be cut anywhere.
"""
from __future__ import annotations

from typing import Any, Dict, Optional

import torch

from ..cache.needs import FixedState
from ..config.spec import PartSpec
from ..kernels import ops
from ..weights.loader import TensorNeed
from .base import Part, register_part


class HyperConnection(Part):
    """spec: ``streams``.  Tensors ``in`` [streams] (a), ``out`` [streams] (b), ``mix`` [streams, streams] (M, indexed
    [from, to]), all float32 on the device."""
    category = "streams"
    graph_safe = True

    @staticmethod
    def tensor_needs(spec: PartSpec) -> Dict[str, TensorNeed]:
        s = spec.streams
        return {"in": TensorNeed((s,), role="vector"), "out": TensorNeed((s,), role="vector"), "mix": TensorNeed((s, s), role="vector")}

    def __init__(self, spec, tensors, rt):
        super().__init__(spec, tensors, rt)
        self.in_weight, self.out_weight, self.mix = tensors["in"], tensors["out"], tensors["mix"]


class TokenShift(Part):
    """spec: ``width``.  Tensor ``weight`` [width] (float32 on the device).  Runs inside the kernel of
    :meth:`ResidualStreams.read`."""
    category = "shift"
    graph_safe = True

    @staticmethod
    def tensor_needs(spec: PartSpec) -> Dict[str, TensorNeed]:
        return {"weight": TensorNeed((spec.width,), role="vector")}

    def __init__(self, spec, tensors, rt):
        super().__init__(spec, tensors, rt)
        self.width, self.weight = int(spec.width), tensors["weight"]

    def cache_need(self) -> FixedState:
        return FixedState((self.width,), "float32")


class ResidualStreams:
    """``count`` streams for a step's tokens, all equal to ``start`` [n, width] (float32) at first."""

    def __init__(self, rt, start: torch.Tensor, count: int):
        self.rt, self.count = rt, count
        self.n, self.width = start.shape
        self.x = start                    # [n, width] while the streams are equal, then [n, count, width]
        self.pending = None               # (y, the connection it goes through): a sublayer's output not yet in the streams
        self._turn = 0

    def _update(self):
        if self.pending is None:
            return None
        y, connection = self.pending
        return y, connection.mix, connection.out_weight

    def read(self, connection: HyperConnection, norm, out: torch.Tensor, step: Any, shift: Optional[TokenShift] = None,
             shift_state: Optional[torch.Tensor] = None, writes_state: bool = True) -> None:
        """The next sublayer's input into ``out``: the pending output enters the streams, then the connection's weighted
        sum, the norm, the shift."""
        update = self._update()
        x_out = None
        if update is not None:            # two buffers in turn: the kernel reads neighbouring tokens' old streams
            x_out = self.rt.scratch(f"residual_streams{self._turn}", (self.rt.max_tokens, self.count, self.width), torch.float32)[:self.n]
            self._turn ^= 1
        before = ops.tag("norm")
        weight, eps, groups = norm.group_params()
        ops.stream_step(self.x, weight, eps, groups, out, connection.in_weight, update, x_out,
                        (shift.weight, shift_state, writes_state) if shift is not None else None, step)
        ops.tag(before)
        if update is not None:
            self.x, self.pending = x_out, None

    def leave(self, connection: HyperConnection, y: torch.Tensor) -> None:
        """A sublayer's output ``y`` [n, width] (float32; must stay until the next read)."""
        if self.pending is not None:
            raise ValueError("the streams take a sublayer's output after each read")
        self.pending = (y, connection)

    def collapse(self, norm, out: torch.Tensor, rows: Optional[torch.Tensor] = None) -> None:
        """The norm of the streams' sum (of the chosen tokens) into ``out``."""
        before = ops.tag("norm")
        weight, eps, groups = norm.group_params()
        ops.stream_step(self.x, weight, eps, groups, out, None, self._update(), None, rows=rows)
        ops.tag(before)


register_part("streams", "hyper_connection", HyperConnection)
register_part("shift", "token_shift", TokenShift)
