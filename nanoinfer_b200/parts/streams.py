"""Several residual streams around a sublayer: instead of one stream x a token has ``n`` of them, all equal to the embedding
output at the start. A sublayer reads a sum of them and gives its result back to all:

    u = sum_s in[s] x_s,    y = sublayer(norm(u)),    x_t <- sum_s mix[s, t] x_s + out[t] y      (all from the old streams)

and what follows the last sublayer reads their sum. All of it is 32-bit. Between two sublayers ONE kernel
(``ops.stream_mix``) takes the first one's result into the streams, forms what the second one reads and norms it, so the
streams are read and written once per sublayer. A sublayer therefore leaves its update pending on the stream
(``parts/base.py``: ``PENDING_STREAM_OP``); the next sublayer does it together with its own sum and norm, and whoever else
reads the stream next (another kind of block, the final norm) has the streams summed into it first.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..registry import register_part
from .base import PENDING_STREAM_OP, Norm, Part, Runtime, StepContext
from .spec import PartSpec, TensorSpec


class StreamMix(Part):
    """The factors of one sublayer. params: ``streams``. tensors: ``in [streams]``, ``out [streams]``,
    ``mix [streams (from), streams (to)]``."""

    graph_safe = True   # launches do not depend on which requests are in the batch

    @staticmethod
    def spec(prefix: str, streams: int) -> PartSpec:
        return PartSpec("stream_mix", {"streams": int(streams)}, {
            "in": TensorSpec(f"{prefix}.in", (streams,), "mix"), "out": TensorSpec(f"{prefix}.out", (streams,), "gain"),
            "mix": TensorSpec(f"{prefix}.mix", (streams, streams), "near_identity")})

    def __init__(self, spec: PartSpec, tensors: Dict[str, torch.Tensor], rt: Runtime):
        super().__init__(spec, tensors, rt)
        self.streams = int(spec.params["streams"])
        self.read, self.share, self.mix = (rt.vector32(tensors[n]) for n in ("in", "out", "mix"))


class StreamSet:
    """The streams of one step, and the update that the last sublayer left to do. ``y32`` is the zeroed buffer that a
    sublayer adds its result into."""

    def __init__(self, rt: Runtime, x32: torch.Tensor, streams: int):
        self.rt, self.x32, self.streams = rt, x32, streams
        self.current = x32                          # one tensor that all streams equal, until the first update
        self.buffer = torch.empty((x32.shape[0], streams, x32.shape[1]), dtype=torch.float32, device=x32.device)
        self.y32 = torch.zeros_like(x32)
        self.h = torch.empty(x32.shape, dtype=rt.dtype, device=x32.device)
        self.update: Optional[StreamMix] = None     # the sublayer whose result is in y32 and not yet in the streams

    @staticmethod
    def of(rt: Runtime, x32: torch.Tensor, ctx: StepContext, streams: int) -> "StreamSet":
        """The step's streams as the block before left them, or new ones that all equal ``x32``."""
        op = ctx.scratch.pop(PENDING_STREAM_OP, None)
        if isinstance(op, StreamSet) and op.x32 is x32 and op.streams == streams:
            return op
        if op is not None:
            op.run(x32, ctx)
        return StreamSet(rt, x32, streams)

    def enter(self, factors: StreamMix, norm: Norm) -> torch.Tensor:
        """What the sublayer with these factors reads: the pending update, the sum and the norm in one pass."""
        fold = norm.fold_into_projection(self.x32)
        if fold is None or fold.kind != "rms":
            raise ValueError("the norm of a sum of streams is an RMS norm with a gain")
        up = self.update
        if up is None:
            self.rt.ops.stream_mix(self.current, self.streams, in32=factors.read, gain32=fold.gain32, eps=fold.eps, h_out=self.h)
        else:
            self.rt.ops.stream_mix(self.current, self.streams, y32=self.y32, mix32=up.mix, out32=up.share, dst32=self.buffer,
                                   in32=factors.read, gain32=fold.gain32, eps=fold.eps, h_out=self.h, clear=True)
            self.current = self.buffer
        self.update = factors
        return self.h

    def run(self, x32: torch.Tensor, ctx: StepContext) -> None:
        """x32 becomes the sum of the streams, the pending update included."""
        up = self.update
        self.rt.ops.stream_mix(self.current, self.streams, y32=self.y32 if up is not None else None, mix32=up.mix if up is not None else None,
                               out32=up.share if up is not None else None, sum_out32=x32)


register_part("stream_mix", StreamMix)
