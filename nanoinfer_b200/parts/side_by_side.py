"""Two mixers side by side: both read the same normed input and add their results to the residual stream, each with
the factor it was given (``out_scale`` of the mixer's own parameters). What the pair keeps per request is the union of
what its halves keep: the pages of the half that caches per position (at most one may), and one flat 32-bit state
whose first part belongs to the left half and the rest to the right one.

Two halves of the form product -> mix -> product (``ProjectedMixer``) share ONE input product, and what lies between the
products runs side by side on two streams where the kernel library has a second one.
"""
from __future__ import annotations

from contextlib import nullcontext
from dataclasses import replace
from typing import Dict, Optional

import torch

from ..registry import get_part, register_part
from .base import CacheNeed, LayerCache, Mixer, ProjectedMixer, Runtime, StateNeed, StepContext, as_tensor
from .spec import PartSpec


class SideBySide(Mixer):
    """params: ``left``, ``right`` (the halves' ``PartSpec``). tensors: the halves' tensors with the roles
    ``left.<role>`` and ``right.<role>``."""

    @staticmethod
    def spec(left: PartSpec, right: PartSpec) -> PartSpec:
        tensors = {f"left.{r}": ts for r, ts in left.tensors.items()}
        tensors.update({f"right.{r}": ts for r, ts in right.tensors.items()})
        return PartSpec("side_by_side", {"left": left, "right": right}, tensors)

    def __init__(self, spec: PartSpec, tensors: Dict[str, torch.Tensor], rt: Runtime):
        super().__init__(spec, tensors, rt)
        self.halves = []
        self.joint = all(issubclass(get_part(spec.params[side].kind), ProjectedMixer) for side in ("left", "right"))
        for side in ("left", "right"):
            sub: PartSpec = spec.params[side]
            if self.joint:
                sub = replace(sub, params=dict(sub.params, joint_input=True))
            mine = {r[len(side) + 1:]: t for r, t in tensors.items() if r.startswith(side + ".")}
            self.halves.append(get_part(sub.kind)(sub, mine, rt))
        if self.joint:
            left, right = self.halves
            # the right half's columns start on a multiple of four, so that its kernels may move 16 bytes at a time
            self.right_at = -(-left.in_width // 4) * 4
            fill = torch.zeros((self.right_at - left.in_width, left.in_rows.shape[1]), dtype=left.in_rows.dtype)
            self.w_in = rt.matrix(torch.cat([left.in_rows, fill, right.in_rows], dim=0))
            self.b_in = None
            if left.in_bias is not None or right.in_bias is not None:
                b = torch.zeros(self.right_at + right.in_width, dtype=torch.float32)
                for half, at in ((left, 0), (right, self.right_at)):
                    if half.in_bias is not None:
                        b[at:at + half.in_width] = half.in_bias
                self.b_in = rt.vector32(b)
            left.in_rows = right.in_rows = None
            prepare = getattr(rt.ops, "prepare_beside", None)
            if prepare is not None:
                prepare()
        needs = [m.cache_need() for m in self.halves]
        if sum(n is not None for n in needs) > 1:
            raise ValueError("at most one half of a pair may cache per position")
        self._offsets = []
        off = 0
        for m in self.halves:
            st = m.state_need()
            if st is not None and (st.dtype != torch.float32 or len(st.shape) != 1):
                raise ValueError("the halves of a pair keep their state as one row of 32-bit floats")
            n = 0 if st is None else int(st.shape[0])
            self._offsets.append((off, n))
            off += n
        self._state_size = off

    @property
    def graph_safe(self) -> bool:
        return all(getattr(m, "graph_safe", False) for m in self.halves)

    def cache_need(self) -> Optional[CacheNeed]:
        for m in self.halves:
            need = m.cache_need()
            if need is not None:
                return need
        return None

    def state_need(self) -> Optional[StateNeed]:
        return StateNeed((self._state_size,), torch.float32) if self._state_size else None

    def bind_positions(self, positions) -> None:
        for m in self.halves:
            m.bind_positions(positions)

    def forward(self, h: torch.Tensor, residual32: torch.Tensor, ctx: StepContext, cache: LayerCache) -> None:
        h = as_tensor(h)
        # each half's state: rows of the slots, a slice of their columns
        caches = [replace(cache, state=cache.state[:, off:off + n] if n else None, writes=cache.writes and m.cache_need() is not None)
                  for m, (off, n) in zip(self.halves, self._offsets)]
        if not self.joint:
            for m, c in zip(self.halves, caches):
                m.forward(h, residual32, ctx, c)
            return
        left, right = self.halves
        p32 = torch.empty((h.shape[0], self.right_at + right.in_width), dtype=torch.float32, device=h.device)
        self.ops.linear(h, self.w_in, self.b_in, p32, "f32")
        beside = getattr(self.ops, "beside", None)
        with (beside() if beside is not None else nullcontext()) as second:
            b = right.mix(p32[:, self.right_at:], ctx, caches[1])
        a = left.mix(p32[:, :left.in_width], ctx, caches[0])
        self.ops.linear(a, left.w_o, left.b_o, residual32, "add")
        if second is not None:
            second.join()       # (both halves add into the stream: one after the other)
        self.ops.linear(b, right.w_o, right.b_o, residual32, "add")


register_part("side_by_side", SideBySide)
