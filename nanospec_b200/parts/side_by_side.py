"""A mixer made of two mixers that read the same input: y = a * left(x) + b * right(x), with constants a and b.

Both run between ONE packed input product [left's columns | right's] of x and ONE output product of the concatenated results by
[W_left | W_right], whose float32 accumulator holds the weighted sum before it is rounded once; the constants ride in the sublayers' own last
step (`out_scale`: an attention kernel's epilogue, a read-out norm's gain), before that step rounds.  What lies between the two products runs
on two streams side by side (`ops.side_lane`).  The mixers keep views of the packed matrices in place of their own, so weights are held once
and replaced in place.

A mixer qualifies when it offers its projections (`packs_projections`, see `GQAAttention`) and takes `out_scale`.  Paged keys and values
and the state slot of the lane go to the one mixer that asks for them: at most one of the two may ask for each.
"""

from __future__ import annotations

import torch

from .. import ops
from ..config.recipe import PartSpec
from .base import CacheNeed, Part, StateNeed, WeightSpec
from .context import LaneView, StepContext
from .registry import build_part, register_part


def _pad_columns(w: torch.Tensor) -> torch.Tensor:
    """Zero columns up to a multiple of 8: the next range of a packed row then starts on 16 bytes in bfloat16."""
    extra = -w.shape[1] % 8
    return torch.cat([w, torch.zeros((w.shape[0], extra), dtype=w.dtype, device=w.device)], dim=1) if extra else w


@register_part("mixer", "side_by_side")
class SideBySide(Part):
    """params: hidden, left and right (PartSpecs of mixers), left_scale, right_scale (default 1), names (optional: keys "left", "right", the
    prefixes of the two mixers' tensors; default "left." and "right.")."""

    SIDES = ("left", "right")

    def __init__(self, spec, dtype, device) -> None:
        super().__init__(spec, dtype, device)
        p = spec.params
        self.hidden = int(p["hidden"])
        names = dict(p.get("names") or {})
        self.prefixes = {s: names.get(s, s + ".") for s in self.SIDES}
        for s in self.SIDES:
            child = p[s]
            part = build_part("mixer", PartSpec(child.kind, {**child.params, "out_scale": float(p.get(s + "_scale", 1.0))}), dtype, device)
            if not getattr(part, "packs_projections", False):
                raise ValueError(f"side_by_side: the mixer {child.kind!r} does not offer its projections")
            setattr(self, s, part)
        if all(m.cache_need() is not None for m in self.mixers) or all(m.state_need() is not None for m in self.mixers):
            raise ValueError("side_by_side: only one of the two mixers can hold pages, and only one a state")
        self.w_in: torch.Tensor | None = None   # [left's columns + right's, hidden]
        self.w_out: torch.Tensor | None = None  # [hidden, left's result + right's]

    @property
    def mixers(self) -> tuple[Part, Part]:
        return self.left, self.right

    def weight_specs(self) -> dict[str, WeightSpec]:
        return {self.prefixes[s] + name: spec for s in self.SIDES for name, spec in getattr(self, s).weight_specs().items()}

    def bind(self, tensors) -> None:
        for s in self.SIDES:
            part = getattr(self, s)
            part.bind({name: tensors[self.prefixes[s] + name] for name in part.weight_specs()})
        w_in, w_out = [m.input_weight for m in self.mixers], [m.output_weight for m in self.mixers]
        self.w_in = torch.cat(w_in, dim=0).contiguous()  # (a mixer's packed projection has rows in multiples of 8)
        self.w_out = torch.cat([_pad_columns(w) for w in w_out], dim=1).contiguous()
        self.ranges = []
        at_in = at_out = 0
        for m, wi, wo in zip(self.mixers, w_in, w_out):
            ri, ro = slice(at_in, at_in + wi.shape[0]), slice(at_out, at_out + wo.shape[1])
            m.adopt(self.w_in[ri], self.w_out[:, ro])
            self.ranges.append((ri, ro))
            at_in, at_out = ri.stop, at_out + -(-wo.shape[1] // 8) * 8

    def cache_need(self) -> CacheNeed | None:
        return next((need for m in self.mixers if (need := m.cache_need()) is not None), None)

    def state_need(self) -> StateNeed | None:
        return next((need for m in self.mixers if (need := m.state_need()) is not None), None)

    def feeds_norm_sink(self, n_tokens: int) -> bool:
        return ops.norm_fusion_ok(n_tokens, self.dtype, self.w_out)

    def forward(self, x, ctx: StepContext, lane: LaneView, writes: bool = True, sink=None):
        proj = ops.linear(x, self.w_in, ctx.buffer("sbs_in", self.w_in.shape[0]))
        (li, lo), (ri, ro) = self.ranges
        # zeroed once: the columns between the two results (none when the first is a multiple of 8 wide) are never written
        mid = ctx.workspace.get(f"sbs_mid_{lo.stop}_{ro.start}_{ro.stop}", ctx.n_tokens, self.w_out.shape[1], self.dtype, zero=True)
        side = ops.side_lane(x.device, "mixer")
        if side is not None:
            side.fork()
            with side.stream():
                self.right.forward_projected(proj[:, ri], ctx, lane, writes, mid[:, ro])
        self.left.forward_projected(proj[:, li], ctx, lane, writes, mid[:, lo])
        if side is not None:
            side.join()
        else:
            self.right.forward_projected(proj[:, ri], ctx, lane, writes, mid[:, ro])
        return ops.linear(mid, self.w_out, ctx.buffer("branch", self.hidden), sink=sink)
