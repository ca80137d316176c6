"""A feed-forward of routed experts: every token runs `top` of `experts` small gated feed-forwards and adds their outputs
up with weights from a router.

    z = W_router h   (a float32 product in every mode)          s = sigmoid(z)   ("score": "softmax" for a softmax over z;
                                                                                 "chosen": z itself chooses, s = softmax over the chosen)
    experts e * per .. (e + 1) * per - 1 form group e (`groups` of them, per = experts / groups); group score = top-2 sum of its s
    (its one s when per is 1); the `keep` groups of highest score stay eligible, the rest are barred (groups <= 1: none barred)
    the `top` eligible experts of largest s are chosen; weight_k = s_k / (sum of the chosen s + 1e-20) * scale
    y = sum_k weight_k * down_k(silu(gate_k h) * (up_k h))

and, all optional:
    correction   a float32 number per expert that is added to the scores that choose (groups and experts), not to the weights
    renormalize  False: weight_k = s_k * scale
    identity     the last so many outputs of the router stand for experts without tensors whose output is h itself
    bias         a float32 number per router output, added to z
    unit         the gated unit's constants {alpha, shift, limit} (`ops.GatedUnit`; default silu(gate) * up)
    shared       {"intermediate": f, "unit": ...}: one more gated feed-forward that every token runs, added with weight 1

Several routes, the same numbers up to rounding.  In bfloat16 the (token, choice) pairs are laid out by expert on the device
(`ops.moe_plan`; up to 128 tokens the choice and the plan are one launch, `ops.moe_route_plan`), and where the experts' width is a multiple
of 64 every step, short or long, brings the pairs' rows side by side (`ops.moe_gather`) and runs all experts as tcgen05 products
whose tiles are found from the plan's counts on the device (`ops.moe_grouped_tc`): each chosen expert's weights are read once per 32 to
256 rows and nothing comes back to the host.  Other widths in multiples of 8: steps of up to `GROUPED_MAX` tokens, and those that a CUDA graph
captures, run the m16n8k16 kernel `ops.moe_grouped` in the same manner; a longer step reads the counts on the host, every expert then owns the
same number of rows (`ops.moe_pad_rows`) and all experts run as one batched library product for gate/up and one for down.  float32 steps of a
few tokens (`ROWS_MAX` or fewer, or captured) run `ops.moe_expert_rows`: the chosen experts' rows are streamed per (token, choice); longer ones
read the counts on the host and run the framework's products per expert.  `ops.moe_combine` adds the results per token in the order of the
choice (float32 sums, one rounding).

params: hidden, experts (those with tensors), top, intermediate (an expert's width), groups, keep, scale, score, correction (bool),
renormalize (default True), identity (default 0), bias (bool), unit, shared, names (optional: "router", "correction", "bias" - default the
router's + ".b"; the experts' tensors are e<k>.gate,
e<k>.up, e<k>.down, the shared one's shared.gate, shared.up, shared.down).

An arrangement that runs its sublayers side by side may take the part in two: `join_stream(h, ctx, resid)` adds the routed experts'
sum to the float32 stream (no rounding in between), and the rest - the shared expert - offers its projections like any
feed-forward (`packs_projections`; `input_weight` None when there is no shared expert), or runs alone (`forward_rest`).
An arrangement that norms what the part returns may take it unsummed: `forward_unsummed(h, ctx)` runs the shared expert on a second stream
beside the routed ones and returns an `ops.RoutedSum` (or a plain pair of branches), which the norm's kernel adds up in float32.
"""

from __future__ import annotations

import torch

from .. import ops
from ..config.recipe import PartSpec
from .base import Part, WeightSpec
from .context import StepContext
from .registry import build_part, register_part

USE_TCGEN05 = True # False: parts built from now on take the m16n8k16 kernel and the library's batched products (measurements)
ROWS_MAX = 16      # steps of up to this many tokens stream the chosen experts' rows (float32, or widths that are no multiple of 8)
# bfloat16 steps of up to this many tokens run every expert over its tokens in one tensor-core kernel that reads the counts on the
# device (None: every step).  Longer steps read the counts on the host and run all experts as ONE batched library product over a
# layout in which every expert owns the same number of rows (the largest count, rounded up to 64): a product per expert would change
# shape with every step's counts, and the library's choice of a kernel for a shape it has not seen costs the host about a
# millisecond a call (a prompt of 2,048 tokens over 32 experts spent 75 ms there); the batched shapes are few and come again.
GROUPED_MAX: int | None = 512
PAD_WASTE_MAX = 4.0  # the batched layout is used while it holds at most this many times the step's rows (else: the grouped kernel)


@register_part("feed_forward", "routed_experts")
class RoutedExperts(Part):
    def __init__(self, spec, dtype, device) -> None:
        super().__init__(spec, dtype, device)
        p = spec.params
        self.hidden, self.experts, self.top, self.inter = int(p["hidden"]), int(p["experts"]), int(p["top"]), int(p["intermediate"])
        self.groups, self.keep = int(p.get("groups") or 1), int(p.get("keep") or 1)
        self.scale = float(p.get("scale") if p.get("scale") is not None else 1.0)
        scores = {"sigmoid": ops.ROUTE_SIGMOID, "softmax": ops.ROUTE_SOFTMAX, "chosen": ops.ROUTE_CHOSEN}
        if p.get("score", "sigmoid") not in scores:
            raise ValueError(f"routed_experts: unknown score {p.get('score')!r} (known: {', '.join(scores)})")
        self.softmax = scores[p.get("score", "sigmoid")]
        self.unit = ops.GatedUnit(**dict(p.get("unit") or {}))
        self.identity = int(p.get("identity") or 0)
        self.choices = self.experts + self.identity  # the router's outputs
        self.renormalize = bool(p.get("renormalize", True))
        if self.top > self.choices or (self.groups > 1 and (self.choices % self.groups or not 1 <= self.keep <= self.groups
                                                             or self.keep * (self.choices // self.groups) < self.top)):
            raise ValueError(f"routed_experts: {self.top} of {self.choices} experts in {self.groups} groups of which {self.keep} stay")
        names = dict(p.get("names") or {})
        self.n_router, self.n_correction = names.get("router", "router"), names.get("correction", "correction")
        self.n_bias = names.get("bias", self.n_router + ".b")
        self.has_correction, self.has_bias = bool(p.get("correction")), bool(p.get("bias"))
        self.router_bias: torch.Tensor | None = None
        self.correction: torch.Tensor | None = None
        shared = p.get("shared")
        self.shared = None if shared is None else build_part("feed_forward", PartSpec("swiglu", {
            "hidden": self.hidden, "intermediate": int(shared["intermediate"]), "unit": shared.get("unit"),
            "names": {k: f"shared.{k}" for k in ("gate", "up", "down")}}), dtype, device)
        self.tcgen05 = USE_TCGEN05 and dtype == torch.bfloat16 and self.hidden % 8 == 0 and self.inter % ops.GATE_BLOCK == 0
        self.w_router = self.w_gate = self.w_up = self.w_down = self.w_gate_up = None
        self.gate_block = 0

    def weight_specs(self) -> dict[str, WeightSpec]:
        specs = {self.n_router: WeightSpec((self.choices, self.hidden), rule="float32", init="normal", std=0.1)}
        if self.has_correction:
            specs[self.n_correction] = WeightSpec((self.choices,), rule="float32", init="normal", std=0.01)
        if self.has_bias:
            specs[self.n_bias] = WeightSpec((self.choices,), rule="float32", init="normal", std=0.1)
        if self.shared is not None:
            specs.update(self.shared.weight_specs())
        for e in range(self.experts):
            specs[f"e{e}.gate"] = WeightSpec((self.inter, self.hidden))
            specs[f"e{e}.up"] = WeightSpec((self.inter, self.hidden))
            specs[f"e{e}.down"] = WeightSpec((self.hidden, self.inter))
        return specs

    def bind(self, tensors) -> None:
        E = self.experts
        self.w_router = tensors[self.n_router].contiguous()
        if self.has_correction:
            self.correction = tensors[self.n_correction].contiguous()
        if self.has_bias:
            self.router_bias = tensors[self.n_bias].contiguous()
        if self.shared is not None:
            self.shared.bind({n: tensors[n] for n in self.shared.weight_specs()})
        self.w_gate = torch.stack([tensors[f"e{e}.gate"] for e in range(E)]).contiguous()   # [E, ff, width]
        self.w_up = torch.stack([tensors[f"e{e}.up"] for e in range(E)]).contiguous()
        self.w_down = torch.stack([tensors[f"e{e}.down"] for e in range(E)]).contiguous()   # [E, width, ff]
        # per expert the packed projection that the gated product takes (see parts/feed_forward.py)
        self.gate_block = ops.GATE_BLOCK if self.inter % ops.GATE_BLOCK == 0 else 0
        if self.gate_block:
            b = self.gate_block
            packed = torch.stack([self.w_gate.view(E, self.inter // b, b, self.hidden), self.w_up.view(E, self.inter // b, b, self.hidden)], dim=2)
            self.w_gate_up = packed.reshape(E, 2 * self.inter, self.hidden).contiguous()
        else:
            self.w_gate_up = torch.cat([self.w_gate, self.w_up], dim=1).contiguous()
        if self.tcgen05:  # every step reads the packed form alone
            self.w_gate = self.w_up = None

    def _logits(self, x, ctx: StepContext) -> torch.Tensor:
        return ops.router_logits(x, self.w_router, ctx.buffer("router_logits", self.choices, torch.float32),
                                 scratch=lambda rows, cols: ctx.buffer("router_in", cols, torch.float32, rows=rows), bias=self.router_bias)

    def route(self, x, ctx: StepContext) -> tuple[torch.Tensor, torch.Tensor]:
        """(chosen experts int32 [N, top], their weights float32 [N, top])"""
        ids = ctx.buffer("expert_ids", self.top, torch.int32)
        weights = ctx.buffer("expert_weights", self.top, torch.float32)
        ops.moe_route(self._logits(x, ctx), self.groups, self.keep, self.top, self.scale, ids, weights, self.softmax, self.correction, self.renormalize)
        return ids, weights

    # ---- the three ways to run the part ------------------------------------------------------------------------------------
    def forward(self, x, ctx: StepContext):
        out = ctx.buffer("branch", self.hidden)
        if self.shared is None:
            return self._routed(x, ctx, out, None)
        y = ops.cast_f32(self.shared.forward(x, ctx, out_name="branch_shared"), ctx.buffer("experts_sum", self.hidden, torch.float32))
        self._routed(x, ctx, out, y)
        return out.copy_(y)

    def join_stream(self, x, ctx: StepContext, resid: torch.Tensor) -> None:
        """The routed experts' sum, added to the float32 stream; everything but the shared expert."""
        self._routed(x, ctx, ctx.buffer("experts_branch", self.hidden), resid)

    def forward_rest(self, x, ctx: StepContext):
        """What `join_stream` leaves: the shared expert's output, or None without one."""
        return None if self.shared is None else self.shared.forward(x, ctx)

    @property
    def gives_unsummed(self) -> bool:
        """Whether `forward_unsummed` may be asked for: every choice has a row of its own (no expert returns its input)."""
        return self.identity == 0

    def forward_unsummed(self, x, ctx: StepContext):
        """The part's output as an `ops.RoutedSum`, or as the branches (routed, shared) where the routed sum is made on the way."""
        rest = None
        side = ops.side_lane(x.device, "shared_expert") if self.shared is not None else None
        if side is not None:
            side.fork()
            with side.stream():
                rest = self.shared.forward(x, ctx, out_name="branch_shared")
        elif self.shared is not None:
            rest = self.shared.forward(x, ctx, out_name="branch_shared")
        y = self._routed(x, ctx, ctx.buffer("branch", self.hidden), None, summed=False)
        if side is not None:
            side.join()
        if isinstance(y, ops.RoutedSum):
            y.rest = rest
            return y
        return (y, rest) if rest is not None else y

    # ---- optional: the shared expert's products inside larger ones of an arrangement (see `GQAAttention.packs_projections`) ------
    packs_projections = True

    @property
    def input_weight(self) -> torch.Tensor | None:
        return None if self.shared is None else self.shared.input_weight

    @property
    def output_weight(self) -> torch.Tensor | None:
        return None if self.shared is None else self.shared.output_weight

    def adopt(self, w_in: torch.Tensor, w_out: torch.Tensor) -> None:
        self.shared.adopt(w_in, w_out)

    def forward_projected(self, u: torch.Tensor, ctx: StepContext, act: torch.Tensor) -> None:
        self.shared.forward_projected(u, ctx, act)

    # ---- the routed experts ---------------------------------------------------------------------------------------------------
    def _choose_and_plan(self, x, ctx: StepContext, offsets, row_of, pair_of=None) -> torch.Tensor:
        """The router, the choice and the pairs' layout by expert; returns the weights float32 [N, top]."""
        if ops.route_plan_ok(x.shape[0], self.choices):
            ids, weights = ctx.buffer("expert_ids", self.top, torch.int32), ctx.buffer("expert_weights", self.top, torch.float32)
            ops.moe_route_plan(self._logits(x, ctx), self.groups, self.keep, self.top, self.scale, ids, weights, self.softmax, self.correction,
                               self.renormalize, self.experts, offsets, row_of, ctx.buffer("expert_pairs", self.top, torch.int32))
            return weights
        ids, weights = self.route(x, ctx)
        ops.moe_plan(ids, self.experts, offsets, row_of, pair_of)
        return weights

    def _finish(self, ys, row_of, weights, out, x, resid, summed: bool):
        return ops.moe_combine(ys, row_of, weights, out, self.top, x=x, resid=resid) if summed else ops.RoutedSum(ys, row_of, weights)

    def _grouped(self, x, ids, weights, offsets, row_of, out, ctx: StepContext, resid, summed: bool = True):
        n = x.shape[0]
        pair_of = ctx.buffer("expert_pairs", self.top, torch.int32)
        if ids is None:
            weights = self._choose_and_plan(x, ctx, offsets, row_of, pair_of)
        else:
            ops.moe_plan(ids, self.experts, offsets, row_of, pair_of)
        act = ctx.buffer("expert_act", self.inter, rows=n * self.top)
        ys = ctx.buffer("expert_out", self.hidden, rows=n * self.top)
        ops.moe_grouped(x, pair_of, offsets, self.w_gate, self.w_up, self.w_down, act, ys, self.top, self.unit)
        return self._finish(ys, row_of, weights, out, x, resid, summed)

    def _routed(self, x, ctx: StepContext, out: torch.Tensor, resid: torch.Tensor | None, summed: bool = True):
        """The routed experts' sum in `out`, or added to the float32 `resid` when that is given; returns where it went.  `summed` False: the
        sum is left to the caller (`ops.RoutedSum`) where the route taken leaves a row per choice."""
        n = x.shape[0]
        captured = bool(ctx.extras.get("graph")) or torch.cuda.is_current_stream_capturing()
        offsets = ctx.buffer("expert_offsets", 1, torch.int32, rows=self.experts + 1).view(-1)
        row_of = ctx.buffer("expert_rows", self.top, torch.int32)
        if self.tcgen05:
            weights = self._choose_and_plan(x, ctx, offsets, row_of)
            xs = ops.moe_gather(x, row_of, ctx.buffer("expert_in", self.hidden, rows=n * self.top), self.top)
            ys = ctx.buffer("expert_out", self.hidden, rows=n * self.top)
            ops.moe_grouped_tc(xs, offsets, self.w_gate_up, self.w_down, ctx.buffer("expert_act", self.inter, rows=n * self.top), ys, self.unit)
            return self._finish(ys, row_of, weights, out, x, resid, summed)
        grouped_ok = ops.moe_grouped_ok(x, self.hidden, self.inter)
        if grouped_ok and (GROUPED_MAX is None or n <= GROUPED_MAX or captured):
            return self._grouped(x, None, None, offsets, row_of, out, ctx, resid, summed)
        ids, weights = self.route(x, ctx)
        if n <= ROWS_MAX or captured:
            act = ctx.buffer("expert_act", self.inter, rows=n * self.top)
            ops.moe_expert_rows(x, ids, weights, self.w_gate, self.w_up, self.w_down, act, out, self.unit)
            return out if resid is None else ops.residual_add(resid, out)
        ops.moe_plan(ids, self.experts, offsets, row_of)
        bounds = offsets.tolist()  # the one host round trip of the step's experts
        if grouped_ok:
            # bfloat16: every expert owns `cap` rows and all run as one batched product each for gate/up and down
            cap = max(64, -(-max(b - a for a, b in zip(bounds, bounds[1:])) // 64) * 64)
            rows = self.experts * cap
            if rows > PAD_WASTE_MAX * n * self.top:  # the tokens crowd a few experts: no layout of equal shares for them
                return self._grouped(x, ids, weights, offsets, row_of, out, ctx, resid, summed)
            ops.moe_pad_rows(ids, offsets, row_of, cap)
            xs = ops.moe_gather(x, row_of, ctx.buffer("expert_in", self.hidden, rows=rows), self.top)
            gu = ctx.buffer("expert_gate_up", 2 * self.inter, rows=rows)
            torch.bmm(xs.view(self.experts, cap, self.hidden), self.w_gate_up.transpose(1, 2), out=gu.view(self.experts, cap, 2 * self.inter))
            act = ops.swiglu(gu, ctx.buffer("expert_act", self.inter, rows=rows), self.gate_block, self.unit)
            ys = ctx.buffer("expert_out", self.hidden, rows=rows)
            torch.bmm(act.view(self.experts, cap, self.inter), self.w_down.transpose(1, 2), out=ys.view(self.experts, cap, self.hidden))
            return self._finish(ys, row_of, weights, out, x, resid, summed)
        xs = ops.moe_gather(x, row_of, ctx.buffer("expert_in", self.hidden, rows=n * self.top), self.top)
        ys = ctx.buffer("expert_out", self.hidden, rows=n * self.top)
        act = ctx.buffer("expert_act", self.inter, rows=n * self.top)
        scratch = ctx.buffer("expert_gate_up", 2 * self.inter, rows=n * self.top)
        for e in range(self.experts):
            lo, hi = bounds[e], bounds[e + 1]
            if hi > lo:
                ops.gated_linear(xs[lo:hi], self.w_gate_up[e], act[lo:hi], scratch[lo:hi], self.gate_block, self.unit)
                ops.linear(act[lo:hi], self.w_down[e], ys[lo:hi])
        return self._finish(ys, row_of, weights, out, x, resid, summed)
