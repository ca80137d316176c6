"""Mixers whose memory is a matrix per head instead of a growing cache: retention (linear attention with a fixed decay
per head), the gated delta rule and the state space of Mamba-2.  All keep S [heads, head_dim, v_dim] in float32 in the request's state slot and walk
a step's tokens in order (csrc/recurrent.cu), so portions of a prompt, single decoded tokens and whole prompts give the
same numbers; under CUDA graphs they address the state through the device's `qo_indptr` and `state_slot`.

    retention   S_t = decay_h S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t;  q and k rotated by position, k times head_dim^-1/2;
                per head o / rms(o), all heads times silu(gate), output projection.
    delta       q, k, v pass a short causal convolution per channel and silu; q and k become unit vectors, q times
                head_dim^-1/2; beta = sigmoid(b h), g = exp(-exp(A_log) softplus(a h + dt_bias));
                S = g S;  u = beta (v - S^T k);  S = S + k u^T;  o = S^T q;  per head o / rms(o) times a gain shared by the
                heads, times silu(gate), output projection.  The last taps - 1 inputs of the convolution are state as well.
    mamba2      one projection [z | x | B | C | dt]; x, B and C pass a short causal convolution per channel (with a bias) and silu;
                a = softplus(dt + dt_bias) is the step size of a head and exp(-exp(A_log) a) its decay g;
                S_t = g S_(t-1) + B_t (a x_t)^T,  o_t = S_t^T C_t + D x_t, B and C shared by the heads of a group;
                (o silu(z)) normed in equal parts, each by its own root mean square, times a gain, output projection.
                Long portions of prompts run in chunks of 64 tokens (csrc/ssm_chunked.cu: products over the chunk's tokens, the state
                carried between chunks), the same sums in another order.

The projections are one packed product; the convolution, the rotation, the unit norms, the decay and the read-out's norm are
float32.
"""

from __future__ import annotations

import torch

from .. import ops
from .base import CacheNeed, Part, StateNeed, WeightSpec
from .context import LaneView, StepContext
from .registry import build_part, register_part


def _pad_rows(w: torch.Tensor, multiple: int = 8) -> torch.Tensor:
    """A packed projection whose row count is a multiple of 8: rows of its output are then 16-byte aligned in bfloat16."""
    extra = -w.shape[0] % multiple
    if extra:
        w = torch.cat([w, torch.zeros((extra, w.shape[1]), dtype=w.dtype, device=w.device)], dim=0)
    return w.contiguous()


@register_part("mixer", "retention")
class Retention(Part):
    """params: hidden, heads, head_dim, v_dim, decay (one per head), eps (of the read-out's norm), position (PartSpec of kind
    "rotary", or None), names (optional: keys "q", "k", "v", "g", "o")."""

    def __init__(self, spec, dtype, device) -> None:
        super().__init__(spec, dtype, device)
        p = spec.params
        self.hidden, self.heads = int(p["hidden"]), int(p["heads"])
        self.head_dim, self.v_dim = int(p["head_dim"]), int(p["v_dim"])
        self.eps = float(p["eps"])
        decay = [float(d) for d in p["decay"]]
        if len(decay) != self.heads:
            raise ValueError(f"retention: {len(decay)} decays for {self.heads} heads")
        self.decay_host = torch.tensor(decay, dtype=torch.float32)
        self._decay: torch.Tensor | None = None
        self.position = build_part("position", p["position"], dtype, device) if p.get("position") is not None else None
        names = dict(p.get("names") or {})
        self.names = {k: names.get(k, k + "_proj.weight") for k in ("q", "k", "v", "g", "o")}
        self.qk_size, self.v_size = self.heads * self.head_dim, self.heads * self.v_dim
        self.dp = ops.scan_padded_dim(self.head_dim)
        self.rec_cols = -(-(2 * self.heads * self.dp + self.v_size + self.heads) // 4) * 4  # q, k, v, k . q
        self.w_in: torch.Tensor | None = None
        self.w_o: torch.Tensor | None = None

    def weight_specs(self) -> dict[str, WeightSpec]:
        n = self.names
        return {n["q"]: WeightSpec((self.qk_size, self.hidden)), n["k"]: WeightSpec((self.qk_size, self.hidden)),
                n["v"]: WeightSpec((self.v_size, self.hidden)), n["g"]: WeightSpec((self.v_size, self.hidden)),
                n["o"]: WeightSpec((self.hidden, self.v_size))}

    def bind(self, tensors) -> None:
        n = self.names
        self.w_in = _pad_rows(torch.cat([tensors[n[k]] for k in ("q", "k", "v", "g")], dim=0))
        self.w_o = tensors[n["o"]].contiguous()

    def cache_need(self) -> CacheNeed | None:
        return None

    def state_need(self) -> StateNeed | None:
        return StateNeed((self.heads * self.head_dim * self.v_dim,), torch.float32)

    def forward(self, x, ctx: StepContext, lane: LaneView, writes: bool = True):
        if not writes:
            raise ValueError("a retention mixer owns its state: its lane cannot be shared")
        if self._decay is None:
            self._decay = self.decay_host.to(self.device)
        proj = ops.linear(x, self.w_in, ctx.buffer("rec_proj", self.w_in.shape[0]))
        rec = ctx.buffer("rec_in", self.rec_cols, torch.float32)
        pos = self.position
        ops.rotary_prepare(proj, ctx, pos.inv_freq if pos is not None and pos.dims else None, pos.magnitude if pos is not None else 1.0,
                           pos.interleaved if pos is not None else False, rec, self.heads, self.head_dim, self.v_dim,
                           1.0, self.head_dim ** -0.5)
        read = ops.linear_scan(rec, lane.state, ctx, ctx.buffer("rec_out", self.v_size, torch.float32), self.heads, self.heads,
                               self.head_dim, self.v_dim, decay=self._decay)
        gate = proj[:, 2 * self.qk_size + self.v_size: 2 * self.qk_size + 2 * self.v_size]
        y = ops.head_norm_gate(read, gate, None, self.eps, ctx.buffer("rec_y", self.v_size), ctx, self.heads, self.v_dim)
        return ops.linear(y, self.w_o, ctx.buffer("branch", self.hidden))


@register_part("mixer", "gated_delta")
class GatedDeltaRule(Part):
    """params: hidden, heads, kv_heads (q and k heads; head h reads q/k head h // (heads / kv_heads)), head_dim, v_dim, conv
    (taps of the short convolution), eps (of the read-out's norm), unit_eps (inside the root of the unit norms; default 1e-6),
    names (optional: keys "q", "k", "v", "g", "o", "a", "b", "q_conv", "k_conv", "v_conv", "A_log", "dt_bias", "norm")."""

    DEFAULT_NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "g": "g_proj.weight", "o": "o_proj.weight",
                     "a": "a_proj.weight", "b": "b_proj.weight", "q_conv": "q_conv.weight", "k_conv": "k_conv.weight",
                     "v_conv": "v_conv.weight", "A_log": "A_log", "dt_bias": "dt_bias", "norm": "o_norm.weight"}

    def __init__(self, spec, dtype, device) -> None:
        super().__init__(spec, dtype, device)
        p = spec.params
        self.hidden, self.heads, self.kv_heads = int(p["hidden"]), int(p["heads"]), int(p["kv_heads"])
        self.head_dim, self.v_dim, self.taps = int(p["head_dim"]), int(p["v_dim"]), int(p["conv"])
        self.eps = float(p["eps"])
        self.unit_eps = float(p.get("unit_eps", 1e-6))
        if self.heads % self.kv_heads or self.taps < 1:
            raise ValueError(f"gated_delta: {self.heads} heads over {self.kv_heads} key heads, {self.taps} taps")
        names = dict(p.get("names") or {})
        self.names = {k: names.get(k, d) for k, d in self.DEFAULT_NAMES.items()}
        self.qk_size, self.v_size = self.kv_heads * self.head_dim, self.heads * self.v_dim
        self.channels = 2 * self.qk_size + self.v_size
        self.dp = ops.scan_padded_dim(self.head_dim)
        self.rec_cols = -(-(2 * self.kv_heads * self.dp + self.v_size + 2 * self.heads + self.kv_heads) // 4) * 4  # q, k, v, g, beta, k . q
        self.s_floats = self.heads * self.head_dim * self.v_dim
        self.off_g = self.channels
        self.off_b = self.channels + self.v_size
        self.off_a = self.off_b + self.heads
        self.w_in = self.w_o = self.conv_taps = self.a_log = self.dt_bias = self.gain = None

    def weight_specs(self) -> dict[str, WeightSpec]:
        n = self.names
        small = dict(rule="float32")
        return {
            n["q"]: WeightSpec((self.qk_size, self.hidden)), n["k"]: WeightSpec((self.qk_size, self.hidden)),
            n["v"]: WeightSpec((self.v_size, self.hidden)), n["g"]: WeightSpec((self.v_size, self.hidden)),
            n["b"]: WeightSpec((self.heads, self.hidden)), n["a"]: WeightSpec((self.heads, self.hidden)),
            n["o"]: WeightSpec((self.hidden, self.v_size)),
            n["q_conv"]: WeightSpec((self.qk_size, self.taps), std=0.5, **small),
            n["k_conv"]: WeightSpec((self.qk_size, self.taps), std=0.5, **small),
            n["v_conv"]: WeightSpec((self.v_size, self.taps), std=0.5, **small),
            n["A_log"]: WeightSpec((self.heads,), std=0.5, **small), n["dt_bias"]: WeightSpec((self.heads,), std=0.5, **small),
            n["norm"]: WeightSpec((self.v_dim,), init="gain", **small),
        }

    def bind(self, tensors) -> None:
        n = self.names
        self.w_in = _pad_rows(torch.cat([tensors[n[k]] for k in ("q", "k", "v", "g", "b", "a")], dim=0))
        self.w_o = tensors[n["o"]].contiguous()
        self.conv_taps = torch.cat([tensors[n[k]] for k in ("q_conv", "k_conv", "v_conv")], dim=0).contiguous()
        self.a_log, self.dt_bias = tensors[n["A_log"]].contiguous(), tensors[n["dt_bias"]].contiguous()
        self.gain = tensors[n["norm"]].contiguous()

    def cache_need(self) -> CacheNeed | None:
        return None

    def state_need(self) -> StateNeed | None:
        # S, then the convolution's last taps - 1 inputs [taps - 1, channels]
        return StateNeed((self.s_floats + (self.taps - 1) * self.channels,), torch.float32)

    def forward(self, x, ctx: StepContext, lane: LaneView, writes: bool = True):
        if not writes:
            raise ValueError("a delta-rule mixer owns its state: its lane cannot be shared")
        proj = ops.linear(x, self.w_in, ctx.buffer("rec_proj", self.w_in.shape[0]))
        rec = ctx.buffer("rec_in", self.rec_cols, torch.float32)
        ops.delta_prepare(proj, self.conv_taps, self.a_log, self.dt_bias, lane.state, self.s_floats, ctx, rec, self.kv_heads,
                          self.heads, self.head_dim, self.v_dim, self.off_b, self.off_a, self.head_dim ** -0.5, self.unit_eps)
        read = ops.linear_scan(rec, lane.state, ctx, ctx.buffer("rec_out", self.v_size, torch.float32), self.heads, self.kv_heads,
                               self.head_dim, self.v_dim, gated=True)
        gate = proj[:, self.off_g: self.off_g + self.v_size]
        y = ops.head_norm_gate(read, gate, self.gain, self.eps, ctx.buffer("rec_y", self.v_size), ctx, self.heads, self.v_dim)
        return ops.linear(y, self.w_o, ctx.buffer("branch", self.hidden))


@register_part("mixer", "mamba2")
class Mamba2(Part):
    """params: hidden, heads, v_dim (features of a head), state (rows of S), groups (of heads that share B and C; head h reads group
    h // (heads / groups)), conv (taps of the short convolution), norm_groups (parts of the read-out's norm), eps, out_scale (the normed read-out is
    multiplied by it, through the norm's gain; default 1), names (optional: keys
    "in", "conv", "conv_bias", "dt_bias", "A_log", "D", "norm", "o"; default those words, the bias "conv.b")."""

    DEFAULT_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D", "norm": "norm", "o": "o"}

    def __init__(self, spec, dtype, device) -> None:
        super().__init__(spec, dtype, device)
        p = spec.params
        self.hidden, self.heads, self.v_dim = int(p["hidden"]), int(p["heads"]), int(p["v_dim"])
        self.state_dim, self.groups, self.taps = int(p["state"]), int(p["groups"]), int(p["conv"])
        self.norm_groups, self.eps = int(p["norm_groups"]), float(p["eps"])
        self.out_scale = float(p.get("out_scale", 1.0))
        self.inner = self.heads * self.v_dim
        if self.heads % self.groups or self.taps < 1 or self.inner % self.norm_groups:
            raise ValueError(f"mamba2: {self.heads} heads in {self.groups} groups, {self.taps} taps, {self.inner} features in {self.norm_groups} parts")
        names = dict(p.get("names") or {})
        self.names = {k: names.get(k, d) for k, d in self.DEFAULT_NAMES.items()}
        self.channels = self.inner + 2 * self.groups * self.state_dim        # what the convolution acts on
        self.columns = self.inner + self.channels + self.heads
        dp = ops.ssm_padded_dim(self.state_dim)
        self.off_x = 2 * self.groups * dp                                    # of x in the preparation's rows
        self.rec_cols = -(-(self.off_x + self.inner + 2 * self.heads + self.groups) // 4) * 4
        self.tail_off = -(-self.heads * self.state_dim * self.v_dim // 4) * 4
        self.state_floats = -(-(self.tail_off + (self.taps - 1) * self.channels) // 4) * 4
        self.w_in = self.w_o = self.conv_taps = self.conv_bias = self.a_log = self.dt_bias = self.skip = self.gain = None

    def weight_specs(self) -> dict[str, WeightSpec]:
        n = self.names
        small = dict(rule="float32")
        return {
            n["in"]: WeightSpec((self.columns, self.hidden)), n["o"]: WeightSpec((self.hidden, self.inner)),
            n["conv"]: WeightSpec((self.channels, self.taps), std=0.5, **small), n["conv_bias"]: WeightSpec((self.channels,), std=0.1, **small),
            n["dt_bias"]: WeightSpec((self.heads,), std=0.5, **small), n["A_log"]: WeightSpec((self.heads,), std=0.5, **small),
            n["D"]: WeightSpec((self.heads,), init="gain", **small), n["norm"]: WeightSpec((self.inner,), init="gain", **small),
        }

    def bind(self, tensors) -> None:
        n = self.names
        self.w_in, self.w_o = _pad_rows(tensors[n["in"]]), tensors[n["o"]].contiguous()
        self.conv_taps = tensors[n["conv"]].t().contiguous()                 # one row per tap, as the kernel reads them
        self.conv_bias, self.dt_bias = tensors[n["conv_bias"]].contiguous(), tensors[n["dt_bias"]].contiguous()
        self.a_log, self.skip, self.gain = (tensors[n[k]].contiguous() for k in ("A_log", "D", "norm"))
        if self.out_scale != 1.0:
            self.gain = self.gain * self.out_scale

    def cache_need(self) -> CacheNeed | None:
        return None

    def state_need(self) -> StateNeed | None:
        # S, then the convolution's last taps - 1 inputs [taps - 1, channels]
        return StateNeed((self.state_floats,), torch.float32)

    def forward(self, x, ctx: StepContext, lane: LaneView, writes: bool = True):
        proj = ops.linear(x, self.w_in, ctx.buffer("rec_proj", self.w_in.shape[0]))
        y = ctx.buffer("rec_y", self.inner)
        self.forward_projected(proj, ctx, lane, writes, y)
        return ops.linear(y, self.w_o, ctx.buffer("branch", self.hidden))

    # ---- optional: an arrangement that runs the two products inside larger ones of its own (see `GQAAttention.packs_projections`)
    packs_projections = True

    @property
    def input_weight(self) -> torch.Tensor:
        return self.w_in

    @property
    def output_weight(self) -> torch.Tensor:
        return self.w_o

    def adopt(self, w_in: torch.Tensor, w_out: torch.Tensor) -> None:
        if w_in.shape != self.w_in.shape or w_out.shape != self.w_o.shape:
            raise ValueError("adopt: views of the projections' own shapes are needed")
        self.w_in, self.w_o = w_in, w_out

    def forward_projected(self, proj: torch.Tensor, ctx: StepContext, lane: LaneView, writes: bool, y: torch.Tensor) -> None:
        """`proj` [N, >= columns] (rows may lie in a wider buffer): preparation, the state's walk, gate and norm into `y` [N, heads * v_dim]."""
        if not writes:
            raise ValueError("a mamba2 mixer owns its state: its lane cannot be shared")
        rec = ctx.buffer("rec_in", self.rec_cols, torch.float32)
        ops.ssm_prepare(proj, self.conv_taps, self.conv_bias, self.a_log, self.dt_bias, lane.state, self.tail_off, ctx, rec, self.groups,
                        self.heads, self.state_dim, self.v_dim)
        read = ops.ssm_scan(rec, self.a_log, lane.state, ctx, ctx.buffer("rec_out", -(-self.inner // 4) * 4, torch.float32), self.heads,
                            self.groups, self.state_dim, self.v_dim)
        ops.ssm_gate_norm(read, rec[:, self.off_x: self.off_x + self.inner], proj, self.skip, self.gain, self.eps, self.norm_groups, y,
                          lane.state, self.tail_off, self.channels, self.taps, ctx, self.heads, self.v_dim)
