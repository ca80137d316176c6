"""The Tafesun decoder as a recipe: layers in the "sandwich" arrangement (a dynamic tanh on what each sublayer reads and on what it returns)
around attention and the Mamba-2 state space side by side on one input, with routed experts and a shared one or no feed-forward; the head is
the embedding's table.

    left     grouped-query attention: biases on q, k and v, rotation in halves with all frequencies divided by one factor, every earlier key,
             a sigmoid gate per feature of the concatenated heads
    right    mamba2: short convolution with a bias, a state per head that decays by a step size per token, gate and then norm in parts
    moe      the largest biased router logits choose, their softmax among themselves weighs; gated units held within a limit

A layer that uses another's tensors is a second run of that layer in the order, on a lane of its own.

Tensor names: `embed`, `l<i>.norm1`, `l<i>.norm1b`, `l<i>.norm2`, `l<i>.norm2b` (each + `.b`, `.alpha`), `l<i>.mix.left.{q, k, v}` (+ `.b`),
`l<i>.mix.left.{g, o}`, `l<i>.mix.right.{in, conv, conv.b, dt_bias, A_log, D, norm, o}`, `l<i>.mlp.{router, router.b}`,
`l<i>.mlp.{e<k>, shared}.{gate, up, down}`, `final.norm` (+ `.b`, `.alpha`)."""

from __future__ import annotations

from ..config.recipe import LayerSpec, ModelRecipe, PartSpec, Run
from ..config.registry import Architecture, register_architecture
from ..config.tafesun import MAX_POSITIONS, TafesunConfig

UNIT_ALPHA, UNIT_SHIFT = 1.702, 1.0  # an expert's unit: g sigmoid(1.702 g) (u + 1)


def _mixer(m: dict, width: int, eps: float) -> PartSpec:
    a, s = m["left"], m["right"]
    position = PartSpec("rotary", {"head_dim": a["dim"], "dims": a["rot"]["dims"], "base": a["rot"]["base"], "layout": "half",
                                   "scaling": a["rot"].get("scaling")})
    left = PartSpec("gqa_attention", {
        "hidden": width, "heads": a["heads"], "kv_heads": a["kv_heads"], "head_dim": a["dim"], "v_dim": a["vdim"], "scale": a["scale"],
        "window": 0, "bias": "qkv", "feature_gate": True, "position": position, "wide_weights": True,
        "names": {k: k for k in ("q", "k", "v", "o", "g")}})
    right = PartSpec("mamba2", {"hidden": width, "heads": s["heads"], "v_dim": s["vdim"], "state": s["state"], "groups": s["groups"],
                                "conv": s["conv"], "norm_groups": s["norm_groups"], "eps": eps})
    return PartSpec("side_by_side", {"hidden": width, "left": left, "right": right, "left_scale": m["left_scale"], "right_scale": m["right_scale"]})


def _unit(limit: float) -> dict:
    return {"alpha": UNIT_ALPHA, "shift": UNIT_SHIFT, "limit": limit}


def _feed_forward(mlp: dict | None, width: int) -> PartSpec | None:
    if mlp is None:
        return None
    r, e, s = mlp["router"], mlp["expert"], mlp["shared"]
    return PartSpec("routed_experts", {
        "hidden": width, "experts": r["experts"], "top": r["top"], "intermediate": e["ff"], "score": "chosen", "bias": True, "unit": _unit(e["limit"]),
        "shared": None if s is None else {"intermediate": s["ff"], "unit": _unit(s["limit"])}})


def tafesun_recipe(cfg: TafesunConfig) -> ModelRecipe:
    norm = PartSpec("dyt", {"hidden": cfg.width, "weight_name": "", "bias_name": ".b", "alpha_name": ".alpha"})
    own = [i for i, layer in enumerate(cfg.layers) if layer.weights_of is None]
    layers = tuple(
        LayerSpec(block="sandwich", prefix=f"l{i}.", mixer=_mixer(cfg.layers[i].mixer, cfg.width, cfg.eps),
                  feed_forward=_feed_forward(cfg.layers[i].mlp, cfg.width), norm=norm,
                  names={"mixer": "mix.", "feed_forward": "mlp.", "norm_mixer": "norm1", "post_mixer": "norm1b", "norm_feed_forward": "norm2",
                         "post_feed_forward": "norm2b"})
        for i in own)
    order = tuple(Run(layer=own.index(i if layer.weights_of is None else layer.weights_of), lane=i) for i, layer in enumerate(cfg.layers))
    return ModelRecipe(
        architecture=cfg.architecture, embedding=PartSpec("table", {"vocab": cfg.vocab, "hidden": cfg.width, "prefix": "", "weight_name": "embed"}),
        layers=layers, order=order, final_norm=norm, final_norm_prefix="final.norm",
        head=PartSpec("linear", {"vocab": cfg.vocab, "hidden": cfg.width, "prefix": "", "weight_name": "head", "tied_to": "embed",
                                 "scale": cfg.logit_scale}),
        vocab_size=cfg.vocab, hidden_size=cfg.width, max_positions=MAX_POSITIONS, eos_token_ids=cfg.eos_token_ids)


TAFESUN = register_architecture(Architecture(
    name="Tafesun", model_type="tafesun", config_from_hf=TafesunConfig.from_hf, recipe=tafesun_recipe))
