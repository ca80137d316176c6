"""The Rasezen decoder as a recipe: layers in the "parallel" arrangement (one RMS norm with a single number for a gain, whose output
the mixer and the feed-forward both read) around windowed grouped-query attention or the Mamba-2 state space, with a dense xielu
feed-forward, routed experts or none; a final norm of the same kind and a head.

    attention   biases on q, k and v, an RMS norm over the whole q and the whole k projection, rotation in halves, values divided by
                their root mean square per head before they are cached, a sliding window
    mamba2      short convolution with a bias, a state per head that decays by a step size per token, gate and then norm in parts
    moe         softmax over all router outputs, the choice by score plus correction, weights not renormalized, the last outputs
                standing for experts that return their input, a shared expert beside them

Tensor names: `embed`, `l<i>.norm1`, `l<i>.mix.{q, k, v}` (+ `.b`), `l<i>.mix.{q, k}.norm`, `l<i>.mix.o`, or `l<i>.mix.{in, conv, conv.b,
dt_bias, A_log, D, norm, o}`; `l<i>.mlp.{up, down, act}`, or `l<i>.mlp.{router, correction, e<k>.{gate, up, down}, shared.{gate, up, down}}`;
`final.norm`, `head`."""

from __future__ import annotations

from ..config.rasezen import MAX_POSITIONS, RasezenConfig
from ..config.recipe import LayerSpec, ModelRecipe, PartSpec, Run
from ..config.registry import Architecture, register_architecture


def _mixer(kind: str, m: dict, width: int, eps: float) -> PartSpec:
    if kind == "mamba2":
        return PartSpec("mamba2", {"hidden": width, "heads": m["heads"], "v_dim": m["vdim"], "state": m["state"], "groups": m["groups"],
                                   "conv": m["conv"], "norm_groups": m["norm_groups"], "eps": eps})
    position = PartSpec("rotary", {"head_dim": m["dim"], "dims": m["rot"]["dims"], "base": m["rot"]["base"], "layout": "half", "scaling": None})
    return PartSpec("gqa_attention", {
        "hidden": width, "heads": m["heads"], "kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_dim": m["vdim"], "scale": m["scale"],
        "window": m["mask"]["size"], "qk_norm": {"eps": eps}, "v_norm": {"eps": eps}, "bias": "qkv", "position": position,
        "wide_weights": True, "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"}})


def _feed_forward(mlp: dict | None, width: int) -> PartSpec | None:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("dense_act", {"hidden": width, "intermediate": mlp["ff"], "activation": "xielu"})
    r = mlp["router"]
    return PartSpec("routed_experts", {
        "hidden": width, "experts": r["experts"], "identity": r["identity"], "top": r["top"], "scale": r["scale"],
        "intermediate": mlp["expert"]["ff"], "score": "softmax", "correction": True, "renormalize": False,
        "shared": None if mlp["shared"] is None else {"intermediate": mlp["shared"]["ff"]}})


def rasezen_recipe(cfg: RasezenConfig) -> ModelRecipe:
    norm = PartSpec("rmsnorm", {"hidden": cfg.width, "eps": cfg.eps, "weight_name": "", "scalar": True})
    layers = tuple(
        LayerSpec(block="parallel", prefix=f"l{i}.", mixer=_mixer(layer.type, layer.mixer, cfg.width, cfg.eps),
                  feed_forward=_feed_forward(layer.mlp, cfg.width), norm=norm,
                  names={"mixer": "mix.", "feed_forward": "mlp.", "norm_mixer": "norm1"})
        for i, layer in enumerate(cfg.layers))
    return ModelRecipe(
        architecture=cfg.architecture, embedding=PartSpec("table", {"vocab": cfg.vocab, "hidden": cfg.width, "prefix": "", "weight_name": "embed"}),
        layers=layers, order=tuple(Run(layer=i, lane=i) for i in range(len(layers))), final_norm=norm, final_norm_prefix="final.norm",
        head=PartSpec("linear", {"vocab": cfg.vocab, "hidden": cfg.width, "prefix": "", "weight_name": "head", "tied_to": None}),
        vocab_size=cfg.vocab, hidden_size=cfg.width, max_positions=MAX_POSITIONS, eos_token_ids=cfg.eos_token_ids)


RASEZEN = register_architecture(Architecture(
    name="Rasezen", model_type="rasezen", config_from_hf=RasezenConfig.from_hf, recipe=rasezen_recipe))
