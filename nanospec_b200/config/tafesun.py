"""Typed configuration of the Tafesun decoder, read from its own config.json.

A Tafesun layer norms what each of its two sublayers reads and what it returns, with a norm without statistics (a dynamic tanh).  The mixer
runs softmax attention and the Mamba-2 state space on the same input and adds the two with constant weights; the feed-forward is a set of
routed experts with a shared one, or absent.  A layer may use another layer's tensors (`weights_of`), with a cache and a state of its
own.  Every size and every constant that can differ between models comes from the file:

    architecture "Tafesun";  vocab, width;  norm.eps;  logit_scale
    layers[i]: type "parallel", mixer {left, right, left_scale, right_scale}, mlp {...} or null, weights_of (absent: its own tensors)
      left:   heads, kv_heads, dim, vdim, scale, rot {dims, base, scaling {factor}}
      right:  heads, vdim, state, groups, conv, norm_groups
      mlp:    kind "moe", expert {ff, limit}, router {experts, top}, shared {ff, limit} or absent
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .files import ConfigError

MIXER_TYPES = ("parallel",)
MAX_POSITIONS = 1 << 20  # the file gives no limit; positions are 32-bit and angles float32

_LEFT = ("heads", "kv_heads", "dim", "vdim")
_RIGHT = ("heads", "vdim", "state", "groups", "conv", "norm_groups")


def _need(d: Any, key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"Tafesun config: {where} lacks {key!r}")
    return d[key]


def _size(d: dict, key: str, where: str, least: int = 1) -> int:
    n = int(_need(d, key, where))
    if n < least:
        raise ConfigError(f"Tafesun config: {where}.{key} = {n}")
    return n


def _attention(entry: dict, where: str) -> dict[str, Any]:
    m = dict(entry)
    if m.get("heads") is not None and m.get("kv_heads") is None:
        m["kv_heads"] = m["heads"]      # a file that leaves it out means one key head per head
    if m.get("dim") is not None and m.get("vdim") is None:
        m["vdim"] = m["dim"]            # ... and values as wide as keys
    out: dict[str, Any] = {key: _size(m, key, where) for key in _LEFT}
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"Tafesun config: {where}: {out['heads']} heads over {out['kv_heads']} key heads")
    out["scale"] = float(_need(m, "scale", where))
    rot = _need(m, "rot", where)
    out["rot"] = {"dims": _size(rot, "dims", where + ".rot", 0), "base": float(_need(rot, "base", where + ".rot"))}
    if out["rot"]["dims"] % 2 or out["rot"]["dims"] > out["dim"]:
        raise ConfigError(f"Tafesun config: {where}.rot turns {out['rot']['dims']} of {out['dim']} features")
    if rot.get("scaling"):
        factor = float(_need(rot["scaling"], "factor", where + ".rot.scaling"))
        if factor <= 0:
            raise ConfigError(f"Tafesun config: {where}.rot.scaling.factor = {factor}")
        out["rot"]["scaling"] = {"factor": factor}
    return out


def _state_space(m: dict, where: str) -> dict[str, Any]:
    out: dict[str, Any] = {key: _size(m, key, where) for key in _RIGHT}
    if out["heads"] % out["groups"]:
        raise ConfigError(f"Tafesun config: {where}: {out['heads']} heads in {out['groups']} groups")
    if out["heads"] * out["vdim"] % out["norm_groups"]:
        raise ConfigError(f"Tafesun config: {where}: {out['heads'] * out['vdim']} features in {out['norm_groups']} equal parts")
    return out


def _mixer(m: dict, where: str) -> dict[str, Any]:
    return {"left": _attention(_need(m, "left", where), where + ".left"), "right": _state_space(_need(m, "right", where), where + ".right"),
            "left_scale": float(_need(m, "left_scale", where)), "right_scale": float(_need(m, "right_scale", where))}


def _expert(d: dict, where: str) -> dict[str, Any]:
    limit = float(_need(d, "limit", where))
    if limit <= 0:
        raise ConfigError(f"Tafesun config: {where}.limit = {limit}")
    return {"ff": _size(d, "ff", where), "limit": limit}


def _feed_forward(mlp: Any, where: str) -> dict[str, Any] | None:
    if mlp is None:
        return None
    if mlp.get("kind", "moe") != "moe":
        raise ConfigError(f"Tafesun config: {where} has the unknown feed-forward kind {mlp.get('kind')!r}")
    r = _need(mlp, "router", where)
    router = {"experts": _size(r, "experts", where + ".router"), "top": _size(r, "top", where + ".router")}
    if router["top"] > router["experts"]:
        raise ConfigError(f"Tafesun config: {where}: {router['top']} of {router['experts']} experts")
    shared = mlp.get("shared")
    return {"kind": "moe", "expert": _expert(_need(mlp, "expert", where), where + ".expert"), "router": router,
            "shared": None if shared is None else _expert(shared, where + ".shared")}


@dataclass(frozen=True)
class TafesunLayer:
    type: str
    mixer: dict[str, Any]
    mlp: dict[str, Any] | None  # None: no feed-forward
    weights_of: int | None = None  # the layer whose tensors this one uses (one that has its own); None: its own

    def to_hf(self) -> dict[str, Any]:
        mlp = self.mlp
        if mlp is not None and mlp["shared"] is None:
            mlp = {k: v for k, v in mlp.items() if k != "shared"}
        out = {"type": self.type, "mixer": self.mixer, "mlp": mlp}
        if self.weights_of is not None:
            out["weights_of"] = self.weights_of
        return out


@dataclass(frozen=True)
class TafesunConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple[TafesunLayer, ...]
    logit_scale: float = 1.0
    eos_token_ids: tuple[int, ...] = ()
    architecture: str = "Tafesun"

    @classmethod
    def from_hf(cls, cfg: dict[str, Any], generation: dict[str, Any] | None = None) -> "TafesunConfig":
        if cfg.get("architecture") != "Tafesun" and "Tafesun" not in (cfg.get("architectures") or []):
            raise ConfigError(f"not a Tafesun config: architecture={cfg.get('architecture')!r}")
        entries = list(_need(cfg, "layers", "config.json"))
        if not entries:
            raise ConfigError("Tafesun config: no layers")
        layers: list[TafesunLayer] = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]"
            kind = _need(entry, "type", where)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"Tafesun config: {where} has the unknown mixer type {kind!r} (known: {', '.join(MIXER_TYPES)})")
            layers.append(TafesunLayer(kind, _mixer(_need(entry, "mixer", where), where + ".mixer"), _feed_forward(entry.get("mlp"), where + ".mlp"),
                                       cls._owner(entries, i)))
        for i, layer in enumerate(layers):
            if layer.weights_of is not None:
                own = layers[layer.weights_of]
                if (layer.mixer, layer.mlp) != (own.mixer, own.mlp):
                    raise ConfigError(f"Tafesun config: layers[{i}] uses the tensors of layers[{layer.weights_of}] but is not like it")
        eos = (generation or {}).get("eos_token_id", cfg.get("eos_token_id"))
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        scale = cfg.get("logit_scale")
        return cls(vocab=_size(cfg, "vocab", "config.json"), width=_size(cfg, "width", "config.json"),
                   eps=float(_need(_need(cfg, "norm", "config.json"), "eps", "norm")), layers=tuple(layers),
                   logit_scale=1.0 if scale is None else float(scale), eos_token_ids=eos_ids)

    @staticmethod
    def _owner(entries: list, i: int) -> int | None:
        """The layer with tensors of its own at the end of layer i's chain of `weights_of`."""
        seen, at = {i}, i
        while entries[at].get("weights_of") is not None:
            at = int(entries[at]["weights_of"])
            if not 0 <= at < len(entries) or at in seen:
                raise ConfigError(f"Tafesun config: layers[{i}].weights_of names no layer with tensors of its own")
            seen.add(at)
        return None if at == i else at

    def to_hf(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                               "logit_scale": self.logit_scale, "layers": [layer.to_hf() for layer in self.layers]}
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
