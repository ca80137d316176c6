"""Typed configuration of the Rasezen decoder, read from its own config.json.

A Rasezen model is a list of layers with one norm each - an RMS norm whose gain is a single number - whose output both the mixer
and the feed-forward read: x = x + (mixer(h) + feed_forward(h)), h = norm(x).  The mixer is windowed softmax attention (biases on q,
k and v, one norm over the whole q and the whole k projection, rotation in halves, values of unit root mean square per head) or the
Mamba-2 state space; the feed-forward is dense (xielu), a set of routed experts (softmax scores, a correction on the choice, experts
that return their input, a shared expert), or absent.  Every size and every constant that can differ between models comes from the
file:

    architecture "Rasezen";  vocab, width;  norm.eps
    layers[i]: type ("attention" | "mamba2"), mixer {...}, mlp {...} or null
      attention: heads, kv_heads, dim, vdim, scale, mask {size}, rot {dims, base}
      mamba2:    heads, vdim, state, groups, conv, norm_groups
      mlp:       {kind "dense", ff}  or  {kind "moe", expert {ff}, router {experts, identity, top, scale}, shared {ff} or absent}
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .files import ConfigError

MIXER_TYPES = ("attention", "mamba2")
MAX_POSITIONS = 1 << 20  # the file gives no limit; positions are 32-bit and angles float32

_SIZES = {"attention": ("heads", "kv_heads", "dim", "vdim"), "mamba2": ("heads", "vdim", "state", "groups", "conv", "norm_groups")}


def _need(d: Any, key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"Rasezen config: {where} lacks {key!r}")
    return d[key]


def _size(d: dict, key: str, where: str, least: int = 1) -> int:
    n = int(_need(d, key, where))
    if n < least:
        raise ConfigError(f"Rasezen config: {where}.{key} = {n}")
    return n


def _mixer(kind: str, entry: dict, where: str) -> dict[str, Any]:
    m = dict(entry)
    if kind == "attention":
        if m.get("heads") is not None and m.get("kv_heads") is None:
            m["kv_heads"] = m["heads"]      # a file that leaves it out means one key head per head
        if m.get("dim") is not None and m.get("vdim") is None:
            m["vdim"] = m["dim"]            # ... and values as wide as keys
    for key in _SIZES[kind]:
        m[key] = _size(m, key, where)
    if kind == "mamba2":
        if m["heads"] % m["groups"]:
            raise ConfigError(f"Rasezen config: {where}: {m['heads']} heads in {m['groups']} groups")
        if m["heads"] * m["vdim"] % m["norm_groups"]:
            raise ConfigError(f"Rasezen config: {where}: {m['heads'] * m['vdim']} features in {m['norm_groups']} equal parts")
        return m
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"Rasezen config: {where}: {m['heads']} heads over {m['kv_heads']} key heads")
    m["scale"] = float(_need(m, "scale", where))
    m["mask"] = {"size": _size(_need(m, "mask", where), "size", where + ".mask")}
    rot = _need(m, "rot", where)
    m["rot"] = {"dims": _size(rot, "dims", where + ".rot", 0), "base": float(_need(rot, "base", where + ".rot"))}
    if m["rot"]["dims"] % 2 or m["rot"]["dims"] > m["dim"]:
        raise ConfigError(f"Rasezen config: {where}.rot turns {m['rot']['dims']} of {m['dim']} features")
    return m


def _feed_forward(mlp: Any, where: str) -> dict[str, Any] | None:
    if mlp is None:
        return None
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        return {"kind": "dense", "ff": _size(mlp, "ff", where)}
    if kind != "moe":
        raise ConfigError(f"Rasezen config: {where} has the unknown feed-forward kind {kind!r}")
    r = _need(mlp, "router", where)
    router = {"experts": _size(r, "experts", where + ".router"), "top": _size(r, "top", where + ".router"),
              "identity": int(r.get("identity") or 0), "scale": float(r["scale"]) if r.get("scale") is not None else 1.0}
    if router["identity"] < 0 or router["top"] > router["experts"] + router["identity"]:
        raise ConfigError(f"Rasezen config: {where}: {router['top']} of {router['experts']} + {router['identity']} experts")
    shared = mlp.get("shared")
    return {"kind": "moe", "expert": {"ff": _size(_need(mlp, "expert", where), "ff", where + ".expert")}, "router": router,
            "shared": None if shared is None else {"ff": _size(shared, "ff", where + ".shared")}}


@dataclass(frozen=True)
class RasezenLayer:
    type: str
    mixer: dict[str, Any]
    mlp: dict[str, Any] | None  # None: no feed-forward

    def to_hf(self) -> dict[str, Any]:
        mlp = self.mlp
        if mlp is not None and mlp.get("shared", 0) is None:
            mlp = {k: v for k, v in mlp.items() if k != "shared"}
        return {"type": self.type, "mixer": self.mixer, "mlp": mlp}


@dataclass(frozen=True)
class RasezenConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple[RasezenLayer, ...]
    eos_token_ids: tuple[int, ...] = ()
    architecture: str = "Rasezen"

    @classmethod
    def from_hf(cls, cfg: dict[str, Any], generation: dict[str, Any] | None = None) -> "RasezenConfig":
        if cfg.get("architecture") != "Rasezen" and "Rasezen" not in (cfg.get("architectures") or []):
            raise ConfigError(f"not a Rasezen config: architecture={cfg.get('architecture')!r}")
        layers = []
        for i, entry in enumerate(_need(cfg, "layers", "config.json")):
            where = f"layers[{i}]"
            kind = _need(entry, "type", where)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"Rasezen config: {where} has the unknown mixer type {kind!r} (known: {', '.join(MIXER_TYPES)})")
            layers.append(RasezenLayer(kind, _mixer(kind, _need(entry, "mixer", where), where + ".mixer"),
                                       _feed_forward(entry.get("mlp"), where + ".mlp")))
        if not layers:
            raise ConfigError("Rasezen config: no layers")
        eos = (generation or {}).get("eos_token_id", cfg.get("eos_token_id"))
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return cls(vocab=_size(cfg, "vocab", "config.json"), width=_size(cfg, "width", "config.json"),
                   eps=float(_need(_need(cfg, "norm", "config.json"), "eps", "norm")), layers=tuple(layers), eos_token_ids=eos_ids)

    def to_hf(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                               "layers": [layer.to_hf() for layer in self.layers]}
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
