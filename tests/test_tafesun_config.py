"""The Tafesun configuration, its recipe, its tensor names and the plain statement's own mechanisms, without a GPU."""

from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_tafesun as plain
import nanospec_b200.architectures  # noqa: F401  (registers the architectures)


def layer(mlp=True, **kw):
    return {"type": "parallel",
            "mixer": {"left": {"heads": 6, "kv_heads": 3, "dim": 10, "vdim": 14, "scale": 0.4, "rot": {"dims": 4, "base": 90.0, "scaling": {"factor": 3.0}}},
                      "right": {"heads": 4, "vdim": 5, "state": 7, "groups": 2, "conv": 4, "norm_groups": 5}, "left_scale": 0.7, "right_scale": 1.3},
            "mlp": {"kind": "moe", "expert": {"ff": 9, "limit": 0.9}, "router": {"experts": 5, "top": 3}, "shared": {"ff": 11, "limit": 2.5}} if mlp else None,
            **kw}


def small_config():
    return {"architecture": "Tafesun", "vocab": 53, "width": 20, "norm": {"eps": 1e-5}, "logit_scale": 0.6,
            "layers": [layer(), layer(mlp=False), layer(weights_of=0), layer(mlp=False, weights_of=1), layer(weights_of=2)]}


def test_config_round_trip_and_recipe():
    from nanospec_b200.config import TafesunConfig, resolve_architecture

    cfg = small_config()
    arch = resolve_architecture(cfg)
    assert arch.name == "Tafesun"
    typed = arch.config_from_hf(cfg, None)
    assert isinstance(typed, TafesunConfig) and typed.width == 20 and typed.eps == 1e-5 and typed.logit_scale == 0.6
    assert TafesunConfig.from_hf(typed.to_hf()) == typed
    recipe = arch.recipe(typed)
    assert [spec.prefix for spec in recipe.layers] == ["l0.", "l1."] and all(spec.block == "sandwich" for spec in recipe.layers)
    assert [run.layer for run in recipe.order] == [0, 1, 0, 1, 0]  # a chain of shared tensors ends at their owner
    assert [run.lane for run in recipe.order] == [0, 1, 2, 3, 4] and all(run.writes for run in recipe.order)
    m = recipe.layers[0].mixer
    assert m.kind == "side_by_side" and (m["left_scale"], m["right_scale"]) == (0.7, 1.3)
    a, s = m["left"].params, m["right"].params
    assert (a["heads"], a["kv_heads"], a["head_dim"], a["v_dim"], a["scale"]) == (6, 3, 10, 14, 0.4) and a["bias"] == "qkv" and a["feature_gate"]
    assert a["position"]["scaling"] == {"factor": 3.0} and a["position"]["dims"] == 4 and a["position"]["layout"] == "half" and a["window"] == 0
    assert (s["heads"], s["v_dim"], s["state"], s["groups"], s["conv"], s["norm_groups"], s["eps"]) == (4, 5, 7, 2, 4, 5, 1e-5)
    f = recipe.layers[0].feed_forward.params
    assert (f["experts"], f["top"], f["intermediate"], f["score"]) == (5, 3, 9, "chosen") and f["bias"] and not f.get("identity")
    assert f["unit"] == {"alpha": 1.702, "shift": 1.0, "limit": 0.9} and f["shared"] == {"intermediate": 11, "unit": {"alpha": 1.702, "shift": 1.0, "limit": 2.5}}
    assert recipe.layers[1].feed_forward is None and recipe.head["tied_to"] == "embed" and recipe.head["scale"] == 0.6


def test_defaults_and_refusals():
    from nanospec_b200.config import ConfigError, TafesunConfig

    cfg = small_config()
    cfg["layers"] = [layer()]
    del cfg["layers"][0]["mlp"]["shared"]
    del cfg["layers"][0]["mixer"]["left"]["kv_heads"]
    del cfg["layers"][0]["mixer"]["left"]["vdim"]
    del cfg["layers"][0]["mixer"]["left"]["rot"]["scaling"]
    typed = TafesunConfig.from_hf(cfg)
    left = typed.layers[0].mixer["left"]
    assert typed.layers[0].mlp["shared"] is None and left["kv_heads"] == 6 and left["vdim"] == 10 and "scaling" not in left["rot"]
    assert TafesunConfig.from_hf(typed.to_hf()) == typed

    def broken(change):
        c = small_config()
        change(c)
        with pytest.raises(ConfigError) as err:
            TafesunConfig.from_hf(c)
        return str(err.value)

    assert "layers[1].mixer lacks 'right'" in broken(lambda c: c["layers"][1]["mixer"].pop("right"))
    assert "unknown mixer type" in broken(lambda c: c["layers"][0].update(type="mamba2"))
    assert "key heads" in broken(lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4))
    assert "rot" in broken(lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=12))
    assert "factor" in broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0))
    assert "groups" in broken(lambda c: c["layers"][0]["mixer"]["right"].update(groups=3))
    assert "equal parts" in broken(lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=3))
    assert "left_scale" in broken(lambda c: c["layers"][0]["mixer"].pop("left_scale"))
    assert "6 of 5 experts" in broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=6))
    assert "limit" in broken(lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0))
    assert "limit" in broken(lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"))
    assert "feed-forward kind" in broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    assert "is not like it" in broken(lambda c: c["layers"][2]["mixer"].update(left_scale=0.5))
    assert "names no layer" in broken(lambda c: c["layers"][2].update(weights_of=9))
    assert "names no layer" in broken(lambda c: c["layers"][0].update(weights_of=2))
    assert "not a Tafesun config" in broken(lambda c: c.update(architecture="Other"))
    assert "norm" in broken(lambda c: c.pop("norm"))


def test_tensor_names_needs_and_loader_errors(tmp_path):
    from nanospec_b200.weights import WeightError, build_model, load_model, write_random_model, write_safetensors
    from nanospec_b200.weights.safetensors_io import SafetensorsFile

    cfg = small_config()
    model, _ = build_model(cfg, None, torch.float32, "cpu")
    specs = model.weight_specs()
    for name in ("l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l1.norm1", "l1.norm1b", "final.norm"):
        assert specs[name].shape == (20,) and specs[name + ".b"].shape == (20,) and specs[name + ".alpha"].shape == ()
    assert specs["l0.mix.left.q"].shape == (60, 20) and specs["l0.mix.left.q.b"].shape == (60,) and specs["l0.mix.left.v"].shape == (42, 20)
    assert specs["l0.mix.left.g"].shape == (84, 20) and specs["l0.mix.left.o"].shape == (20, 84) and "l0.mix.left.o.b" not in specs
    assert specs["l0.mix.right.in"].shape == (2 * 20 + 2 * 14 + 4, 20) and specs["l0.mix.right.conv"].shape == (48, 4) and specs["l0.mix.right.conv.b"].shape == (48,)
    assert all(specs[f"l1.mix.right.{n}"].shape == (4,) for n in ("dt_bias", "A_log", "D")) and specs["l1.mix.right.norm"].shape == (20,)
    assert specs["l0.mlp.router"].shape == (5, 20) and specs["l0.mlp.router.b"].shape == (5,) and specs["l0.mlp.e4.down"].shape == (20, 9)
    assert specs["l0.mlp.shared.up"].shape == (11, 20) and not any(n.startswith(("l1.mlp", "l1.norm2", "l2.", "l3.", "l4.")) for n in specs)
    needs = model.lane_needs()
    assert len(needs) == 5 and all(c.kv_heads == 3 and c.v_dim == 14 and c.window == 0 for c, _ in needs)
    assert all(s.shape[0] >= 4 * 7 * 5 + 3 * 48 for _, s in needs)
    folder = write_random_model(tmp_path / "m", cfg, seed=3)
    with SafetensorsFile(folder / "model.safetensors") as f:
        tensors = {k: f.tensor(k).clone() for k in f.keys()}
    assert set(tensors) | {"head"} == set(specs) and "head" not in tensors  # the head is the embedding's table
    loaded = load_model(folder, device="cpu", dtype=torch.float32)
    assert loaded.head.weight.data_ptr() == loaded.embedding.table.data_ptr()
    del tensors["l0.mlp.router.b"]
    tensors["l2.mix.left.q"] = torch.zeros(60, 20, dtype=torch.bfloat16)
    tensors["l0.norm1.alpha"] = torch.zeros(1, dtype=torch.bfloat16)
    write_safetensors(folder / "model.safetensors", tensors)
    with pytest.raises(WeightError) as err:
        load_model(folder, device="cpu", dtype=torch.float32)
    assert all(n in str(err.value) for n in ("l0.mlp.router.b", "l2.mix.left.q", "l0.norm1.alpha"))


def test_side_by_side_takes_one_holder_of_pages_and_one_of_state():
    from nanospec_b200.config import PartSpec
    from nanospec_b200.parts import build_part
    from nanospec_b200.config import TafesunConfig
    from nanospec_b200.architectures.tafesun import tafesun_recipe

    spec = tafesun_recipe(TafesunConfig.from_hf(small_config())).layers[0].mixer
    part = build_part("mixer", spec, torch.float32, torch.device("cpu"))
    assert part.left.out_scale == 0.7 and part.right.out_scale == 1.3
    for side in ("left", "right"):
        both = PartSpec("side_by_side", {**spec.params, "left": spec[side], "right": spec[side]})
        with pytest.raises(ValueError, match="only one"):
            build_part("mixer", both, torch.float32, torch.device("cpu"))
    with pytest.raises(ValueError, match="does not offer"):
        build_part("mixer", PartSpec("side_by_side", {**spec.params, "left": PartSpec("retention", {
            "hidden": 20, "heads": 2, "head_dim": 4, "v_dim": 4, "decay": [0.5, 0.5], "eps": 1e-5})}), torch.float32, torch.device("cpu"))


# ---- the plain statement's own mechanisms: a second, independent writing of each ----------------------------------------

def test_plain_norm_unit_and_rotation():
    W = {"n": torch.tensor([2.0, -1.0], dtype=torch.float64), "n.b": torch.tensor([0.5, 0.25], dtype=torch.float64), "n.alpha": torch.tensor(0.3, dtype=torch.float64)}
    y = plain.dynamic_tanh(torch.tensor([[1.5, -4.0]], dtype=torch.float64), W, "n")
    assert torch.allclose(y, torch.tensor([[2 * math.tanh(0.45) + 0.5, -math.tanh(-1.2) + 0.25]], dtype=torch.float64))
    eye = {f"e.{n}": torch.eye(3, dtype=torch.float64) for n in ("gate", "up", "down")}
    z = torch.tensor([[2.0, -3.0, 0.5]], dtype=torch.float64)  # gate and up both see z
    want = []
    for v in (2.0, -3.0, 0.5):
        g, u = min(v, 1.2), max(min(v, 1.2), -1.2)
        want.append(g / (1 + math.exp(-1.702 * g)) * (u + 1))
    assert torch.allclose(plain.expert(z, eye, "e.", 1.2), torch.tensor([want], dtype=torch.float64))
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 9.0]]], dtype=torch.float64)
    rot = {"dims": 4, "base": 100.0, "scaling": {"factor": 2.0}}
    got = plain.rotate_half(x, torch.tensor([3]), rot)[0, 0]
    c = complex(1.0, 3.0) * complex(math.cos(1.5), math.sin(1.5)), complex(2.0, 4.0) * complex(math.cos(0.15), math.sin(0.15))
    assert torch.allclose(got, torch.tensor([c[0].real, c[1].real, c[0].imag, c[1].imag, 9.0], dtype=torch.float64))
    plain_rot = {"dims": 4, "base": 100.0}
    assert torch.allclose(plain.rotate_half(x, torch.tensor([6]), rot), plain.rotate_half(x, torch.tensor([3]), plain_rot))


def test_framework_frequencies_with_one_factor():
    from nanospec_b200.parts.position import rotary_frequencies

    f, magnitude = rotary_frequencies(12, 5000.0, {"factor": 2.5})
    assert magnitude == 1.0 and torch.allclose(f.double(), plain.frequencies({"dims": 12, "base": 5000.0, "scaling": {"factor": 2.5}}), rtol=1e-6)


def test_plain_route_and_state_space():
    g = torch.Generator().manual_seed(5)
    W = {"router": torch.randn(6, 4, generator=g, dtype=torch.float64), "router.b": torch.randn(6, generator=g, dtype=torch.float64)}
    h = torch.randn(3, 4, generator=g, dtype=torch.float64)
    chosen, weights = plain.route(h, {"top": 2}, W, "")
    for t in range(3):
        z = [float(W["router"][e] @ h[t] + W["router.b"][e]) for e in range(6)]
        best = sorted(range(6), key=lambda e: -z[e])[:2]
        assert chosen[t].tolist() == best
        assert math.isclose(float(weights[t, 0]), 1 / (1 + math.exp(z[best[1]] - z[best[0]])), rel_tol=1e-9) and math.isclose(float(weights[t].sum()), 1.0)
    T, H, G, N, V = 5, 4, 2, 3, 2
    x, B, C = (torch.randn(T, n, m, generator=g, dtype=torch.float64) for n, m in ((H, V), (G, N), (G, N)))
    dt, a_log, D = torch.rand(T, H, generator=g, dtype=torch.float64), torch.randn(H, generator=g, dtype=torch.float64), torch.randn(H, generator=g, dtype=torch.float64)
    y = plain.state_space_walk(x, B, C, dt, a_log, D)
    for h_ in range(H):
        for t in range(T):  # the sum over the past, written out
            want = D[h_] * x[t, h_]
            for s in range(t + 1):
                decay = math.exp(-math.exp(float(a_log[h_])) * float(dt[s + 1: t + 1, h_].sum()))
                want = want + decay * dt[s, h_] * (B[s, h_ // 2] @ C[t, h_ // 2]) * x[s, h_]
            assert torch.allclose(y[t, h_], want, atol=1e-9)


def test_plain_forward_shares_tensors_and_depends_on_every_piece():
    from nanospec_b200.weights import build_model

    cfg = small_config()
    model, _ = build_model(cfg, None, torch.float32, "cpu")
    g = torch.Generator().manual_seed(1)
    w = {n: torch.randn(s.shape, generator=g) * 0.4 for n, s in sorted(model.weight_specs().items()) if n != "head"}
    w["l0.norm2"], w["l0.norm2.b"], w["l0.mlp.router.b"] = torch.ones(20), torch.zeros(20), torch.zeros(5)  # every expert has tokens
    ids = torch.randint(0, 53, (30,), generator=g).tolist()
    base = plain.forward(cfg, w, ids)
    assert torch.allclose(plain.forward(cfg, w, ids[:4]), base[:4])  # causal
    one = copy.deepcopy(cfg)
    one["layers"] = one["layers"][:2]
    assert not torch.allclose(plain.forward(one, w, ids), base)
    for name in w:
        other = dict(w)
        other[name] = w[name] + 0.3 * torch.randn(w[name].shape, generator=g)
        assert float((plain.forward(cfg, other, ids) - base).abs().max()) > 1e-9, name
