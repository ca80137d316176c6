"""The Rasezen configuration, its recipe, its tensor names and the plain statement's own mechanisms, without a GPU."""

from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_rasezen as plain
import nanospec_b200.architectures  # noqa: F401  (registers the architectures)


def small_config():
    return {
        "architecture": "Rasezen", "vocab": 53, "width": 20, "norm": {"eps": 1e-5},
        "layers": [
            {"type": "mamba2", "mixer": {"heads": 6, "vdim": 5, "state": 7, "groups": 3, "conv": 3, "norm_groups": 5},
             "mlp": {"kind": "moe", "expert": {"ff": 9}, "router": {"experts": 4, "identity": 2, "scale": 1.7, "top": 3}, "shared": {"ff": 11}}},
            {"type": "attention", "mlp": {"kind": "dense", "ff": 26},
             "mixer": {"heads": 4, "kv_heads": 2, "dim": 10, "vdim": 6, "scale": 0.4, "mask": {"size": 5}, "rot": {"dims": 4, "base": 90.0}}},
            {"type": "attention", "mlp": None,
             "mixer": {"heads": 3, "kv_heads": 3, "dim": 8, "vdim": 8, "scale": 0.3, "mask": {"size": 2}, "rot": {"dims": 8, "base": 7000.0}}},
        ]}


def test_config_round_trip_and_recipe():
    from nanospec_b200.config import RasezenConfig, resolve_architecture

    cfg = small_config()
    arch = resolve_architecture(cfg)
    assert arch.name == "Rasezen"
    typed = arch.config_from_hf(cfg, None)
    assert isinstance(typed, RasezenConfig) and typed.width == 20 and typed.eps == 1e-5
    assert RasezenConfig.from_hf(typed.to_hf()) == typed
    recipe = arch.recipe(typed)
    assert [layer.block for layer in recipe.layers] == ["parallel"] * 3 and all(layer.norm["scalar"] for layer in recipe.layers)
    assert [run.lane for run in recipe.order] == [0, 1, 2] and all(run.writes for run in recipe.order)
    m, a, b = (layer.mixer.params for layer in recipe.layers)
    assert recipe.layers[0].mixer.kind == "mamba2" and (m["heads"], m["v_dim"], m["state"], m["groups"], m["conv"], m["norm_groups"]) == (6, 5, 7, 3, 3, 5)
    assert a["window"] == 5 and a["bias"] == "qkv" and a["v_norm"] == {"eps": 1e-5} and a["scale"] == 0.4 and a["position"]["layout"] == "half"
    assert a["position"]["dims"] == 4 and a["v_dim"] == 6 and b["kv_heads"] == 3
    f = recipe.layers[0].feed_forward.params
    assert (f["experts"], f["identity"], f["top"], f["scale"], f["intermediate"]) == (4, 2, 3, 1.7, 9)
    assert f["score"] == "softmax" and f["correction"] and not f["renormalize"] and f["shared"] == {"intermediate": 11}
    assert recipe.layers[1].feed_forward["activation"] == "xielu" and recipe.layers[2].feed_forward is None


def test_defaults_and_refusals():
    from nanospec_b200.config import ConfigError, RasezenConfig

    cfg = small_config()
    del cfg["layers"][0]["mlp"]["shared"]
    del cfg["layers"][0]["mlp"]["router"]["identity"]
    del cfg["layers"][2]["mixer"]["kv_heads"]
    del cfg["layers"][2]["mixer"]["vdim"]
    typed = RasezenConfig.from_hf(cfg)
    assert typed.layers[0].mlp["shared"] is None and typed.layers[0].mlp["router"]["identity"] == 0
    assert typed.layers[2].mixer["kv_heads"] == 3 and typed.layers[2].mixer["vdim"] == 8
    assert RasezenConfig.from_hf(typed.to_hf()) == typed

    def broken(change):
        c = small_config()
        change(c)
        with pytest.raises(ConfigError) as err:
            RasezenConfig.from_hf(c)
        return str(err.value)

    assert "layers[1]" in broken(lambda c: c["layers"][1]["mixer"].pop("mask"))
    assert "unknown mixer type" in broken(lambda c: c["layers"][0].update(type="mamba3"))
    assert "key heads" in broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=3))
    assert "rot" in broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=12))
    assert "mask.size" in broken(lambda c: c["layers"][1]["mixer"]["mask"].update(size=0))
    assert "groups" in broken(lambda c: c["layers"][0]["mixer"].update(groups=4))
    assert "equal parts" in broken(lambda c: c["layers"][0]["mixer"].update(norm_groups=4))
    assert "conv" in broken(lambda c: c["layers"][0]["mixer"].update(conv=0))
    assert "7 of 4 + 2 experts" in broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=7))
    assert "feed-forward kind" in broken(lambda c: c["layers"][1]["mlp"].update(kind="gated"))
    assert "not a Rasezen config" in broken(lambda c: c.update(architecture="Other"))
    assert "norm" in broken(lambda c: c.pop("norm"))


def test_tensor_names_states_and_loader_errors(tmp_path):
    from nanospec_b200.weights import WeightError, build_model, load_model, write_random_model, write_safetensors
    from nanospec_b200.weights.safetensors_io import SafetensorsFile

    cfg = small_config()
    model, _ = build_model(cfg, None, torch.float32, "cpu")
    specs = model.weight_specs()
    assert specs["l0.norm1"].shape == () and specs["final.norm"].shape == ()
    assert specs["l0.mix.in"].shape == (2 * 30 + 2 * 21 + 6, 20) and specs["l0.mix.conv"].shape == (30 + 42, 3) and specs["l0.mix.conv.b"].shape == (72,)
    assert all(specs[f"l0.mix.{n}"].shape == (6,) for n in ("dt_bias", "A_log", "D")) and specs["l0.mix.norm"].shape == (30,)
    assert specs["l0.mlp.router"].shape == (6, 20) and specs["l0.mlp.correction"].shape == (6,) and "l0.mlp.e4.up" not in specs
    assert specs["l0.mlp.e3.down"].shape == (20, 9) and specs["l0.mlp.shared.gate"].shape == (11, 20)
    assert specs["l1.mix.q.b"].shape == (40,) and specs["l1.mix.v.b"].shape == (12,) and "l1.mix.o.b" not in specs
    assert specs["l1.mix.q.norm"].shape == (40,) and specs["l1.mix.k.norm"].shape == (20,) and specs["l1.mix.o"].shape == (20, 24)
    assert specs["l1.mlp.act"].shape == (2,) and not any(n.startswith("l2.mlp") or ".norm2" in n for n in specs)
    needs = model.lane_needs()
    assert needs[0][0] is None and needs[0][1].shape[0] >= 6 * 7 * 5 + 2 * 72
    assert needs[1][0].window == 5 and needs[1][0].v_dim == 6 and needs[2][0].window == 2 and needs[2][1] is None
    folder = write_random_model(tmp_path / "m", cfg, seed=3)
    with SafetensorsFile(folder / "model.safetensors") as f:
        tensors = {k: f.tensor(k).clone() for k in f.keys()}
    assert set(tensors) == set(specs)
    del tensors["l0.mlp.correction"]
    tensors["l1.mix.o.b"] = torch.zeros(20, dtype=torch.bfloat16)
    tensors["l0.norm1"] = torch.zeros(20, dtype=torch.bfloat16)
    write_safetensors(folder / "model.safetensors", tensors)
    with pytest.raises(WeightError) as err:
        load_model(folder, device="cpu", dtype=torch.float32)
    text = str(err.value)
    assert "l0.mlp.correction" in text and "l1.mix.o.b" in text and "l0.norm1" in text


# ---- the plain statement's own mechanisms: a second, independent writing of each ----------------------------------------

def test_plain_activation_norms_and_window():
    p, q = torch.tensor(0.3, dtype=torch.float64), torch.tensor(-0.6, dtype=torch.float64)
    sp, sq = math.log(1.0 + math.exp(0.3)), math.log(1.0 + math.exp(-0.6))
    z = torch.tensor([-2.0, 0.0, 1.5], dtype=torch.float64)
    want = [(0.5 + sq) * (math.exp(-2.0) - 1.0 + 2.0) - 1.0, 0.0, sp * 2.25 + 0.75]
    assert torch.allclose(plain.xielu(z, p, q), torch.tensor(want, dtype=torch.float64))
    x = torch.tensor([[3.0, 4.0]], dtype=torch.float64)
    assert torch.allclose(plain.rms_norm(x, 0.5, 2.0), x * 2.0 / math.sqrt(13.0))
    y, gate = torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=torch.float64), torch.tensor([[0.5, -1.0, 2.0, 0.1]], dtype=torch.float64)
    u = [a * b / (1.0 + math.exp(-b)) for a, b in zip(y[0].tolist(), gate[0].tolist())]
    g = torch.tensor([1.0, 2.0, 3.0, 4.0], dtype=torch.float64)
    want = [u[i] * float(g[i]) / math.sqrt((u[i // 2 * 2] ** 2 + u[i // 2 * 2 + 1] ** 2) / 2 + 1e-3) for i in range(4)]
    assert torch.allclose(plain.gated_norm(y, gate, 1e-3, g, 2), torch.tensor([want], dtype=torch.float64))
    m = plain.window_mask(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[1].tolist() == [True, True] + [False] * 4


def test_plain_state_walk_is_the_sum_it_stands_for():
    """y_t = sum over s <= t of (product of the decays after s) * step_s * (C_t . B_s) x_s, plus D x_t."""
    g = torch.Generator().manual_seed(0)
    T, H, V, G, N = 7, 4, 3, 2, 5
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    x, B, C, dt, a_log, D = r(T, H, V), r(T, G, N), r(T, G, N), r(T, H).abs(), r(H) * 0.3, r(H)
    y = plain.state_space_walk(x, B, C, dt, a_log, D)
    for h in range(H):
        for t in range(T):
            want = D[h] * x[t, h]
            for s in range(t + 1):
                decay = math.exp(-math.exp(float(a_log[h])) * float(dt[s + 1: t + 1, h].sum()))
                want = want + decay * dt[s, h] * float(C[t, h // 2] @ B[s, h // 2]) * x[s, h]
            assert torch.allclose(y[t, h], want)


def test_plain_routing_rule():
    W = {"router": torch.eye(4, dtype=torch.float64), "correction": torch.tensor([0.0, 0.5, 0.0, 0.0], dtype=torch.float64)}
    h = torch.tensor([[2.0, 0.0, 1.0, -1.0]], dtype=torch.float64)
    s = torch.softmax(h[0], -1)
    chosen, weights = plain.route(h, {"top": 2, "scale": 3.0}, W, "")
    assert sorted(chosen[0].tolist()) == [0, 1]  # expert 2 scores more than 1, whose correction puts it ahead
    assert torch.allclose(weights[0], 3.0 * s[chosen[0]])


def test_plain_forward_is_causal_and_uses_every_mechanism():
    """A later token never moves an earlier position, and taking a mechanism away moves the logits."""
    cfg = small_config()
    from nanospec_b200.weights import build_model

    model, _ = build_model(cfg, None, torch.float32, "cpu")
    g = torch.Generator().manual_seed(4)
    w = {n: (torch.randn(s.shape, generator=g) * (0.4 if len(s.shape) == 2 else 1.0)).to(torch.bfloat16).float() for n, s in sorted(model.weight_specs().items())}
    ids = torch.randint(0, 53, (14,), generator=g).tolist()
    z = plain.forward(cfg, w, ids)
    assert z.shape == (14, 53) and torch.isfinite(z).all()
    other = list(ids)
    other[9] = (other[9] + 1) % 53
    z2 = plain.forward(cfg, w, other)
    assert torch.equal(z2[:9], z[:9]) and not torch.allclose(z2[9:], z[9:])

    def without(change):
        c = copy.deepcopy(cfg)
        change(c)
        return float((plain.forward(c, w, ids) - z).abs().max())

    assert without(lambda c: c["layers"][1]["mixer"]["mask"].update(size=6)) > 1e-6
    assert without(lambda c: c["layers"][1]["mixer"].update(scale=0.41)) > 1e-6
    assert without(lambda c: c["layers"][0]["mixer"].update(norm_groups=3)) > 1e-6
    assert without(lambda c: c["layers"][0]["mlp"]["router"].update(scale=1.6)) > 1e-6
    assert without(lambda c: c["layers"][0]["mlp"].update(shared=None)) > 1e-6
    for name in ("l0.mix.D", "l0.mix.A_log", "l0.mix.conv.b", "l0.mix.dt_bias", "l0.mlp.correction", "l1.mix.q.b", "l1.mix.v.b", "l1.mix.k.norm",
                 "l1.mlp.act", "l2.norm1"):
        lost = dict(w)
        lost[name] = torch.zeros_like(w[name]) if "norm1" not in name else w[name] * 0.5
        assert float((plain.forward(cfg, lost, ids) - z).abs().max()) > 1e-6, name
