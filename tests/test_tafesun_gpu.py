"""The Tafesun parts on the GPU against the plain statement in plain_tafesun.py: each kernel and each mechanism alone, whole prompts
against token-by-token decoding, portions down to two tokens, unequal batches, pages and state slots that are used again, keys far away
and at page borders, a token far back seen through the state alone, the first tokens, long decoding, sizes that differ everywhere (also
those that the tensor-core kernels take), and greedy generation through the engine.  Each test makes its own small configuration and
weights."""

from __future__ import annotations

import copy
import json
import math
from types import SimpleNamespace

import pytest
import torch

import plain_tafesun as plain

pytestmark = pytest.mark.gpu

F32, BF16 = torch.float32, torch.bfloat16
BOTH = pytest.mark.parametrize("dtype", [F32, BF16], ids=["float32", "bfloat16"])


# ---- configurations ---------------------------------------------------------------------------------------------------

def moe(experts=5, top=3, ff=24, limit=1.1, shared=32, shared_limit=0.7):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared, "limit": shared_limit}
    return out


def left(heads=4, kv_heads=2, dim=8, vdim=12, scale=None, dims=4, base=300.0, factor=1.5):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5,
            "rot": {"dims": dims, "base": base, "scaling": {"factor": factor}}}


def right(heads=4, vdim=6, state=8, groups=2, conv=3, norm_groups=2):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def layer(a=None, s=None, mlp=None, left_scale=0.7, right_scale=1.2, **kw):
    return {"type": "parallel", "mixer": {"left": a or left(), "right": s or right(), "left_scale": left_scale, "right_scale": right_scale}, "mlp": mlp, **kw}


def config(layers, width=40, vocab=89, eps=1e-5, logit_scale=0.5):
    return {"architecture": "Tafesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


def full_config(**kw):
    """Sizes that differ from layer to layer, layers with and without a feed-forward, two that use another's tensors."""
    layers = [layer(left(heads=6, kv_heads=2, dim=12, vdim=10, dims=8), right(heads=6, vdim=8, state=16, groups=3, conv=4, norm_groups=4), moe(shared=40)),
              layer(left(heads=2, kv_heads=2, dim=16, vdim=24, dims=16, factor=3.0), right(heads=3, vdim=10, state=5, groups=1, conv=2, norm_groups=5), None,
                    left_scale=1.0, right_scale=-0.4),
              layer(left(heads=5, kv_heads=1, dim=6, vdim=6, dims=0), right(heads=2, vdim=8, state=24, groups=2, conv=1, norm_groups=1),
                    moe(experts=3, top=1, ff=16, limit=0.4, shared=None), left_scale=2.0, right_scale=1.0)]
    layers += [dict(copy.deepcopy(layers[0]), weights_of=0), dict(copy.deepcopy(layers[1]), weights_of=1)]
    return config(layers, **kw)


def routed(cfg):
    return any(entry["mlp"] for entry in cfg["layers"])


def random_weights(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """Names and shapes from the framework's own list, values from here, bfloat16-representable."""
    from nanospec_b200.weights import build_model

    model, _ = build_model(cfg, None, F32, "cpu")
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, spec in sorted(model.weight_specs().items()):
        if name == "head":
            continue  # the embedding's table
        t = torch.randn(spec.shape, generator=g)
        leaf = name.split(".")[-1]
        if leaf == "conv":
            t = 0.6 * t
        elif leaf == "router":
            t = t * (2.0 / math.sqrt(spec.shape[1]))
        elif leaf == "embed":
            pass
        elif len(spec.shape) == 2:
            t = t * (1.5 / math.sqrt(spec.shape[1]))
        elif leaf == "alpha":
            t = 0.8 + 0.2 * t
        elif leaf in ("norm", "norm1", "norm1b", "norm2", "norm2b", "D"):
            t = 1.0 + 0.2 * t
        elif leaf == "b":
            t = 0.3 * t
        elif leaf == "dt_bias":
            t = 0.5 * t - 1.0
        elif leaf == "A_log":
            t = 0.7 * t - 1.5  # decays from a few tokens to hundreds
        out[name] = t.to(BF16).float()
    return out


def write_folder(folder, cfg, weights):
    from nanospec_b200.weights import write_safetensors

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(folder / "model.safetensors", {k: v.to(BF16) for k, v in weights.items()})
    return folder


def make(tmp_path, cfg, seed=0, dtype=F32, blocks=64, page=4, slots=4, weights=None):
    from nanospec_b200 import load_model
    from nanospec_b200.engine.step import ModelRunner

    w = weights if weights is not None else random_weights(cfg, seed)
    model = load_model(write_folder(tmp_path / f"m{seed}{'f' if dtype == F32 else 'b'}", cfg, w), device="cuda", dtype=dtype)
    return ModelRunner(model, num_blocks=blocks, block_size=page, max_requests=slots), w


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_cut(runner, req_id, ids, cuts):
    """One request alone, its tokens in portions of the given sizes (the rest one by one); logits of every position."""
    from nanospec_b200.engine.step import StepEntry

    runner.begin(req_id)
    rows, at, sizes = [], 0, list(cuts)
    while at < len(ids):
        n = min(sizes.pop(0) if sizes else 1, len(ids) - at)
        rows.append(runner.step([StepEntry(req_id, ids[at: at + n], list(range(n)))]).float().cpu())
        at += n
    runner.end(req_id)
    runner.manager.check()
    return torch.cat(rows)


def distance(got, want):
    """Per position: root mean square over the vocabulary of the difference, the mean taken off, over the logits' spread."""
    d = got.double() - want.double()
    return (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().std()


def rounding(cfg, w, ids, want, samples=3):
    """Per position: how far bfloat16 storage of the activations alone moves the plain logits: the largest of the rounding
    itself and of `samples` draws of a relative error of that size on every stored activation."""
    worst = distance(plain.forward(cfg, w, ids, rounded=BF16), want)
    for seed in range(samples):
        g = torch.Generator().manual_seed(seed)
        draw = lambda t: t * (1.0 + (torch.rand(t.shape, generator=g, dtype=t.dtype) - 0.5) * 2.0 ** -7)
        worst = torch.maximum(worst, distance(plain.forward(cfg, w, ids, rounded=draw), want))
    return worst


def close(got, want, dtype, what="", noise=None, experts=True):
    """float32: a few roundings against the logits' spread at every position.  bfloat16: small at the median position, and at
    every position within a few times of what rounding alone does there (`noise`, from `rounding`), never of the size that a
    wrong mask, a lost state or a wrong page gives elsewhere.  `experts`: two experts that nearly tie can change places under
    bfloat16 rounding and take a token's output with them, so one position in ten may leave the limit."""
    r = distance(got, want)
    if dtype == F32:
        assert float(r.max()) <= 2e-4, f"{what}: {float(r.max())} at position {int(r.argmax())} (limit 2e-4)"
        return
    noise = torch.zeros_like(r) if noise is None else noise[: len(r)]
    median, typical = float(r.median()), float(noise.median())
    assert median <= max(0.06, 3 * typical) or len(r) < 8, f"{what}: {median:.3f} at the median position (rounding alone: {typical:.3f})"
    over = r - torch.maximum(torch.full_like(r, 0.25), 4 * noise)
    allowed = max(1, len(r) // 10) if experts else 0
    assert int((over > 0).sum()) <= allowed, f"{what}: {float(r[over.argmax()]):.3f} at position {int(over.argmax())} (rounding alone: {float(noise[over.argmax()]):.3f})"


# ---- the kernels alone ----------------------------------------------------------------------------------------------------

@BOTH
@pytest.mark.parametrize("hidden", [40, 2056, 37])
def test_the_norm_on_a_branch_and_the_norm_after_it(hidden, dtype):
    """A branch, a pair, a routed sum with and without a rest: the stream takes the normed branch, the next norm reads the sum; with
    selected rows the stream stays; without a next norm only the stream moves."""
    from nanospec_b200 import ops

    g = torch.Generator().manual_seed(hidden)
    N, top = 7, 3
    W = {}
    for name in ("p", "n"):
        W[name], W[name + ".b"], W[name + ".alpha"] = 1 + torch.randn(hidden, generator=g), torch.randn(hidden, generator=g), torch.tensor(0.7 if name == "p" else 0.4)
    norms = {k: ops.TanhNorm(W[k].cuda(), W[k + ".b"].cuda(), W[k + ".alpha"].reshape(1).cuda()) for k in ("p", "n")}
    Wd = {k: v.double() for k, v in W.items()}
    x = torch.randn(N, hidden, generator=g) * 2
    a, b = (torch.randn(N, hidden, generator=g).to(dtype) for _ in range(2))
    ys = torch.randn(N * top, hidden, generator=g).to(dtype)
    rows = torch.randperm(N * top, generator=g).int().view(N, top)
    weights = torch.rand(N, top, generator=g)
    sums = (weights[:, :, None].double() * ys.double()[rows.long()]).sum(1)
    cases = [(a.cuda(), a.double()), ((a.cuda(), b.cuda()), a.double() + b.double()),
             (ops.RoutedSum(ys.cuda(), rows.cuda(), weights.cuda()), sums), (ops.RoutedSum(ys.cuda(), rows.cuda(), weights.cuda(), b.cuda()), sums + b.double())]
    pick = torch.tensor([5, 0, 5], dtype=torch.int32)
    for branch, y in cases:
        want = x.double() + plain.dynamic_tanh(y, Wd, "p")
        out_want = plain.dynamic_tanh(want, Wd, "n")
        tol = 2e-6 if dtype == F32 else 1e-2
        resid = x.cuda()
        out = ops.dyt_join(resid, branch, norms["p"], norms["n"], torch.empty(N, hidden, dtype=dtype, device="cuda"))
        assert (resid.cpu() - want).abs().max() <= 4e-6 and (out.cpu().double() - out_want).abs().max() <= tol * (1 + out_want.abs().max())
        resid = x.cuda()
        assert ops.dyt_join(resid, branch, norms["p"]) is None and (resid.cpu() - want).abs().max() <= 4e-6
        resid = x.cuda()
        got = ops.dyt_join(resid, branch, norms["p"], norms["n"], torch.empty(3, hidden, dtype=dtype, device="cuda"), rows=pick.cuda())
        assert torch.equal(got, out[pick.long().cuda()]) and torch.equal(resid.cpu(), x)


@pytest.mark.parametrize("dtype", [F32, BF16], ids=["float32", "bfloat16"])
def test_tanh_over_its_range(dtype):
    """The norm's tanh on the stream (float32 in both types): tiny arguments, both sides of where its two forms meet, saturation."""
    from nanospec_b200 import ops

    a = torch.cat([torch.logspace(-6, 3, 3000), torch.linspace(0.2, 0.3, 1000), torch.zeros(96)])
    x = torch.cat([a, -a]).view(1, -1).contiguous()
    norm = ops.TanhNorm(torch.ones(x.shape[1]).cuda(), None, torch.ones(1).cuda())
    want = torch.tanh(x.to(dtype).double())
    resid = torch.zeros_like(x).cuda()
    ops.dyt_join(resid, x.to(dtype).cuda(), norm)
    err = (resid.cpu().double() - want).abs()
    assert float(err.max()) <= 4e-7 and float((err / want.abs().clamp(min=1e-30)).max()) <= 2e-6


def test_gated_units_in_every_kernel_that_runs_them():
    """g held below the limit, u within it, g sigmoid(alpha g) (u + shift): the activation kernel (contiguous and column ranges, both
    layouts), and the tcgen05 product of a short step; a limit that few inputs reach and one that most do."""
    from nanospec_b200 import ops

    g = torch.Generator().manual_seed(3)

    def ref(gate, up, unit):
        gate, up = gate.double(), up.double()
        if unit.limit:
            gate, up = gate.clamp(max=unit.limit), up.clamp(-unit.limit, unit.limit)
        return gate / (1 + torch.exp(-unit.alpha * gate)) * (up + unit.shift)

    for unit in (ops.GatedUnit(1.702, 1.0, 2.0), ops.GatedUnit(1.702, 1.0, 0.3), ops.GatedUnit(0.9, -0.4, 0.0)):
        for inter, block in ((64, 0), (128, 64), (12, 0), (7, 0)):
            for dtype in (F32, BF16):
                rows = (2 * torch.randn(6, 2 * inter + 24, generator=g)).to(dtype).cuda()
                gu = rows[:, 16: 16 + 2 * inter]
                parts = gu.view(6, -1) if block == 0 else gu.reshape(6, inter // block, 2, block).transpose(1, 2).reshape(6, 2 * inter)
                want = ref(parts[:, :inter].cpu(), parts[:, inter:].cpu(), unit)
                out = torch.zeros(6, inter + 8, dtype=dtype, device="cuda")
                ops.swiglu(gu, out[:, :inter], block, unit)
                tol = 2e-6 if dtype == F32 else 1e-2
                assert (out[:, :inter].cpu().double() - want).abs().max() <= tol * (1 + want.abs().max()) and not out[:, inter:].any()
                assert torch.equal(ops.swiglu(gu.contiguous(), torch.empty(6, inter, dtype=dtype, device="cuda"), block, unit), out[:, :inter])
        for M, K, inter in ((5, 72, 64), (33, 128, 192), (64, 520, 128)):
            x, wg, wu = torch.randn(M, K, generator=g).to(BF16), *((torch.randn(inter, K, generator=g) * 2 / math.sqrt(K)).to(BF16) for _ in range(2))
            packed = torch.stack([wg.view(-1, 64, K), wu.view(-1, 64, K)], dim=1).reshape(2 * inter, K).contiguous()
            out = ops.gated_linear(x.cuda(), packed.cuda(), torch.empty(M, inter, dtype=BF16, device="cuda"), torch.empty(M, 2 * inter, dtype=BF16, device="cuda"), 64, unit)
            want = ref(x.double() @ wg.double().T, x.double() @ wu.double().T, unit)
            assert (out.cpu().double() - want).abs().max() <= 1e-2 * (1 + want.abs().max())


@pytest.mark.parametrize("kernel,ff", [("tcgen05", 64), ("m16n8k16", 24), ("rows", 10)])
def test_experts_with_clamped_units(kernel, ff):
    """The three kernels that run routed experts without the host, with units of their own, against the plain expert."""
    from nanospec_b200 import ops

    g = torch.Generator().manual_seed(ff)
    E, top, N, width, limit = 4, 2, 50, 72, 0.8
    dtype = F32 if kernel == "rows" else BF16
    x = torch.randn(N, width, generator=g).to(dtype)
    w = {f"e{e}.{n}": (torch.randn((ff, width) if n != "down" else (width, ff), generator=g) * 2 / math.sqrt(width if n != "down" else ff)).to(dtype)
         for e in range(E) for n in ("gate", "up", "down")}
    wg, wu, wd = (torch.stack([w[f"e{e}.{n}"] for e in range(E)]).contiguous() for n in ("gate", "up", "down"))
    unit = ops.GatedUnit(1.702, 1.0, limit)
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(N)]).int()
    weights = torch.rand(N, top, generator=g)
    wide = {k: v.double() for k, v in w.items()}
    want = torch.stack([sum(weights[t, k].double() * plain.expert(x[t: t + 1].double(), wide, f"e{int(ids[t, k])}.", limit)[0] for k in range(top)) for t in range(N)])
    buf = lambda cols, rows=N * top: torch.full((rows, cols), float("nan"), dtype=dtype, device="cuda")
    if kernel == "rows":
        got = ops.moe_expert_rows(x.cuda(), ids.cuda(), weights.cuda(), wg.cuda(), wu.cuda(), wd.cuda(), buf(ff), buf(width, N), unit)
    else:
        offsets, row_of = torch.empty(E + 1, dtype=torch.int32, device="cuda"), torch.empty(N, top, dtype=torch.int32, device="cuda")
        pair_of = torch.empty(N, top, dtype=torch.int32, device="cuda")
        ops.moe_plan(ids.cuda(), E, offsets, row_of, pair_of)
        if kernel == "tcgen05":
            packed = torch.stack([wg.view(E, ff // 64, 64, width), wu.view(E, ff // 64, 64, width)], dim=2).reshape(E, 2 * ff, width).contiguous()
            ys = ops.moe_grouped_tc(ops.moe_gather(x.cuda(), row_of, buf(width), top), offsets, packed.cuda(), wd.cuda(), buf(ff), buf(width), unit)
        else:
            ys = ops.moe_grouped(x.cuda(), pair_of, offsets, wg.cuda(), wu.cuda(), wd.cuda(), buf(ff), buf(width), top, unit)
        got = ops.moe_combine(ys, row_of, weights.cuda(), buf(width, N), top)
    ops.check_kernel_errors()
    assert (got.cpu().double() - want).abs().max() <= (1e-5 if dtype == F32 else 0.03) * (1 + want.abs().max())


@pytest.mark.parametrize("E,top,N,K", [(5, 3, 9, 40), (60, 6, 200, 64), (1, 1, 5, 33), (40, 36, 4, 24), (12, 12, 600, 16)])
def test_routing_by_biased_logits(E, top, N, K):
    """Bias in the router's product; the largest logits choose, their softmax among themselves weighs - also where a softmax over all would
    have nothing left for the chosen but the first."""
    from nanospec_b200 import ops

    g = torch.Generator().manual_seed(E)
    x, router, bias = torch.randn(N, K, generator=g), torch.randn(E, K, generator=g), torch.randn(E, generator=g)
    if E > 4:
        bias[2] += 130.0  # far ahead of every other
    for dtype in (F32, BF16):
        xd = x.to(dtype)
        want_ids, want_w = plain.route(xd.double(), {"top": top}, {"router": router.double(), "router.b": bias.double()}, "")
        z = ops.router_logits(xd.cuda(), router.cuda(), torch.empty(N, E, device="cuda"), bias=bias.cuda())
        assert (z.cpu() - (xd.double() @ router.double().T + bias)).abs().max() <= 2e-5 * (K ** 0.5 + 130)
        ids, weights = torch.empty(N, top, dtype=torch.int32, device="cuda"), torch.empty(N, top, device="cuda")
        ops.moe_route(z, 1, 1, top, 1.0, ids, weights, ops.ROUTE_CHOSEN)
        assert torch.equal(ids.cpu().long(), want_ids) and (weights.cpu() - want_w).abs().max() <= 1e-4
        assert (weights.sum(-1).cpu() - 1).abs().max() <= 1e-5
        if ops.route_plan_ok(N, E):
            ids2, w2 = torch.empty_like(ids), torch.empty_like(weights)
            offsets = torch.empty(E + 1, dtype=torch.int32, device="cuda")
            row_of, pair_of = (torch.empty(N, top, dtype=torch.int32, device="cuda") for _ in range(2))
            ops.moe_route_plan(z, 1, 1, top, 1.0, ids2, w2, ops.ROUTE_CHOSEN, None, True, E, offsets, row_of, pair_of)
            assert torch.equal(ids, ids2) and torch.equal(weights, w2) and int(offsets[-1]) == N * top


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 16, 24), (6, 2, 128, 256), (2, 1, 8, 136), (6, 3, 64, 64), (2, 2, 40, 264), (34, 2, 16, 16), (3, 1, 10, 14), (2, 1, 24, 500)])
@BOTH
def test_attention_with_a_gate_per_feature_and_wide_values(H, G, d, dv, dtype):
    """Prompt portions and single tokens over scattered pages, values of any width (in slices where they are wide), the sigmoid of a gate per
    feature and a constant factor on the output, gates in a wider buffer; keys scaled so that one score stands out at a page's border."""
    from nanospec_b200 import ops
    from nanospec_b200.parts.context import Workspace

    g = torch.Generator().manual_seed(d + dv)
    page, lens, news = 4, [150, 9, 131], [30, 1, 1]
    table = torch.randperm(90, generator=g).int()[: 3 * 40].view(-1)
    pages, at, bt = [-(-n // page) for n in lens], 0, torch.zeros(3, 40, dtype=torch.int32)
    for b, n in enumerate(pages):
        bt[b, :n] = table[at: at + n]
        at += n
    kc, vc = torch.randn(90, G, page, d, generator=g).to(dtype), torch.randn(90, G, page, dv, generator=g).to(dtype)
    N = sum(news)
    wide = torch.randn(N, H * d + 8 + H * dv + 8, generator=g)
    gates = (wide[:, H * d + 8: H * d + 8 + H * dv]).to(dtype)
    token_req = torch.tensor([b for b, n in enumerate(news) for _ in range(n)], dtype=torch.int32)
    positions = torch.tensor([lens[b] - n + i for b, n in enumerate(news) for i in range(n)], dtype=torch.int32)
    for b in range(3):  # the first key of the second page points where the request's last query points
        row = int((token_req == b).nonzero()[-1])
        for k in range(G):
            kc[bt[b, 1], k, 0] = (2.0 * wide[row, (k * (H // G)) * d: (k * (H // G) + 1) * d]).to(dtype)
    buf = wide.to(dtype).cuda()
    ctx = SimpleNamespace(token_req=token_req.cuda(), positions=positions.cuda(), qo_indptr=torch.tensor([0, 30, 31, 32], dtype=torch.int32).cuda(),
                          extras={}, q_lens=news, kv_lens=lens, n_tokens=N, device=torch.device("cuda"), workspace=Workspace(torch.device("cuda")))
    lane = SimpleNamespace(k=kc.cuda(), v=vc.cuda(), block_table=bt.cuda(), page_size=page)
    out = torch.zeros(N, H * dv + 16, dtype=dtype, device="cuda")
    scale, factor = d ** -0.5, 0.8
    ops.attention(buf, lane, ctx, out[:, 8: 8 + H * dv], H, G, d, scale, v_dim=dv, wide_weights=True,
                  gate=buf[:, H * d + 8: H * d + 8 + H * dv], feature_gate=True, out_scale=factor)
    assert not out[:, :8].any() and not out[:, 8 + H * dv:].any()
    for n in range(N):
        b, p = int(token_req[n]), int(positions[n])
        slots = [(int(bt[b, j // page]), j % page) for j in range(p + 1)]
        for h in range(H):
            k = torch.stack([kc[pg, h // (H // G), o] for pg, o in slots]).double()
            v = torch.stack([vc[pg, h // (H // G), o] for pg, o in slots]).double()
            want = torch.softmax(k @ buf[n, h * d: (h + 1) * d].cpu().double() * scale, 0) @ v * plain.sigmoid(gates[n, h * dv: (h + 1) * dv].double()) * factor
            got = out[n, 8 + h * dv: 8 + (h + 1) * dv].cpu().double()
            assert (got - want).abs().max() <= (1e-5 if dtype == F32 else 2e-2) * (1 + want.abs().max()), (n, h)


@pytest.mark.parametrize("M,N,K", [(1, 128, 64), (17, 256, 200), (64, 384, 1032)])
def test_both_norms_in_the_product(M, N, K):
    """The tcgen05 product whose epilogue norms the product, adds it to the stream and norms the sum."""
    from nanospec_b200 import ops
    from nanospec_b200.parts.context import Workspace

    g = torch.Generator().manual_seed(N)
    x, w = torch.randn(M, K, generator=g).to(BF16), (torch.randn(N, K, generator=g) / math.sqrt(K)).to(BF16)
    resid = torch.randn(M, N, generator=g)
    W = {n + s: torch.randn(N, generator=g) if s != ".alpha" else torch.tensor(0.6 if n == "p" else 1.3) for n in ("p", "n") for s in ("", ".b", ".alpha")}
    t = {k: v.reshape(-1).cuda() for k, v in W.items()}
    sink = ops.TanhSink(resid.cuda(), t["n"], t["n.b"], t["n.alpha"], Workspace(torch.device("cuda")), ops.TanhNorm(t["p"], t["p.b"], t["p.alpha"]))
    got = ops.linear(x.cuda(), w.cuda(), torch.empty(M, N, dtype=BF16, device="cuda"), sink=sink)
    assert isinstance(got, ops.Normed)
    Wd = {k: v.double() for k, v in W.items()}
    want = resid.double() + plain.dynamic_tanh(x.double() @ w.double().T, Wd, "p")
    assert (sink.resid.cpu() - want).abs().max() <= 2e-5
    want = plain.dynamic_tanh(want, Wd, "n")
    assert (got.x.cpu().double() - want).abs().max() <= 1e-2 * want.abs().max()


# ---- mechanisms as models of their own ------------------------------------------------------------------------------------

SINGLE = {
    "attention alone": lambda: config([layer(left(heads=4, kv_heads=1, vdim=20), None, None, right_scale=0.0)]),
    "state space alone": lambda: config([layer(None, right(heads=6, groups=3, conv=5), None, left_scale=0.0)]),
    "both, no feed-forward": lambda: config([layer(), layer(left(dim=16, vdim=8), right(vdim=8, state=20))]),
    "one head, one key head": lambda: config([layer(left(heads=1, kv_heads=1, dim=2, vdim=2, dims=2), right(heads=1, groups=1, vdim=1, state=1, conv=1, norm_groups=1), moe())]),
    "heads that do not turn": lambda: config([layer(left(dims=0), None, moe(experts=1, top=1))]),
    "heads that turn whole": lambda: config([layer(left(dim=16, dims=16, base=50.0, factor=0.5), None, None)]),
    "a shared expert alone beside one": lambda: config([layer(None, None, moe(experts=1, top=1, shared=16, shared_limit=0.2))]),
    "every expert chosen": lambda: config([layer(None, None, moe(experts=4, top=4, ff=8, limit=0.3))]),
    "no shared expert": lambda: config([layer(None, None, moe(shared=None, limit=5.0)), layer(None, None, moe(shared=None, top=1))]),
    "one layer run three times": lambda: config([layer(None, None, moe()), layer(None, None, moe(), weights_of=0), layer(None, None, moe(), weights_of=1)]),
    "odd widths": lambda: config([layer(left(heads=3, kv_heads=3, dim=6, vdim=5, dims=2), right(heads=3, vdim=7, state=3, groups=1, norm_groups=3), moe(ff=9, shared=13))], width=37),
    "expert widths of 64": lambda: config([layer(None, None, moe(ff=64, shared=64))], width=64),
    "norm parts of one feature": lambda: config([layer(None, right(heads=2, vdim=3, groups=1, norm_groups=6), None)]),
    "a negative scale": lambda: config([layer(left_scale=-1.1, right_scale=0.9, mlp=moe())], logit_scale=2.0),
}


@BOTH
@pytest.mark.parametrize("name", list(SINGLE))
def test_each_mechanism(name, dtype, tmp_path):
    """Whole, token by token and in portions (down to two tokens), against the plain statement."""
    cfg = SINGLE[name]()
    runner, w = make(tmp_path, cfg, seed=len(name), dtype=dtype)
    ids = tokens(37, cfg["vocab"], 5)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want) if dtype == BF16 else None
    for cuts in ([37], [], [2, 3, 2, 11, 5, 2], [20, 1, 1, 15]):
        close(run_cut(runner, 0, ids, cuts), want, dtype, f"{name}, portions {cuts or 'of one'}", noise, routed(cfg))


def test_layers_one_by_one(tmp_path):
    """The stream after every layer, in float32, against the plain statement's."""
    from nanospec_b200.engine.step import StepEntry
    from nanospec_b200.parts.norm import PostNormed

    cfg = full_config()
    runner, w = make(tmp_path, cfg, seed=3)
    ids = tokens(29, cfg["vocab"], 8)
    want, got = [], []
    plain.forward(cfg, w, ids, layers_out=want)

    def probe(i, resid, pending):
        x = resid.clone()
        if isinstance(pending, PostNormed):  # what the next norm's kernel will add
            pending.settle(x)
        got.append(x.cpu().double())

    runner.begin(0)
    ctx, rows, _ = runner.build_context([StepEntry(0, ids, [])])
    ctx.extras["probe"] = probe
    runner.forward(ctx, rows)
    runner.end(0)
    assert len(got) == len(want) == 5
    for i, (a, b) in enumerate(zip(got, want)):
        assert (a - b).abs().max() <= 2e-5 * float(b.abs().max()), f"layer {i}: {float((a - b).abs().max())}"


@BOTH
def test_what_could_be_lost(dtype, tmp_path):
    """Lost biases, gates, a lost tap, skip, norm, shared or routed expert, another rotation factor, scale or limit: each moves the plain logits by
    far more than the engine differs from the right ones - in a prompt, in portions and token by token."""
    cfg = config([layer(left(dim=16, vdim=24, heads=4, kv_heads=2, dims=8, factor=2.0, scale=0.6), right(vdim=8, state=16, conv=3), moe(ff=16, shared=24, limit=0.6))])
    w = random_weights(cfg, 14)
    w["l0.mlp.router.b"] = (w["l0.mlp.router.b"] * 4).to(BF16).float()
    runner, w = make(tmp_path, cfg, seed=14, dtype=dtype, page=4, weights=w)
    ids = tokens(45, cfg["vocab"], 17)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want)
    calm = noise <= 0.05  # bfloat16: the variants are told apart at the positions that rounding leaves alone
    wrong = {}
    for name in ("l0.mix.left.q.b", "l0.mix.left.v.b", "l0.mix.left.g", "l0.mix.right.D", "l0.mix.right.conv.b", "l0.mix.right.dt_bias", "l0.mlp.shared.down",
                 "l0.mlp.e0.down", "l0.mlp.router.b", "l0.norm1.b", "l0.norm1b.b", "l0.norm2.b", "l0.norm2b.b", "final.norm.b"):
        wrong[name] = plain.forward(cfg, {**w, name: torch.zeros_like(w[name])}, ids)
    for name in ("l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "final.norm"):
        wrong[name + ".alpha"] = plain.forward(cfg, {**w, name + ".alpha": torch.ones(()) * 2.0}, ids)
    tap = w["l0.mix.right.conv"].clone()
    tap[:, 0] = 0.0
    wrong["the tap two tokens back"] = plain.forward(cfg, {**w, "l0.mix.right.conv": tap}, ids)
    for what, change in {"factor": lambda c: c["mixer"]["left"]["rot"]["scaling"].update(factor=1.0), "left_scale": lambda c: c["mixer"].update(left_scale=1.0),
                         "right_scale": lambda c: c["mixer"].update(right_scale=1.0), "limit": lambda c: c["mlp"]["expert"].update(limit=50.0),
                         "shared limit": lambda c: c["mlp"]["shared"].update(limit=0.6), "norm_groups": lambda c: c["mixer"]["right"].update(norm_groups=1),
                         "scale": lambda c: c["mixer"]["left"].update(scale=0.25)}.items():
        other = copy.deepcopy(cfg)
        change(other["layers"][0])
        wrong[what] = plain.forward(other, w, ids)
    for cuts in ([45], [], [2, 3, 2, 11, 5, 2]):
        got = run_cut(runner, 0, ids, cuts)
        close(got, want, dtype, f"portions {cuts or 'of one'}", noise)
        keepers = torch.ones_like(calm) if dtype == F32 else calm
        right_one = float(distance(got, want)[keepers].quantile(0.9))
        for what, z in wrong.items():
            off = float(distance(got, z)[keepers].max())
            assert off > (10 if dtype == F32 else 2) * right_one and off > 0.03, f"{what} is not told apart: {off} against {right_one}"


# ---- keys and tokens far back ---------------------------------------------------------------------------------------------

def far_key_case():
    """One layer whose state forgets within a few tokens and whose query map is the key map with the halves of its input swapped: tokens B have
    the embeddings of tokens A with the halves swapped, so a B's query points where its A's key points and that one score stands out.  The
    A's sit on the first and the last slot of a page and in its middle; the B's hundreds of positions on."""
    width, dim, n = 64, 16, 420
    cfg = config([layer(left(heads=4, kv_heads=2, dim=dim, vdim=24, dims=0, scale=2.5), right(vdim=8, conv=2), None, left_scale=4.0, right_scale=0.3)], width=width, vocab=80)
    w = random_weights(cfg, 24)
    w["l0.mix.right.A_log"], w["l0.mix.right.dt_bias"] = torch.full((4,), 2.0), torch.full((4,), 2.0)
    w["l0.mix.left.q"] = torch.roll(w["l0.mix.left.k"], width // 2, dims=1).view(2, 1, dim, width).expand(2, 2, dim, width).reshape(4 * dim, width).clone()
    w["l0.mix.left.q.b"], w["l0.mix.left.k.b"] = torch.zeros(4 * dim), torch.zeros(2 * dim)
    w["l0.norm1"], w["l0.norm1.b"] = torch.ones(width), torch.zeros(width)
    w["embed"][:70] *= 0.5
    for i in range(4):
        w["embed"][70 + i] *= 2.0
        w["embed"][74 + i] = torch.roll(w["embed"][70 + i], width // 2)
    w = {k: v.to(BF16).float() for k, v in w.items()}
    ids = [t % 70 for t in tokens(n, 80, 25)]
    pairs = [(0, 300), (15, 401), (16, 417), (39, 419)]
    for i, (a, b) in enumerate(pairs):
        ids[a], ids[b] = 70 + i, 74 + i
    return cfg, w, ids, pairs


@BOTH
def test_keys_far_away_and_at_page_borders(dtype, tmp_path):
    cfg, w, ids, pairs = far_key_case()
    runner, w = make(tmp_path, cfg, seed=24, dtype=dtype, page=16, blocks=40, weights=w)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want, samples=1)
    lost = {}
    for a, b in pairs:
        other = list(ids)
        other[a] = 3
        lost[b] = plain.forward(cfg, w, other)[b]
        assert float(distance(lost[b][None], want[b][None])[0]) > 0.15, (a, b)
    for cuts in ([420], [400], [299, 2, 100, 2, 14, 2], [16] * 25, [290] + [1] * 10 + [100]):
        got = run_cut(runner, 0, ids, cuts)
        close(got, want, dtype, f"portions {cuts[:5]}", noise, False)
        for _, b in pairs:
            assert float(distance(got[b][None], want[b][None])[0]) < 0.25 * float(distance(got[b][None], lost[b][None])[0]), (cuts[:5], b)


def far_token_case():
    """One layer that mixes through the state alone, with slow decays and one token whose trace is the largest: token 48's embedding points
    where every head's step size grows, and where no other token's does."""
    cfg = config([layer(None, right(heads=4, vdim=8, state=16, groups=2, conv=4, norm_groups=2), None, left_scale=0.0, right_scale=4.0)], width=64, vocab=50)
    w = random_weights(cfg, 41)
    p = "l0.mix.right."
    w[p + "A_log"], w[p + "dt_bias"], w[p + "D"] = torch.full((4,), -6.0), torch.full((4,), -5.0), torch.zeros(4)
    w["embed"][:, 0], w[p + "in"][:, 0], w["l0.norm1"], w["l0.norm1.b"] = 0.0, 0.0, torch.ones(64), torch.zeros(64)
    w[p + "in"][-4:] = 0.0
    w[p + "in"][-4:, 0] = 12.0
    w["embed"][48, 0] = 8.0
    w = {k: v.to(BF16).float() for k, v in w.items()}
    ids = tokens(450, 48, 42)
    ids[31] = 48          # the last position of the second page of 16
    lost = list(ids)
    lost[31] = 47
    return cfg, w, ids, lost


@BOTH
def test_a_token_far_back_through_the_state(dtype, tmp_path):
    """A state that had lost one token 418 positions back would answer otherwise - in a whole prompt, as decoded tokens and in portions."""
    cfg, w, ids, lost = far_token_case()
    runner, w = make(tmp_path, cfg, seed=41, dtype=dtype, page=16, blocks=40, weights=w)
    want = plain.forward(cfg, w, ids)
    assert float(distance(plain.forward(cfg, w, lost)[-1:], want[-1:]).max()) > 0.3
    for cuts in ([450], [430], [200, 100, 2, 140]):
        got = run_cut(runner, 0, ids, cuts)
        assert float(distance(got[-1:], want[-1:]).max()) <= (2e-4 if dtype == F32 else 0.1), cuts


@BOTH
@pytest.mark.parametrize("least", [2, 1 << 30], ids=["in chunks", "token by token"])
def test_the_logits_do_not_depend_on_the_cut(least, dtype, tmp_path, monkeypatch):
    """Portions that begin and end inside the state's chunks, on their edges and one beside them, the state walked in chunks and token by token."""
    from nanospec_b200 import ops

    monkeypatch.setattr(ops, "SSM_CHUNKED_MIN", least)
    cfg = config([layer(left(dim=16, vdim=8), right(heads=4, vdim=12, state=24, groups=2, conv=4), moe(ff=16)), layer(left(heads=2, kv_heads=1), right(heads=6, vdim=5, state=7, groups=3))])
    runner, w = make(tmp_path, cfg, seed=58, dtype=dtype, page=16, blocks=40)
    ids = tokens(260, cfg["vocab"], 59)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want, samples=1) if dtype == BF16 else None
    for cuts in ([260], [64, 64, 65, 63], [2, 127, 1, 2, 66], [100, 3, 100]):
        close(run_cut(runner, 0, ids, cuts), want, dtype, f"portions {cuts}", noise)


@BOTH
def test_the_first_tokens_and_one_token_requests(dtype, tmp_path):
    cfg = full_config()
    runner, w = make(tmp_path, cfg, seed=21, dtype=dtype)
    for n in (1, 2, 3):
        ids = tokens(n, cfg["vocab"], 30 + n)
        want = plain.forward(cfg, w, ids)
        noise = rounding(cfg, w, ids, want) if dtype == BF16 else None
        close(run_cut(runner, n, ids, [n]), want, dtype, f"a prompt of {n}", noise)
        close(run_cut(runner, n, ids, []), want, dtype, f"a prompt of {n}, token by token", noise)


def test_long_decoding(tmp_path):
    cfg = full_config()
    runner, w = make(tmp_path, cfg, seed=23, blocks=48, page=4)
    ids = tokens(180, cfg["vocab"], 24)
    close(run_cut(runner, 0, ids, [5]), plain.forward(cfg, w, ids), F32, "long decoding")


# ---- batches, pages and slots that are used again ---------------------------------------------------------------------------

@BOTH
@pytest.mark.parametrize("seed", [31, 32])
def test_unequal_batches_and_reuse(seed, dtype, tmp_path):
    """Up to four requests of unequal lengths side by side, portions of some beside single tokens of others, on a pool
    that only their peak fits and four state slots, requests ending and new ones taking their pages and slots: every position
    as alone."""
    from nanospec_b200.engine.step import StepEntry

    cfg = full_config()
    runner, w = make(tmp_path, cfg, seed=seed, dtype=dtype, blocks=30, page=4, slots=4)
    g = torch.Generator().manual_seed(seed)
    lengths = [23, 5, 41, 2, 17, 30, 9, 1, 12]
    prompts = [tokens(n, cfg["vocab"], seed * 100 + i) for i, n in enumerate(lengths)]
    want = [plain.forward(cfg, w, p) for p in prompts]
    got, at = [[] for _ in prompts], [0] * len(prompts)
    waiting, live = list(range(len(prompts))), []
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
            runner.begin(live[-1])
        entries = []
        for i in live:
            left_over = len(prompts[i]) - at[i]
            n = min(left_over, int(torch.randint(1, 9, (1,), generator=g)))
            if left_over > 6 and torch.rand(1, generator=g) < 0.2:
                continue  # left out of this step, goes on later
            entries.append((i, n))
        if not entries:
            continue
        logits = runner.step([StepEntry(i, prompts[i][at[i]: at[i] + n], list(range(n))) for i, n in entries]).float().cpu()
        row = 0
        for i, n in entries:
            got[i].append(logits[row: row + n])
            row += n
            at[i] += n
            if at[i] == len(prompts[i]):
                runner.end(i)
                live.remove(i)
        runner.manager.check()
    for i in range(len(prompts)):
        close(torch.cat(got[i]), want[i], dtype, f"request {i} in a batch", rounding(cfg, w, prompts[i], want[i], samples=1) if dtype == BF16 else None)


def test_one_stream_and_two_give_the_same_bits(tmp_path, monkeypatch):
    """What runs beside the main stream touches nothing that the main stream works on: the same kernels on one stream, bit for bit."""
    from nanospec_b200 import ops

    cfg = full_config(width=48)
    for dtype in (F32, BF16):
        runner, w = make(tmp_path, cfg, seed=36, dtype=dtype, page=16, blocks=40)
        ids = tokens(200, cfg["vocab"], 37)
        runs = []
        for beside in (True, False, True, True):
            monkeypatch.setattr(ops, "RUN_BESIDE", beside)
            runs.append(run_cut(runner, 0, ids, [120, 2, 60]))
        assert all(torch.equal(runs[0], r) for r in runs[1:])


# ---- other sizes, drawn from seeds ----------------------------------------------------------------------------------------

@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_from_seeds(seed, tmp_path):
    g = torch.Generator().manual_seed(4000 + seed)
    pick = lambda xs: xs[int(torch.randint(0, len(xs), (1,), generator=g))]
    layers = []
    for i in range(pick([1, 2, 3, 5])):
        own = [j for j, entry in enumerate(layers) if "weights_of" not in entry]
        if own and pick([0, 0, 1]):
            j = pick(own)
            layers.append(dict(copy.deepcopy(layers[j]), weights_of=j))
            continue
        experts = pick([1, 4, 9])
        mlp = pick([None, moe(experts=experts, top=pick([1, min(2, experts), experts]), ff=pick([8, 12, 64, 9]), limit=pick([0.2, 1.0, 7.0]), shared=pick([None, 8, 30, 64]),
                              shared_limit=pick([0.3, 2.0]))])
        kv, dim = pick([1, 2, 3]), pick([2, 8, 12, 16, 32])
        groups = pick([1, 2, 3])
        heads, vdim = groups * pick([1, 2, 4]), pick([2, 5, 8, 24])
        layers.append(layer(left(heads=kv * pick([1, 2, 4]), kv_heads=kv, dim=dim, vdim=pick([2, 8, 20, dim, 2 * dim, 152]), dims=pick([0, 2, dim]), base=pick([100.0, 50000.0]),
                                 scale=pick([None, 0.6, 0.11]), factor=pick([1.0, 2.0, 8.0, 0.5])),
                            right(heads=heads, vdim=vdim, state=pick([1, 4, 16, 33, 64]), groups=groups, conv=pick([1, 2, 4, 5]),
                                  norm_groups=pick([1, heads, heads * vdim // 2 if heads * vdim % 2 == 0 else 1])),
                            mlp, left_scale=pick([1.0, 0.5, -0.8]), right_scale=pick([1.0, 0.4, 2.0])))
    cfg = config(layers, width=pick([16, 24, 72, 33, 128]), vocab=pick([50, 131]), eps=pick([1e-5, 1e-6, 1e-3]), logit_scale=pick([1.0, 0.3, 4.0]))
    w = random_weights(cfg, seed)
    ids = tokens(48, cfg["vocab"], seed)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want)
    for dtype in (F32, BF16):
        runner, _ = make(tmp_path, cfg, seed=seed, dtype=dtype, page=pick([2, 4, 16]), weights=w)
        for cuts in ([48], [7, 2, 2, 19, 3], []):
            close(run_cut(runner, 0, ids, cuts), want, dtype, f"seed {seed}, portions {cuts or 'of one'}: {json.dumps(cfg)[:300]}", noise)


@pytest.mark.parametrize("dim,vdim,heads,kv_heads,state", [(64, 32, 8, 2, 64), (128, 200, 4, 4, 128), (32, 64, 6, 1, 16), (64, 136, 4, 2, 200), (96, 96, 4, 2, 48), (144, 160, 2, 1, 24)])
def test_tensor_core_sizes(dim, vdim, heads, kv_heads, state, tmp_path):
    """Head sizes that the tensor-core attention kernels take (values as wide as keys, narrower, wider, in slices) and one that they do not,
    states up to 200 rows, experts on the tensor cores, in bfloat16, over prompts long enough for several key tiles, with portions
    and single tokens; float32 beside it."""
    cfg = config([layer(left(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, dims=dim // 2, base=10000.0), right(heads=heads, vdim=24, state=state, groups=2 if heads > 1 else 1, conv=4),
                        moe(experts=6, top=2, ff=64, shared=64)), layer(left(dim=16), None, None)], width=64)
    ids = tokens(200, cfg["vocab"], dim)
    w = random_weights(cfg, dim)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want, samples=1)
    for dtype in (BF16, F32):
        runner, _ = make(tmp_path, cfg, seed=dim, dtype=dtype, blocks=80, page=16, weights=w)
        for cuts in ([200], [90, 2, 67, 14] + [1] * 20 + [7]):
            close(run_cut(runner, 0, ids, cuts), want, dtype, f"head size {dim}, portions {cuts[:4]}", noise)


@pytest.mark.parametrize("ff", [64, 16, 9], ids=["tcgen05 products", "multiples of 8", "other widths"])
@pytest.mark.parametrize("crowded", [False, True], ids=["spread", "crowded"])
def test_experts_in_long_steps(crowded, ff, tmp_path):
    """A step of 600 tokens, its experts chosen evenly or nearly all of them the same two; every kind of expert width."""
    experts = 30 if crowded else 6
    cfg = config([layer(left(dim=16), None, moe(experts=experts, top=3, ff=ff, shared=16))])
    w = random_weights(cfg, 66)
    w["l0.mlp.router.b"] = torch.zeros(experts)
    if crowded:
        w["l0.mlp.router.b"][torch.tensor([1, 2, 7])] = 8.0
    ids = tokens(600, cfg["vocab"], 67)
    want = plain.forward(cfg, w, ids)
    for dtype in (F32, BF16):
        runner, _ = make(tmp_path, cfg, seed=66, dtype=dtype, blocks=160, page=4, weights=w)
        close(run_cut(runner, 0, ids, [600]), want, dtype, "experts in a long step", torch.full((600,), 0.03))


# ---- through the engine: scheduler, graphs, sampling, command line ------------------------------------------------------------

def greedy(eng, cfg, w, prompts, n, dtype):
    """Greedy generation: every token is the plain statement's best one for what came before, up to near ties."""
    from nanospec_b200 import SamplingParams

    outs = eng.generate(prompts, SamplingParams(max_tokens=n, ignore_eos=True))
    gaps = []
    for p, out in zip(prompts, outs):
        assert len(out) == n
        z = plain.forward(cfg, w, p + out)
        for j, tok in enumerate(out):
            row = z[len(p) + j - 1]
            gaps.append(float(row.max() - row[tok]) / float(z.std()))
    gaps = torch.tensor(gaps)
    # (bfloat16: two experts that nearly tie may change places at one position in ten)
    assert float(gaps.max()) <= 1e-3 if dtype == F32 else float(gaps.quantile(0.9)) <= 0.1, f"another token is ahead by up to {float(gaps.max())} of the logits' spread"


@BOTH
@pytest.mark.parametrize("graphs", [False, True], ids=["eager", "graphs"])
def test_greedy_generation_through_the_engine(dtype, graphs, tmp_path):
    from nanospec_b200 import Engine, EngineConfig, load_model

    cfg = full_config()
    w = random_weights(cfg, 71)
    model = load_model(write_folder(tmp_path / "gen", cfg, w), device="cuda", dtype=dtype)
    eng = Engine(model, EngineConfig(num_blocks=64, block_size=4, max_running=3, prefill_chunk=11, cuda_graphs=graphs,
                                     graph_buckets=(1, 2, 4)))
    greedy(eng, cfg, w, [tokens(n, cfg["vocab"], 80 + n) for n in (3, 30, 1, 17, 12)], 12, dtype)


@pytest.mark.parametrize("graphs", [False, True], ids=["eager", "graphs"])
def test_both_norms_in_the_output_product(graphs, tmp_path):
    """bfloat16, a width in multiples of 128, steps of up to 64 tokens: the mixer's output product norms its result, adds it to the stream and
    applies the norm that the feed-forward (or the next layer) reads.  Portions of every size beside it, and generation."""
    from nanospec_b200 import Engine, EngineConfig
    from nanospec_b200.ops import lib

    cfg = config([layer(left(dim=16, vdim=24), right(heads=8, vdim=16), moe(ff=64, shared=64)), layer(left(dim=32, vdim=32), right(vdim=16, heads=4), None),
                  layer(None, None, moe(ff=24, shared=None)), layer(left(dim=32, vdim=32), right(vdim=16, heads=4), None, weights_of=1)], width=128)
    runner, w = make(tmp_path, cfg, seed=91, dtype=BF16, page=16, blocks=40)
    ids = tokens(150, cfg["vocab"], 6)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want, samples=2)
    lib.start_kernel_timing()
    got = run_cut(runner, 0, ids, [64, 2, 30, 3])
    seen = lib.stop_kernel_timing()
    assert seen.get("ns_gemm_bf16_tc_dyt", (0, 0.0))[0] > 0 and "ns_dyt_join" in seen, sorted(seen)
    close(got, want, BF16, "the norms in the product", noise)
    close(run_cut(runner, 1, ids, [150]), want, BF16, "the same model, a whole prompt", noise)
    eng = Engine(runner.model, EngineConfig(num_blocks=64, block_size=16, max_running=3, prefill_chunk=40, cuda_graphs=graphs, graph_buckets=(1, 2, 4)))
    greedy(eng, cfg, w, [tokens(n, cfg["vocab"], 60 + n) for n in (3, 70, 1, 17)], 10, BF16)


@pytest.mark.parametrize("width", [36, 128])
def test_weights_replaced_in_place(width, tmp_path):
    """`update_weights` on a bound model: the mixers hold views of the packed matrices, and new tensors land there."""
    from nanospec_b200.weights import update_weights

    cfg = config([layer(left(dim=16, vdim=8), right(vdim=8), moe(ff=32, shared=64)), layer(left(vdim=6), right(vdim=5, heads=3, groups=1, norm_groups=1), None)], width=width)
    runner, w = make(tmp_path, cfg, seed=5)
    ids = tokens(40, cfg["vocab"], 9)
    close(run_cut(runner, 0, ids, [17, 2]), plain.forward(cfg, w, ids), F32, "before")
    w2 = random_weights(cfg, 6)
    update_weights(runner.model, {k: v.clone() for k, v in w2.items()})
    got = run_cut(runner, 1, ids, [17, 2])
    close(got, plain.forward(cfg, w2, ids), F32, "after")
    assert float(distance(got, plain.forward(cfg, w, ids)).max()) > 0.1


@pytest.mark.parametrize("norm", ["dyt", "rmsnorm"])
def test_the_arrangement_beside_other_blocks_and_norms(norm, tmp_path):
    """Sandwich layers before and after a layer of the usual arrangement, one that runs again with the model's input added, with norms that
    fold and norms that join the stream in a kernel of their own."""
    from nanospec_b200.config import LayerSpec, ModelRecipe, PartSpec, Run
    from nanospec_b200.engine.step import ModelRunner
    from nanospec_b200.parts import DecoderModel

    width, vocab = 48, 60
    spec = PartSpec(norm, {"hidden": width, "weight_name": "w", **({"eps": 1e-5} if norm == "rmsnorm" else {})})
    mixer = PartSpec("gqa_attention", {"hidden": width, "heads": 4, "kv_heads": 2, "head_dim": 8, "position": PartSpec("rotary", {"head_dim": 8, "base": 100.0}),
                                       "bias": "qkv", "names": {"q": "q", "k": "k", "v": "v", "o": "o"}})
    ff = PartSpec("swiglu", {"hidden": width, "intermediate": 24, "names": {"gate": "gate", "up": "up", "down": "down"}})
    names = {"mixer": "m.", "feed_forward": "f.", "norm_mixer": "n1.", "post_mixer": "n1b.", "norm_feed_forward": "n2.", "post_feed_forward": "n2b."}
    layers = tuple(LayerSpec(block=b, prefix=f"{i}.", mixer=mixer, feed_forward=f, norm=spec, names=names) for i, (b, f) in enumerate(
        (("sandwich", ff), ("prenorm", ff), ("sandwich", None), ("sandwich", ff))))
    order = (Run(0, 0), Run(1, 1), Run(2, 2), Run(3, 3), Run(2, 4, add_input=True), Run(3, 5))
    model = DecoderModel(ModelRecipe("toy", PartSpec("table", {"vocab": vocab, "hidden": width, "prefix": "", "weight_name": "embed"}), layers, order, spec, "end.",
                                     PartSpec("linear", {"vocab": vocab, "hidden": width, "prefix": "", "weight_name": "embed2"}), vocab, width, 4096), F32, "cuda")
    g = torch.Generator().manual_seed(8)
    W = {n: torch.randn(s.shape, generator=g) * (0.2 if len(s.shape) == 2 else 0.3) + (1.0 if s.init == "gain" else 0.0) for n, s in sorted(model.weight_specs().items())}
    W["embed"] = W["embed"] * 5
    model.bind({n: t.cuda() for n, t in W.items()})
    D = {n: t.double() for n, t in W.items()}
    ids = tokens(25, vocab, 3)
    positions = torch.arange(25)

    def nrm(x, name):
        if norm == "dyt":
            return plain.dynamic_tanh(x, D, name + "w")
        return x / torch.sqrt((x * x).mean(-1, keepdim=True) + 1e-5) * D[name + "w"]

    def mix(h, p):
        q, k, v = ((h @ D[p + n].T + D[p + n + ".b"]).view(25, -1, 8) for n in ("q", "k", "v"))
        rot = {"dims": 8, "base": 100.0}
        return plain.attend(plain.rotate_half(q, positions, rot), plain.rotate_half(k, positions, rot), v, 8 ** -0.5) @ D[p + "o"].T

    def feed(h, p):
        return (plain.silu(h @ D[p + "gate"].T) * (h @ D[p + "up"].T)) @ D[p + "down"].T

    x = first = D["embed"][ids]
    for run in order:
        p = f"{run.layer}."
        x = x + first if run.add_input else x
        sandwich = layers[run.layer].block == "sandwich"
        y = mix(nrm(x, p + "n1."), p + "m.")
        x = x + (nrm(y, p + "n1b.") if sandwich else y)
        if layers[run.layer].feed_forward is not None:
            y = feed(nrm(x, p + "n2."), p + "f.")
            x = x + (nrm(y, p + "n2b.") if sandwich else y)
    want = nrm(x, "end.") @ D["embed2"].T
    runner = ModelRunner(model, num_blocks=40, block_size=4, max_requests=2)
    for cuts in ([25], [7, 2, 10], []):
        close(run_cut(runner, 0, ids, cuts), want, F32, f"portions {cuts}")


def test_command_line(tmp_path):
    """Random weights from a config.json, seeded sampling twice the same, greedy generation in float32, a trace replayed."""
    import subprocess
    import sys
    from pathlib import Path

    root = Path(__file__).resolve().parent.parent
    cfg_path = tmp_path / "cfg.json"
    cfg_path.write_text(json.dumps(full_config()))
    run = lambda *a, **kw: subprocess.run([sys.executable, "-m", "nanospec_b200", *a], cwd=root, capture_output=True, text=True, timeout=600, **kw)
    r = run("random-weights", "--config", str(cfg_path), "--out", str(tmp_path / "model"), "--seed", "4")
    assert r.returncode == 0, r.stderr
    outs = []
    for _ in range(2):
        r = run("generate", "--model", str(tmp_path / "model"), "--prompt-lens", "5", "21", "--max-tokens", "9", "--temperature", "0.8",
                "--top-k", "20", "--top-p", "0.9", "--seed", "3", "--ignore-eos")
        assert r.returncode == 0, r.stderr
        outs.append([json.loads(line)["output_ids"] for line in r.stdout.splitlines() if '"output_ids"' in line])
    assert outs[0] == outs[1] and [len(o) for o in outs[0]] == [9, 9]
    r = run("generate", "--model", str(tmp_path / "model"), "--dtype", "float32", "--prompt-ids", "1 2 3 4", "--max-tokens", "6", "--ignore-eos")
    assert r.returncode == 0, r.stderr
    assert len(json.loads(r.stdout.splitlines()[0])["output_ids"]) == 6
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3, 4, 5], "want": [4]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [6], "want": [0]}, {"id": "b", "tokens": [7, 8], "want": []}], "end": ["a"]}]
    r = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(tmp_path / "model"), "--dtype", "float32", "--out", str(tmp_path / "o"),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0 and "done 0" in r.stdout and "done 1" in r.stdout, r.stderr
    assert (tmp_path / "o" / "0.f32").stat().st_size == 4 * full_config()["vocab"]
