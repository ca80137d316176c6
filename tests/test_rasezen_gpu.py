"""The Rasezen parts on the GPU against the plain statement in plain_rasezen.py: each kernel and each mechanism alone, whole prompts
against token-by-token decoding, portions down to two tokens, unequal batches, pages and state slots that are used again, keys just
inside and just outside a window (in prompts and in decoding), a token far back seen through the state, the first tokens, long
decoding, sizes that differ everywhere (also those that the tensor-core kernels take), and greedy generation through the engine.
Each test makes its own small configuration and weights."""

from __future__ import annotations

import copy
import json
import math
from types import SimpleNamespace

import pytest
import torch

import plain_rasezen as plain

pytestmark = pytest.mark.gpu

F32, BF16 = torch.float32, torch.bfloat16
BOTH = pytest.mark.parametrize("dtype", [F32, BF16], ids=["float32", "bfloat16"])


# ---- configurations ---------------------------------------------------------------------------------------------------

def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, identity=2, top=3, ff=24, scale=1.8, shared=32):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "scale": scale, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def attn(mlp=None, heads=4, kv_heads=2, dim=8, vdim=6, size=7, dims=4, base=300.0, scale=None):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5,
        "mask": {"size": size}, "rot": {"dims": dims, "base": base}}}


def mamba(mlp=None, heads=4, vdim=6, state=8, groups=2, conv=3, norm_groups=2):
    return {"type": "mamba2", "mlp": mlp, "mixer": {
        "heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def config(layers, width=40, vocab=89, eps=1e-5):
    return {"architecture": "Rasezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def full_config(**kw):
    """Both mixers and every kind of feed-forward; sizes differ from layer to layer."""
    return config([attn(dense(56), heads=6, kv_heads=2, dim=12, vdim=10, size=9, dims=8),
                   mamba(moe(shared=40), heads=6, vdim=8, state=16, groups=3, conv=4, norm_groups=4),
                   attn(moe(experts=3, identity=0, top=2, ff=16, shared=None), heads=2, kv_heads=2, dim=16, vdim=16, size=5, dims=16),
                   mamba(dense(24), heads=3, vdim=10, state=5, groups=1, conv=2, norm_groups=5),
                   attn(None, heads=5, kv_heads=1, dim=6, vdim=4, size=13, dims=0)], **kw)


def routed(cfg):
    return any((layer["mlp"] or {}).get("kind") == "moe" for layer in cfg["layers"])


def random_weights(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """Names and shapes from the framework's own list, values from here, bfloat16-representable."""
    from nanospec_b200.weights import build_model

    model, _ = build_model(cfg, None, F32, "cpu")
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, spec in sorted(model.weight_specs().items()):
        t = torch.randn(spec.shape, generator=g)
        leaf = name.split(".")[-1]
        if leaf == "conv":
            t = 0.6 * t
        elif leaf == "router":
            t = t * (2.0 / math.sqrt(spec.shape[1]))
        elif leaf == "correction":
            t = 0.05 * t
        elif len(spec.shape) == 2:
            t = t * (1.5 / math.sqrt(spec.shape[1]))
        elif leaf in ("norm", "norm1", "D"):
            t = 1.0 + 0.2 * t
        elif leaf == "b":
            t = 0.3 * t
        elif leaf == "dt_bias":
            t = 0.5 * t - 1.0
        elif leaf == "A_log":
            t = 0.7 * t - 1.5  # decays from a few tokens to hundreds
        out[name] = t.to(BF16).float()   # (xielu's two numbers: standard normal)
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


def close(got, want, dtype, what="", noise=None, experts=False):
    """float32: a few roundings against the logits' spread at every position.  bfloat16: small at the median position, and at
    every position within a few times of what rounding alone does there (`noise`, from `rounding`), never of the size that a
    wrong mask, a lost state or a wrong page gives elsewhere.  `experts`: two experts whose scores nearly tie can change places
    under bfloat16 rounding and take a token's output with them, so one position in ten may leave the limit."""
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

def test_xielu_kernel_alone():
    """Contiguous and as column ranges of wider rows; both branches, large and tiny inputs."""
    from nanospec_b200 import ops

    g = torch.Generator().manual_seed(2)
    p, q = torch.tensor(0.4, dtype=torch.float64), torch.tensor(-1.3, dtype=torch.float64)
    coef = torch.tensor([math.log1p(math.exp(0.4)), 0.5 + math.log1p(math.exp(-1.3))], dtype=F32).cuda()
    for shape in ((5, 24), (3, 7)):
        for dtype in (F32, BF16):
            x = torch.randn(shape, generator=g) * 3
            x[0, :6] = torch.tensor([0.0, 1e-4, -1e-4, -30.0, 40.0, -0.02])
            x = x.to(dtype)
            want = plain.xielu(x.double(), p, q)
            tol = 1e-6 if dtype == F32 else 1e-2
            got = ops.activation(x.cuda(), torch.empty(shape, dtype=dtype, device="cuda"), "xielu", coef)
            assert ((got.float().cpu() - want).abs() <= tol * want.abs() + 1e-7).all()
            wide = torch.zeros(shape[0], shape[1] + 16, dtype=dtype, device="cuda")
            wide[:, 8: 8 + shape[1]] = x.cuda()
            out = torch.zeros_like(wide)
            ops.activation(wide[:, 8: 8 + shape[1]], out[:, 8: 8 + shape[1]], "xielu", coef)
            assert torch.equal(out[:, 8: 8 + shape[1]], got) and not out[:, :8].any() and not out[:, 8 + shape[1]:].any()


def test_gated_activation_over_column_ranges():
    from nanospec_b200 import ops

    g = torch.Generator().manual_seed(3)
    for inter, block in ((64, 0), (128, 64), (12, 0)):
        for dtype in (F32, BF16):
            rows = torch.randn(6, 2 * inter + 24, generator=g).to(dtype).cuda()
            gu = rows[:, 16: 16 + 2 * inter]
            want = ops.swiglu(gu.contiguous(), torch.empty(6, inter, dtype=dtype, device="cuda"), block)
            out = torch.zeros(6, inter + 8, dtype=dtype, device="cuda")
            ops.swiglu(gu, out[:, :inter], block)
            assert torch.equal(out[:, :inter], want) and not out[:, inter:].any()


@pytest.mark.parametrize("E,identity,top,N", [(5, 2, 3, 9), (60, 10, 6, 33), (40, 0, 36, 4), (1, 1, 1, 5), (1, 0, 1, 3), (3, 7, 4, 20)])
def test_routing_with_a_correction_and_identity_experts(E, identity, top, N):
    """Scores over every router output, the choice by corrected score, bare weights; the plan skips the experts that return their
    input; the combination, rounded and into a float32 stream, takes the input for them; the few-token kernel agrees."""
    from nanospec_b200 import ops

    g = torch.Generator().manual_seed(E + top)
    C = E + identity
    logits = torch.randn(N, C, generator=g) * 1.5
    correction = torch.randn(C, generator=g) * 0.2
    ids = torch.empty(N, top, dtype=torch.int32, device="cuda")
    weights = torch.empty(N, top, dtype=F32, device="cuda")
    ops.moe_route(logits.cuda(), 1, 1, top, 2.5, ids, weights, softmax=True, correction=correction.cuda(), renormalize=False)
    s = torch.softmax(logits.double(), -1)
    want_ids = torch.argsort(s + correction.double(), dim=-1, descending=True, stable=True)[:, :top].contiguous()
    assert torch.equal(ids.cpu().long(), want_ids)
    assert (weights.cpu().double() - 2.5 * s.gather(1, want_ids)).abs().max() <= 1e-6
    offsets = torch.empty(E + 1, dtype=torch.int32, device="cuda")
    row_of, pair_of = torch.empty_like(ids), torch.full_like(ids, -7)
    ops.moe_plan(ids, E, offsets, row_of, pair_of)
    real = want_ids < E
    assert torch.equal(row_of.cpu() < 0, ~real) and int(offsets[-1]) == int(real.sum())
    rows = row_of.cpu()[real]
    assert sorted(rows.tolist()) == list(range(len(rows)))
    flat = pair_of.cpu().view(-1)
    for r, pair in zip(rows.tolist(), torch.nonzero(real.view(-1)).view(-1).tolist()):
        assert int(flat[r]) == pair and int(offsets[want_ids.view(-1)[pair]]) <= r < int(offsets[want_ids.view(-1)[pair] + 1])
    for width in (24, 10):
        for dtype in (F32, BF16):
            ys = torch.randn(N * top, width, generator=g).to(dtype)
            x = torch.randn(N, width, generator=g).to(dtype)
            want = torch.zeros(N, width, dtype=torch.float64)
            for n in range(N):
                for k in range(top):
                    r = int(row_of[n, k])
                    want[n] += float(weights[n, k]) * (ys[r] if r >= 0 else x[n]).double()
            out = ops.moe_combine(ys.cuda(), row_of, weights, torch.empty(N, width, dtype=dtype, device="cuda"), top, x=x.cuda())
            size = float(want.abs().max())
            assert (out.cpu().double() - want).abs().max() <= (1e-6 if dtype == F32 else 8e-3) * size
            resid = torch.randn(N, width, generator=g)
            got = ops.moe_combine(ys.cuda(), row_of, weights, None, top, x=x.cuda(), resid=resid.cuda().contiguous())
            assert (got.cpu().double() - (want + resid.double())).abs().max() <= 2e-6 * max(size, 1.0)
    width, ff = 16, 8
    for dtype in (F32, BF16):
        wg, wu = (torch.randn(E, ff, width, generator=g) * 0.3 for _ in range(2))
        wd = torch.randn(E, width, ff, generator=g) * 0.3
        wg, wu, wd, x = (t.to(dtype) for t in (wg, wu, wd, torch.randn(N, width, generator=g)))
        out = ops.moe_expert_rows(x.cuda(), ids, weights, wg.cuda(), wu.cuda(), wd.cuda(), torch.empty(N * top, ff, dtype=dtype, device="cuda"),
                                  torch.empty(N, width, dtype=dtype, device="cuda"))
        want = torch.zeros(N, width, dtype=torch.float64)
        for n in range(N):
            for k in range(top):
                e, w = int(ids[n, k]), float(weights[n, k])
                if e < E:
                    a = plain.silu(x[n].double() @ wg[e].double().T) * (x[n].double() @ wu[e].double().T)
                    want[n] += w * (a @ wd[e].double().T)
                else:
                    want[n] += w * x[n].double()
        assert (out.cpu().double() - want).abs().max() <= (1e-5 if dtype == F32 else 2e-2) * float(want.abs().max())


@BOTH
@pytest.mark.parametrize("H,G,d,dv,dims", [(4, 2, 8, 6, 4), (4, 2, 16, 24, 16), (3, 3, 64, 64, 32), (2, 1, 24, 8, 16), (2, 1, 8, 264, 0), (6, 1, 10, 20, 10)])
def test_preparation_with_biases_norms_and_unit_values(H, G, d, dv, dims, dtype):
    """Biases, one norm over all of q and one over all of k, the rotation in halves and unit values per head: the rows that the
    attention reads and what lands in the pages, at positions near zero and far on."""
    from nanospec_b200 import ops

    g = torch.Generator().manual_seed(H * d + dv)
    N, page, eps, base = 11, 4, 1e-3, 300.0
    positions = torch.tensor([0, 1, 2, 3, 4, 9, 10, 11, 12, 30, 31])
    cols = H * d + G * (d + dv)
    rows = torch.randn(N, cols + 8, generator=g).to(dtype)
    bias = torch.randn(cols, generator=g)
    qg, kg = 1.0 + 0.3 * torch.randn(H * d, generator=g), 1.0 + 0.3 * torch.randn(G * d, generator=g)
    u = rows[:, :cols].double() + bias.double()
    want_q = plain.rotate_half(plain.rms_norm(u[:, : H * d], eps, qg.double()).view(N, H, d), positions, dims, base)
    want_k = plain.rotate_half(plain.rms_norm(u[:, H * d: (H + G) * d], eps, kg.double()).view(N, G, d), positions, dims, base)
    want_v = plain.rms_norm(u[:, (H + G) * d:].reshape(N, G, dv), eps, 1.0)
    table = torch.tensor([[5, 2, 7, 0, 1, 3, 4, 6]], dtype=torch.int32)
    kc, vc = torch.zeros(8, G, page, d, dtype=dtype, device="cuda"), torch.zeros(8, G, page, dv, dtype=dtype, device="cuda")
    lane = SimpleNamespace(k=kc, v=vc, block_table=table.cuda(), page_size=page)
    ctx = SimpleNamespace(positions=positions.int().cuda(), token_req=torch.zeros(N, dtype=torch.int32, device="cuda"))
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F32).cuda() if dims else None
    r = rows.cuda()
    ops.qk_norm_rope_store(r, ctx, lane, f, 1.0, False, H, G, d, dv, qg.cuda(), kg.cuda(), eps, bias=bias.cuda(), v_norm=True)
    tol = 3e-6 if dtype == F32 else 1e-2
    out = r.cpu().double()
    assert (out[:, : H * d].view(N, H, d) - want_q).abs().max() <= tol * float(want_q.abs().max())
    assert torch.equal(out[:, cols:], rows.double()[:, cols:])
    for n, p in enumerate(positions.tolist()):
        pg = int(table[0, p // page])
        assert (kc[pg, :, p % page].cpu().double() - want_k[n]).abs().max() <= tol * float(want_k.abs().max())
        assert (vc[pg, :, p % page].cpu().double() - want_v[n]).abs().max() <= tol * float(want_v.abs().max())


@BOTH
@pytest.mark.parametrize("H,V,N,G,taps,parts", [(4, 6, 5, 2, 3, 3), (2, 16, 16, 1, 4, 1), (6, 8, 24, 3, 2, 4), (3, 5, 40, 3, 1, 5), (8, 64, 64, 2, 4, 2),
                                               (1, 40, 130, 1, 6, 20), (12, 8, 8, 4, 5, 12), (2, 150, 70, 1, 4, 3), (4, 6, 300, 2, 3, 1)])
@pytest.mark.parametrize("chunked", [False, True], ids=["token by token", "in chunks"])
def test_state_space_kernels_alone(chunked, H, V, N, G, taps, parts, dtype, monkeypatch):
    """Preparation, the state's walk, gate and norm over two requests in portions (state and convolution tail carried in their slots)
    against the plain walk over the whole sequences; rows wider than the projection; decays from fast to slow, one step size near
    zero and one head that forgets nearly everything.  In chunks: portions of one chunk, of several and of a part of one, beside
    a request of one token."""
    from nanospec_b200 import ops
    from nanospec_b200.parts.recurrent import Mamba2
    from nanospec_b200.config.recipe import PartSpec

    g = torch.Generator().manual_seed(H * V + N)
    inner, chan = H * V, H * V + 2 * G * N
    part = Mamba2(PartSpec("mamba2", {"hidden": 8, "heads": H, "v_dim": V, "state": N, "groups": G, "conv": taps, "norm_groups": parts, "eps": 1e-4}), dtype, "cuda")
    t = {n: torch.randn(s.shape, generator=g) for n, s in part.weight_specs().items()}
    t["A_log"], t["dt_bias"], t["conv"] = 0.8 * t["A_log"] - 1.0, t["dt_bias"] - 1.0, 0.5 * t["conv"]
    t["dt_bias"][0] = -9.0
    t["A_log"][-1] = 2.5
    monkeypatch.setattr(ops, "SSM_CHUNKED_MIN", 2 if chunked else 1 << 30)
    part.bind({n: v.to(dtype if n in ("in", "o") else F32).cuda() for n, v in t.items()})
    lengths, cuts = [240, 80], [[130, 1, 2, 107], [3, 64, 1, 12]]
    seqs = [torch.randn(n, part.columns + 8, generator=g).to(dtype) for n in lengths]
    want = []
    rnd = (lambda x: x) if dtype == F32 else (lambda x: x.to(BF16).double())  # the convolution's result is rounded like a projection's
    for x in seqs:
        p = x.double()
        z, xbc, dt = p[:, :inner], p[:, inner: inner + chan], p[:, inner + chan: inner + chan + H]
        xbc = rnd(plain.silu(plain.causal_convolution(xbc, t["conv"].double(), t["conv.b"].double())))
        T = len(x)
        y = plain.state_space_walk(xbc[:, :inner].reshape(T, H, V), xbc[:, inner: inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N),
                                   plain.softplus(dt + t["dt_bias"].double()), t["A_log"].double(), t["D"].double())
        want.append(plain.gated_norm(y.reshape(T, inner), z, 1e-4, t["norm"].double(), parts))
    lane = SimpleNamespace(state=torch.zeros(3, part.state_floats, dtype=F32, device="cuda"))
    bufs = {}

    def buffer(name, cols, dt=None, rows=None):
        bufs[name] = torch.full((rows or n_rows, cols), float("nan"), dtype=dt or dtype, device="cuda")
        return bufs[name]

    at, got = [0, 0], [[], []]
    for step in range(4):
        ns = [cuts[b][step] for b in range(2)]
        n_rows = sum(ns)
        rows = torch.cat([seqs[b][at[b]: at[b] + ns[b]] for b in range(2)]).cuda()
        ctx = SimpleNamespace(
            token_req=torch.tensor([b for b in range(2) for _ in range(ns[b])], dtype=torch.int32, device="cuda"),
            qo_indptr=torch.tensor([0, ns[0], n_rows], dtype=torch.int32, device="cuda"),
            state_slot=torch.tensor([2, 0], dtype=torch.int32, device="cuda"), n_requests=2, max_q_len=max(ns), q_lens=ns, extras={}, buffer=buffer)
        out = torch.zeros(n_rows, inner + 8, dtype=dtype, device="cuda")
        part.forward_projected(rows, ctx, lane, True, out[:, :inner])
        o = out.cpu().double()
        assert not o[:, inner:].any()
        got[0].append(o[: ns[0], :inner])
        got[1].append(o[ns[0]:, :inner])
        at = [at[b] + ns[b] for b in range(2)]
    assert not lane.state[1].any()  # the slot that nobody holds
    for b in range(2):
        off = (torch.cat(got[b]) - want[b]).abs()  # (nothing may stay unwritten: a NaN fails the comparison)
        size = float(want[b].abs().max())
        if dtype == F32:
            assert off.max() <= 5e-5 * size, (b, float(off.max()), size)
        else:  # a rounding at the convolution's output that falls the other way moves a state a little
            assert off.max() <= 3e-2 * size and off.mean() <= 3e-3 * size, (b, float(off.max()), float(off.mean()), size)


# ---- each mechanism alone -----------------------------------------------------------------------------------------------

SINGLE = {
    "attention alone": lambda: config([attn()]),
    "a window of one": lambda: config([attn(size=1, heads=2, kv_heads=1)]),
    "every query head with keys of its own, whole heads turn": lambda: config([attn(heads=3, kv_heads=3, dims=8)]),
    "five query heads to a key head, nothing turns, values wider than keys": lambda: config([attn(heads=5, kv_heads=1, dim=6, vdim=14, dims=0, size=11)]),
    "a window wider than the prompt": lambda: config([attn(size=100, scale=1.1)]),
    "state space alone": lambda: config([mamba()]),
    "one head, one group, one part, one tap": lambda: config([mamba(heads=1, groups=1, norm_groups=1, conv=1, vdim=10, state=3)]),
    "a group for every head, parts across heads, six taps": lambda: config([mamba(heads=6, groups=6, norm_groups=4, conv=6, vdim=10, state=12)]),
    "a part for every feature but two": lambda: config([mamba(heads=4, vdim=4, norm_groups=8, groups=1, state=20)]),
    "dense beside attention": lambda: config([attn(dense(24))]),
    "dense beside the state space": lambda: config([mamba(dense(24)), attn()]),
    "experts beside attention": lambda: config([attn(moe())]),
    "no identity experts, no shared one": lambda: config([attn(moe(identity=0, shared=None)), mamba(dense(16))]),
    "one expert": lambda: config([mamba(moe(experts=1, identity=0, top=1, shared=8))]),
    "more identity experts than real ones, all chosen": lambda: config([mamba(moe(experts=2, identity=4, top=6, scale=0.7))]),
    "everything": full_config,
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


@BOTH
def test_sublayers_with_products_of_their_own(dtype, tmp_path):
    """The arrangement with its packing switched off, beside the packed form of the same model."""
    from nanospec_b200.parts.block import ParallelBlock

    cfg = config([attn(dense(16), dim=16, vdim=8), mamba(moe(ff=16, shared=24), vdim=8), attn(moe(ff=8, shared=None), dim=16, vdim=16), mamba(None, vdim=8)])
    ids = tokens(37, cfg["vocab"], 5)
    ParallelBlock.PACK = False
    try:
        runner, w = make(tmp_path, cfg, seed=77, dtype=dtype)
    finally:
        ParallelBlock.PACK = True
    assert all(b.w_in is None for b in runner.model.blocks)
    packed, _ = make(tmp_path / "p", cfg, seed=77, dtype=dtype, weights=w)
    assert all(b.w_in is not None for b in packed.model.blocks)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want) if dtype == BF16 else None
    for cuts in ([37], [], [2, 3, 2, 11, 5, 2]):
        close(run_cut(runner, 0, ids, cuts), want, dtype, f"own products, portions {cuts or 'of one'}", noise, True)
        close(run_cut(packed, 0, ids, cuts), want, dtype, f"packed products, portions {cuts or 'of one'}", noise, True)


@pytest.mark.parametrize("graphs", [False, True], ids=["eager", "graphs"])
def test_the_next_norm_in_the_output_product(graphs, tmp_path):
    """bfloat16, a width in multiples of 128, steps of up to 64 tokens: the packed output product adds its result to the stream and
    prepares the norm of a layer whose feed-forward is dense or absent.  Portions of every size beside it, and generation."""
    from nanospec_b200 import Engine, EngineConfig, SamplingParams
    from nanospec_b200.ops import lib

    cfg = config([attn(dense(128), dim=16, vdim=16), mamba(dense(64), heads=8, vdim=16), attn(dense(40), dim=32, vdim=16),
                  mamba(moe(ff=64, shared=64), heads=4, vdim=16), attn(None, heads=2, kv_heads=1, dim=32, vdim=32, size=20)], width=128)
    runner, w = make(tmp_path, cfg, seed=91, dtype=BF16, page=16, blocks=40)
    ids = tokens(150, cfg["vocab"], 6)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want, samples=2)
    lib.start_kernel_timing()
    got = run_cut(runner, 0, ids, [64, 2, 30, 3])
    seen = lib.stop_kernel_timing()
    assert seen.get("ns_gemm_bf16_tc_norm", (0, 0.0))[0] > 0, sorted(seen)
    close(got, want, BF16, "the norm in the products", noise, True)
    close(run_cut(runner, 1, ids, [150]), want, BF16, "the same model, a whole prompt", noise, True)
    eng = Engine(runner.model, EngineConfig(num_blocks=64, block_size=16, max_running=3, prefill_chunk=40, cuda_graphs=graphs, graph_buckets=(1, 2, 4)))
    greedy(eng, cfg, w, [tokens(n, cfg["vocab"], 60 + n) for n in (3, 70, 1, 17)], 10, BF16)


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


@pytest.mark.parametrize("width", [36, 128], ids=["own products", "packed products"])
def test_weights_replaced_in_place(width, tmp_path):
    """`update_weights` on a bound model: the sublayers hold views of the block's packed matrices, and new tensors land there."""
    from nanospec_b200.weights import update_weights

    cfg = config([attn(dense(64), dim=16, vdim=8), mamba(moe(ff=32, shared=64), vdim=8), mamba(None, vdim=16)], width=width)
    runner, w = make(tmp_path, cfg, seed=5)
    assert (runner.model.blocks[0].w_in is not None) == (width == 128)
    ids = tokens(40, cfg["vocab"], 9)
    close(run_cut(runner, 0, ids, [17, 2]), plain.forward(cfg, w, ids), F32, "before")
    w2 = random_weights(cfg, 6)
    update_weights(runner.model, {k: v.clone() for k, v in w2.items()})
    got = run_cut(runner, 1, ids, [17, 2])
    close(got, plain.forward(cfg, w2, ids), F32, "after")
    assert float(distance(got, plain.forward(cfg, w, ids)).max()) > 0.1


def test_layers_one_by_one(tmp_path):
    """The stream after every layer, in float32, against the plain statement's."""
    from nanospec_b200.engine.step import StepEntry

    cfg = full_config()
    runner, w = make(tmp_path, cfg, seed=3)
    ids = tokens(29, cfg["vocab"], 8)
    want, got = [], []
    plain.forward(cfg, w, ids, layers_out=want)

    def probe(i, resid, pending):
        x = resid.detach().cpu().double().clone()
        for p in pending if isinstance(pending, (tuple, list)) else (pending,):
            if p is not None:
                x += p.detach().cpu().double()
        got.append(x)

    runner.begin(0)
    ctx, rows, _ = runner.build_context([StepEntry(0, ids, [])])
    ctx.extras["probe"] = probe
    runner.forward(ctx, rows)
    runner.end(0)
    assert len(got) == len(want)
    for i, (a, b) in enumerate(zip(got, want)):
        assert (a - b).abs().max() <= 2e-5 * float(b.abs().max()), f"layer {i}: {float((a - b).abs().max())}"


# ---- window edges, lost pieces, the state ---------------------------------------------------------------------------------

def window_edge_case(dim):
    """Attention first, the state space after it.  In the first layer every query head's map is its key head's with the halves of its
    input swapped (biases and gains alike), and four tokens B have the embeddings of four tokens A with the halves swapped: a B's
    query points where its A's key points, nothing turns, and the scale makes that one score stand out.  The pairs sit on the
    window's last key (size - 1 back) and just outside it (size back), in the same page and across pages."""
    size, width = 9, 40
    cfg = config([attn(dense(16), heads=4, kv_heads=2, dim=dim, vdim=dim, size=size, dims=0, scale=1.5),
                  mamba(moe(ff=16, shared=24), vdim=8, conv=3), attn(None, heads=2, kv_heads=2, dim=dim, vdim=8, size=4, dims=dim, scale=0.9)], width=width)
    w = random_weights(cfg, 14)
    w["l0.mix.q"] = torch.roll(w["l0.mix.k"], width // 2, dims=1).view(2, 1, dim, width).expand(2, 2, dim, width).reshape(4 * dim, width).clone()
    w["l0.mix.q.b"] = w["l0.mix.k.b"].view(2, 1, dim).expand(2, 2, dim).reshape(-1).clone()
    w["l0.mix.q.norm"], w["l0.mix.k.norm"] = torch.ones(4 * dim), torch.ones(2 * dim)
    for i in range(4):
        w["embed"][84 + i] = torch.roll(w["embed"][80 + i], width // 2)
    ids = [t % 80 for t in tokens(45, cfg["vocab"], 17)]
    for i, (at, back) in enumerate(((3, size - 1), (12, size), (21, size - 1), (30, size))):
        ids[at], ids[at + back] = 80 + i, 84 + i
    return cfg, w, ids, size


@BOTH
@pytest.mark.parametrize("dim", [8, 16], ids=["exact", "tensor-core"])
def test_window_edges_and_what_else_could_be_lost(dim, dtype, tmp_path):
    """A window one key longer or shorter, values that are not normed, lost biases, a lost tap, skip, correction or shared expert, an
    identity expert that returns nothing: each moves the plain logits by far more than the engine differs from the right ones - in a
    prompt, in portions that cut through windows and pages, and token by token.  Heads of 8 run in the exact kernel in both types,
    heads of 16 in the tensor-core kernels in bfloat16."""
    cfg, w, ids, size = window_edge_case(dim)
    runner, w = make(tmp_path, cfg, seed=14, dtype=dtype, page=4, weights=w)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want)
    calm = noise <= 0.05  # bfloat16: the variants are told apart at the positions that rounding leaves alone
    wrong = {}
    for delta in (-1, 1):
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["mask"]["size"] = size + delta
        wrong[f"window {delta:+d}"] = plain.forward(other, w, ids)
    for name in ("l0.mix.q.b", "l0.mix.v.b", "l1.mix.D", "l1.mix.conv.b", "l1.mix.dt_bias", "l1.mlp.shared.down", "l1.mlp.e0.down"):
        wrong[name] = plain.forward(cfg, {**w, name: torch.zeros_like(w[name])}, ids)
    tap = w["l1.mix.conv"].clone()
    tap[:, 0] = 0.0
    wrong["the tap two tokens back"] = plain.forward(cfg, {**w, "l1.mix.conv": tap}, ids)
    keep = plain.rms_norm
    plain.rms_norm = lambda x, eps, g: x if isinstance(g, float) else keep(x, eps, g)
    try:
        wrong["values as projected"] = plain.forward(cfg, w, ids)
    finally:
        plain.rms_norm = keep
    for cuts in ([45], [], [size - 1, 2, size, 3, 2, 2, size + 1], [4, 4, 4, 4, 4], [size, size, size]):
        got = run_cut(runner, 0, ids, cuts)
        close(got, want, dtype, f"window edges, portions {cuts or 'of one'}", noise, True)
        keepers = torch.ones_like(calm) if dtype == F32 else calm
        right = float(distance(got, want)[keepers].max())
        for what, z in wrong.items():
            off = float(distance(got, z)[keepers].max())
            assert off > (10 if dtype == F32 else 2) * right and off > 0.03, f"{what} is not told apart: {off} against {right}"


def far_token_case():
    """One state-space layer with slow decays and one token whose trace is the largest: token 48's embedding points where every
    head's step size grows, and where no other token's does."""
    cfg = config([mamba(None, heads=4, vdim=8, state=16, groups=2, conv=4, norm_groups=2)], width=64, vocab=50)
    w = random_weights(cfg, 41)
    w["l0.mix.A_log"], w["l0.mix.dt_bias"] = torch.full((4,), -6.0), torch.full((4,), -5.0)
    w["embed"][:, 0], w["l0.mix.in"][:, 0] = 0.0, 0.0
    w["l0.mix.in"][-4:] = 0.0
    w["l0.mix.in"][-4:, 0] = 3.0
    w["embed"][48, 0] = 8.0
    w["l0.mix.D"], w["l0.mix.o"] = torch.zeros(4), w["l0.mix.o"] * 4.0
    w = {k: v.to(BF16).float() for k, v in w.items()}
    ids = tokens(450, 48, 42)
    ids[31] = 48          # the last position of the second page of 16
    lost = list(ids)
    lost[31] = 47
    return cfg, w, ids, lost


@BOTH
@pytest.mark.parametrize("least", [2, 1 << 30], ids=["in chunks", "token by token"])
def test_the_walk_does_not_depend_on_the_cut(least, dtype, tmp_path, monkeypatch):
    """Portions that begin and end inside chunks, on their edges and one beside them, with the state walked in chunks and token by token."""
    from nanospec_b200 import ops

    monkeypatch.setattr(ops, "SSM_CHUNKED_MIN", least)
    cfg = config([mamba(dense(16), heads=4, vdim=12, state=24, groups=2, conv=4), attn(None, dim=16, vdim=8, size=30), mamba(None, heads=6, vdim=5, state=7, groups=3)])
    runner, w = make(tmp_path, cfg, seed=58, dtype=dtype, page=16, blocks=40)
    ids = tokens(260, cfg["vocab"], 59)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want, samples=1) if dtype == BF16 else None
    for cuts in ([260], [64, 64, 65, 63], [2, 127, 1, 2, 66], [100, 3, 100]):
        close(run_cut(runner, 0, ids, cuts), want, dtype, f"portions {cuts}", noise)


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
def test_window_edges_far_on(dtype, tmp_path):
    """Two hundred positions on, in decoding and in portions, with the pages behind the window given back and used again."""
    cfg = config([attn(dense(16), heads=4, kv_heads=2, dim=16, vdim=16, size=21, dims=8, scale=1.5), attn(None, dim=16, vdim=8, size=50, scale=1.0)])
    runner, w = make(tmp_path, cfg, seed=52, dtype=dtype, page=4, blocks=60)
    ids = tokens(230, cfg["vocab"], 53)
    want = plain.forward(cfg, w, ids)
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["mask"]["size"] = 20
    assert float(distance(plain.forward(other, w, ids)[200:], want[200:]).max()) > 0.05
    noise = rounding(cfg, w, ids, want, samples=1) if dtype == BF16 else None
    for cuts in ([230], [30], [100, 2, 61, 40, 3]):
        close(run_cut(runner, 0, ids, cuts), want, dtype, f"windows, portions {cuts}", noise)


@BOTH
def test_the_first_tokens_and_one_token_requests(dtype, tmp_path):
    cfg = full_config()
    runner, w = make(tmp_path, cfg, seed=21, dtype=dtype)
    for n in (1, 2, 3):
        ids = tokens(n, cfg["vocab"], 30 + n)
        want = plain.forward(cfg, w, ids)
        noise = rounding(cfg, w, ids, want) if dtype == BF16 else None
        close(run_cut(runner, n, ids, [n]), want, dtype, f"a prompt of {n}", noise, True)
        close(run_cut(runner, n, ids, []), want, dtype, f"a prompt of {n}, token by token", noise, True)


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
            left = len(prompts[i]) - at[i]
            n = min(left, int(torch.randint(1, 9, (1,), generator=g)))
            if left > 6 and torch.rand(1, generator=g) < 0.2:
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
        close(torch.cat(got[i]), want[i], dtype, f"request {i} in a batch", rounding(cfg, w, prompts[i], want[i], samples=1) if dtype == BF16 else None, True)


# ---- other sizes, drawn from seeds ----------------------------------------------------------------------------------------

@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_from_seeds(seed, tmp_path):
    g = torch.Generator().manual_seed(4000 + seed)
    pick = lambda xs: xs[int(torch.randint(0, len(xs), (1,), generator=g))]
    layers = []
    for _ in range(pick([1, 2, 3, 5])):
        experts, identity = pick([1, 4, 9]), pick([0, 1, 3])
        mlp = pick([None, dense(pick([8, 20, 64])), moe(experts=experts, identity=identity, top=pick([1, min(2, experts + identity), experts]), ff=pick([8, 12, 40]),
                                                        scale=pick([1.0, 0.3, 3.0]), shared=pick([None, 8, 30, 64]))])
        if pick([0, 1]):
            kv = pick([1, 2, 3])
            dim = pick([2, 8, 12, 16, 32])
            layers.append(attn(mlp, heads=kv * pick([1, 2, 4]), kv_heads=kv, dim=dim, vdim=pick([2, 8, 20, dim]), size=pick([1, 2, 8, 33, 100]),
                               dims=pick([0, 2, dim]), base=pick([100.0, 50000.0]), scale=pick([None, 0.6, 0.11])))
        else:
            groups = pick([1, 2, 3])
            heads, vdim = groups * pick([1, 2, 4]), pick([2, 5, 8, 24])
            layers.append(mamba(mlp, heads=heads, vdim=vdim, state=pick([1, 4, 16, 33, 64]), groups=groups, conv=pick([1, 2, 4, 5]),
                                norm_groups=pick([1, heads, heads * vdim // 2 if heads * vdim % 2 == 0 else 1])))
    cfg = config(layers, width=pick([16, 24, 72, 33]), vocab=pick([50, 131]), eps=pick([1e-5, 1e-6, 1e-3]))
    w = random_weights(cfg, seed)
    ids = tokens(48, cfg["vocab"], seed)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want)
    for dtype in (F32, BF16):
        runner, _ = make(tmp_path, cfg, seed=seed, dtype=dtype, page=pick([2, 4, 16]), weights=w)
        for cuts in ([48], [7, 2, 2, 19, 3], []):
            close(run_cut(runner, 0, ids, cuts), want, dtype, f"seed {seed}, portions {cuts or 'of one'}: {json.dumps(cfg)[:300]}", noise, routed(cfg))


@pytest.mark.parametrize("dim,vdim,heads,kv_heads,size,state", [(64, 32, 8, 2, 88, 64), (128, 128, 4, 4, 70, 128), (32, 64, 6, 1, 130, 16), (48, 24, 2, 1, 75, 200)])
def test_tensor_core_sizes(dim, vdim, heads, kv_heads, size, state, tmp_path):
    """Head sizes that the tensor-core attention kernels take (values as wide as keys, narrower, wider), states up to 200 rows, experts
    on the tensor cores, in bfloat16, over prompts long enough for several key tiles and windows, with portions and single tokens;
    float32 beside it."""
    cfg = config([attn(dense(64), heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, size=size, dims=dim // 2, base=10000.0),
                  mamba(moe(experts=6, identity=1, top=2, ff=64, shared=64), heads=heads, vdim=vdim, state=state, groups=2, conv=4, norm_groups=2),
                  attn(None, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, size=size + 40, dims=dim, base=10000.0)], width=64)
    ids = tokens(200, cfg["vocab"], size)
    w = random_weights(cfg, size)
    want = plain.forward(cfg, w, ids)
    noise = rounding(cfg, w, ids, want, samples=1)
    for dtype in (BF16, F32):
        runner, _ = make(tmp_path, cfg, seed=size, dtype=dtype, blocks=80, page=16, weights=w)
        for cuts in ([200], [90, 2, 67, 14] + [1] * 20 + [7]):
            close(run_cut(runner, 0, ids, cuts), want, dtype, f"head size {dim}, portions {cuts[:4]}", noise, True)


@pytest.mark.parametrize("tile", [32, 128, 256])
@pytest.mark.parametrize("E,identity,top,N,width,ff", [(6, 2, 3, 300, 72, 64), (3, 1, 2, 7, 64, 128), (40, 0, 2, 90, 136, 192), (1, 1, 1, 40, 8, 64)])
def test_experts_as_tcgen05_products(E, identity, top, N, width, ff, tile):
    """The products whose tiles are found from the plan on the device, against float64 on their own operands: experts with no token,
    with one, with more than a tile holds; rows behind the last pair hold garbage that nothing may pick up."""
    from nanospec_b200 import ops

    g = torch.Generator().manual_seed(E + N)
    x = torch.randn(N, width, generator=g).to(BF16)
    wg, wu = ((torch.randn(E, ff, width, generator=g) / math.sqrt(width)).to(BF16) for _ in range(2))
    wd = (torch.randn(E, width, ff, generator=g) / math.sqrt(ff)).to(BF16)
    ids = torch.stack([torch.randperm(E + identity, generator=g)[:top] for _ in range(N)]).int()
    if E > 2:
        ids[ids == 0] = E - 1            # expert 0 gets nobody, the last one more than its share (some tokens twice)
    packed = torch.stack([wg.view(E, ff // 64, 64, width), wu.view(E, ff // 64, 64, width)], dim=2).reshape(E, 2 * ff, width).contiguous().cuda()
    offsets = torch.empty(E + 1, dtype=torch.int32, device="cuda")
    row_of = torch.empty(N, top, dtype=torch.int32, device="cuda")
    ops.moe_plan(ids.cuda(), E, offsets, row_of)
    buf = lambda cols: torch.full((N * top, cols), float("nan"), dtype=BF16, device="cuda")
    xs, act, ys = ops.moe_gather(x.cuda(), row_of, buf(width), top), buf(ff), buf(width)
    old, ops.MOE_TILE = ops.MOE_TILE, tile
    try:
        ops.moe_grouped_tc(xs, offsets, packed, wd.cuda(), act, ys)
    finally:
        ops.MOE_TILE = old
    torch.cuda.synchronize()
    ops.check_kernel_errors()
    n = int(offsets[-1])
    assert n == int((ids < E).sum()) and torch.isnan(ys[n:]).all()
    for t in range(N):
        for k in range(top):
            e, row = int(ids[t, k]), int(row_of[t, k])
            if e >= E:
                assert row == -1
                continue
            a = plain.silu(x[t].double() @ wg[e].double().T) * (x[t].double() @ wu[e].double().T)
            want = a.to(BF16).double() @ wd[e].double().T
            assert (ys[row].cpu().double() - want).abs().max() <= 0.02 * max(1.0, float(want.abs().max())), (t, k)


@pytest.mark.parametrize("ff", [64, 16], ids=["tcgen05 products", "other widths"])
@pytest.mark.parametrize("crowded", [False, True], ids=["spread", "crowded"])
def test_experts_in_long_steps(crowded, ff, tmp_path):
    """A step of 600 tokens, its experts chosen evenly or nearly all of them the same two, identity experts among the chosen; expert widths
    in multiples of 64, and others: one batched product over equal shares while the choice is even."""
    from nanospec_b200.ops import lib

    experts = 30 if crowded else 6
    cfg = config([attn(moe(experts=experts, identity=2, top=3, ff=ff, shared=16), size=40)])
    w = random_weights(cfg, 66)
    w["l0.mlp.correction"] = torch.zeros(experts + 2)
    if crowded:
        w["l0.mlp.correction"][torch.tensor([1, 2, experts + 1])] = 2.0
    w = {k: v.to(BF16).float() for k, v in w.items()}
    ids = tokens(600, cfg["vocab"], 67)
    want = plain.forward(cfg, w, ids)
    for dtype in (F32, BF16):
        runner, _ = make(tmp_path, cfg, seed=66, dtype=dtype, blocks=160, page=4, weights=w)
        lib.start_kernel_timing()
        got = run_cut(runner, 0, ids, [600])
        seen = lib.stop_kernel_timing()
        if dtype == BF16:
            assert ("ns_moe_grouped_tc" if ff == 64 else "ns_moe_grouped" if crowded else "ns_moe_pad_rows") in seen, sorted(seen)
        close(got, want, dtype, "experts in a long step", torch.full((600,), 0.03), True)
        close(run_cut(runner, 1, ids, [600]), want, dtype, "the same on two streams", torch.full((600,), 0.03), True)


# ---- through the engine: scheduler, graphs, sampling, command line ------------------------------------------------------------

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


def test_a_state_larger_than_the_token_walk_takes(tmp_path):
    """More rows of the state than the token walk holds: single tokens too run as chunks, under graphs as well."""
    from nanospec_b200 import Engine, EngineConfig

    cfg = config([mamba(dense(16), heads=2, vdim=8, state=260, groups=1), mamba(None, heads=2, vdim=8, state=16, groups=1)])
    runner, w = make(tmp_path, cfg, seed=61)
    ids = tokens(80, cfg["vocab"], 62)
    want = plain.forward(cfg, w, ids)
    for cuts in ([80], [], [30, 2, 40]):
        close(run_cut(runner, 0, ids, cuts), want, F32, f"portions {cuts}")
    eng = Engine(runner.model, EngineConfig(num_blocks=64, block_size=4, max_running=3, prefill_chunk=11, graph_buckets=(1, 2, 4)))
    greedy(eng, cfg, w, [tokens(n, cfg["vocab"], 70 + n) for n in (3, 30, 1)], 8, F32)


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
