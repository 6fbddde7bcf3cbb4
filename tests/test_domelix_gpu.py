"""Domelix on the GPU against the plain implementation (tests/plain_domelix.py): the small kernels, each mechanism alone
through portions and batches, biases made to show at every edge of the distance buckets, a key that stands out from far
away, memories that carry their first token to the end, the matrix form against the walk, then whole models in every cut,
batches, reuse of pages and slots, long decoding and greedy generation through the engine's entry point."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_domelix as plain
from domelix_models import CONFIGS, make_folder
from harness import Replayer, assert_close
from test_binupel_gpu import MixerBench, part_weights

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 2e-5, "bfloat16": 2e-2}
F64 = torch.float64


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {key: make_folder(str(tmp_path_factory.mktemp(f"domelix_{key}")), config, seed)
            for key, (config, seed) in CONFIGS.items()}


def tokens(vocab, n, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def close(got, want, dtype, what="", tol=None):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} vs {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite values"
    err = float((got - want).abs().max()) / max(float(want.abs().max()), 1e-9)
    bound = TOL[dtype] if tol is None else tol
    assert err <= bound, f"{what}: relative error {err:.3g} > {bound:g}"


def part(kind, name, params):
    from qwen3_from_scratch_b200.parts.base import PartSpec
    from qwen3_from_scratch_b200.registry import create_part
    return create_part(kind, PartSpec(name, params), name="m")


def rotation(dims, base=1000.0):
    from qwen3_from_scratch_b200.parts.base import PartSpec
    return PartSpec("rotary_stretched", {"dims": dims, "base": base})


# ---------------------------------------------------------------------- the small kernels
@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("W,T", [(48, 5), (64, 33), (201, 7), (1030, 19), (5000, 3)])
def test_open_terms_into_the_stream_and_both_norms(W, T, dtype):
    """What a layer left open (a plain term and two that are brought to unit root mean square, weighted and scaled) into
    the stream and two norms with weights around zero, in one kernel; with fewer terms; for chosen rows with the stream
    left alone."""
    from qwen3_from_scratch_b200.parts.base import PendingSum, PendingTerm, Runtime
    rt = Runtime(torch.device("cuda:0"), DT[dtype], 64, 2)
    eps, term_eps = 1e-5, 1e-3
    norms, refs = [], []
    for seed in (1, 2):
        n = part("norm", "rms_norm", {"dim": W, "eps": eps, "one_plus": True})
        dev, ref = part_weights(n, dtype, seed=W + seed)
        n.setup(rt, dict(dev))
        norms.append(n)
        refs.append(ref["weight"])
    g = torch.Generator().manual_seed(W + T)
    stream0 = 2 * torch.randn(T, W, generator=g)
    deltas = [((0.02 if i == 0 else 1.5) * torch.randn(T, W, generator=g)).to(DT[dtype]) for i in range(3)]
    weights = [1 + 0.2 * torch.randn(W, generator=g) for _ in range(2)]
    tight = 2e-6 if dtype == "float32" else 8e-3
    terms = (PendingTerm(deltas[0].cuda(), weights[0].cuda(), 0.5), PendingTerm(deltas[1].cuda(), weights[1].cuda(), 0.7),
             PendingTerm(deltas[2].cuda()))
    wants = [0.5 * plain.unit_rms(deltas[0].double(), term_eps) * weights[0].double(),
             0.7 * plain.unit_rms(deltas[1].double(), term_eps) * weights[1].double(), deltas[2].double()]
    for chosen in ((0, 1, 2), (2,), (1, 2), ()):
        total = stream0.double() + sum((wants[i] for i in chosen), torch.zeros(T, W, dtype=F64))
        pending = PendingSum(tuple(terms[i] for i in chosen), term_eps) if chosen else None
        stream = stream0.clone().cuda()
        first, second = norms[0].add_norm_pair(stream, pending, norms[1])
        close(stream, total, "float32", f"stream {chosen}", tol=1e-6)
        close(first, plain.norm_one_plus(total, refs[0], eps), dtype, f"first {chosen}", tol=tight)
        close(second, plain.norm_one_plus(total, refs[1], eps), dtype, f"second {chosen}", tol=tight)
        if chosen:
            stream = stream0.clone().cuda()
            close(norms[0].add_norm(stream, pending), plain.norm_one_plus(total, refs[0], eps), dtype, "alone", tol=tight)
            close(stream, total, "float32", "stream, one norm", tol=1e-6)
            stream = stream0.clone().cuda()
            rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32).cuda()
            got = norms[1].norm_rows(stream, pending, rows)
            close(got, plain.norm_one_plus(total, refs[1], eps)[rows.cpu().long()], dtype, "rows", tol=tight)
            assert torch.equal(stream.cpu(), stream0)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("n,parts,weight,gate", [(96, 3, "all", "sigmoid"), (96, 3, None, "silu"), (2048, 16, "part", "silu"),
                                                 (130, 5, "part", "sigmoid"), (1024, 1, "all", "sigmoid"), (4099, 1, "all", "silu"),
                                                 (24, 1, None, "silu")])
def test_norm_and_gate_behind_a_memory(n, parts, weight, gate, dtype):
    from qwen3_from_scratch_b200.kernels import ops
    g = torch.Generator().manual_seed(n + parts)
    T = 11
    o = torch.randn(T, n, generator=g) * torch.logspace(-2, 1, T)[:, None]
    proj = torch.randn(T, n + 16, generator=g).to(DT[dtype])
    w = None if weight is None else 1 + 0.2 * torch.randn(n if weight == "all" else n // parts, generator=g)
    wide = torch.full((T, n + 8), 3.0, dtype=DT[dtype], device="cuda")
    ops.memory_out(o.cuda(), proj.cuda(), 8, None if w is None else w.cuda(), 1e-4, gate, wide[:, 4:4 + n], parts)
    want = plain.unit_rms(o.double().view(T, parts, -1), 1e-4).reshape(T, n)
    if w is not None:
        want = want * (w.double() if weight == "all" else w.double().repeat(parts))
    z = proj[:, 8:8 + n].double()
    want = want * (plain.silu(z) if gate == "silu" else plain.sigmoid(z))
    close(wide[:, 4:4 + n], want, dtype, "gated", tol=2e-6 if dtype == "float32" else 8e-3)
    assert float(wide[:, :4].min()) == 3.0 and float(wide[:, 4 + n:].min()) == 3.0


@pytest.mark.parametrize("dtype", list(DT))
def test_rotation_in_place(dtype):
    from qwen3_from_scratch_b200.kernels import ops
    g = torch.Generator().manual_seed(3)
    T, heads, D, dims, base = 7, 5, 24, 10, 300.0
    x = torch.randn(T, heads * D + 12, generator=g).to(DT[dtype])
    pos = [0, 1, 5, 90, 1000, 3, 17]
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64).float()
    dev = x.cuda()
    ops.rotate_columns(dev, 4, heads, D, dims, freq.cuda(), 1.0, torch.tensor(pos, dtype=torch.int32).cuda())
    want = plain.rotate_halves(x[:, 4:4 + heads * D].double().view(T, heads, D), pos, base, dims).reshape(T, -1)
    close(dev[:, 4:4 + heads * D], want, dtype, "rotated", tol=1e-4 if dtype == "float32" else 8e-3)
    assert torch.equal(dev[:, :4].cpu(), x[:, :4]) and torch.equal(dev[:, 4 + heads * D:].cpu(), x[:, 4 + heads * D:])


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("W,E,top,groups,keep", [(40, 12, 3, 4, 2), (64, 5, 2, 1, 1), (40, 1, 1, 1, 1), (128, 32, 8, 8, 3),
                                                 (64, 40, 5, 8, 3), (33, 36, 2, 2, 1), (64, 96, 6, 48, 6), (48, 7, 7, 7, 7)])
@pytest.mark.parametrize("rows", [3, 70, 1100])
def test_router_by_softmax_within_groups(W, E, top, groups, keep, rows, dtype):
    """Up to a warp's lanes of experts and more, groups of every kind, a token per block and eight: the chosen experts in
    order and their renormalised weights (rows with a near tie are left out); a token's choice bit for bit the same
    whatever else is in the step."""
    from qwen3_from_scratch_b200.kernels import ops
    g = torch.Generator().manual_seed(W + E + rows)
    h = torch.randn(rows, W, generator=g).to(DT[dtype])
    router = torch.randn(E, W, generator=g) * (3.0 / W ** 0.5)
    hd, rd = h.cuda(), router.cuda()

    def route(x):
        ids = torch.full((x.shape[0], top), -1, dtype=torch.int32, device="cuda")
        wts = torch.zeros(x.shape[0], top, device="cuda")
        ops.moe_route(x.contiguous(), rd, None, ids, wts, 1.0, "softmax", groups, keep, True)
        return ids.cpu(), wts.cpu()

    ids, wts = route(hd)
    z = h.double() @ router.double().t()
    spec = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}}
    clear = 0
    for t in range(min(rows, 150)):
        s = z[t].sort(descending=True).values
        if E > 1 and float((s[:-1] - s[1:]).min()) < 1e-5:
            continue
        clear += 1
        chosen, weights = plain.route(z[t], spec)
        assert ids[t].tolist() == chosen, t
        close(wts[t], weights, "float32", f"weights of row {t}", tol=1e-5)
    assert clear > 0.8 * min(rows, 150)
    for lo, hi in ((0, 1), (rows // 2, rows // 2 + 2)):
        part_ids, part_wts = route(hd[lo:hi])
        assert torch.equal(part_ids, ids[lo:hi]) and torch.equal(part_wts, wts[lo:hi])


# ---------------------------------------------------------------------- each mechanism alone
ATTENTION = {"hidden_size": 40, "num_heads": 6, "num_kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.25, "gate": True, "sink": True,
             "bias": {"most": 20, "rows": 8}}
LIGHTNING = {"hidden_size": 40, "num_heads": 3, "dim": 24, "vdim": 40, "decay": [0.0, 0.7, 0.995], "norm_eps": 1e-5,
             "activation": "silu", "norm": "row", "norm_weight": True, "gate": "sigmoid"}
RETENTION = {"hidden_size": 40, "num_heads": 3, "dim": 24, "vdim": 40, "decay": [0.5, 0.9, 0.999], "norm_eps": 1e-5,
             "norm": "heads", "gate": "silu"}
DELTA = {"hidden_size": 40, "num_heads": 4, "num_kv_heads": 2, "dim": 24, "vdim": 40, "conv": 3, "norm_eps": 1e-5}


def plain_attention(p):
    m = {"heads": p["num_heads"], "kv_heads": p["num_kv_heads"], "dim": p["dim"], "vdim": p["vdim"], "scale": p["scale"],
         "bias_max": p["bias"]["most"]}

    def fn(h, ref, st):
        st = st or {"k": torch.zeros(0, m["kv_heads"], m["dim"], dtype=F64), "v": torch.zeros(0, m["kv_heads"], m["vdim"], dtype=F64)}
        start = st["k"].shape[0]
        return plain.attention(h, ref, "", m, list(range(start, start + h.shape[0])), st), st
    return fn


def plain_memory(p, dims=None, base=1000.0):
    m = {"heads": p["num_heads"], "dim": p["dim"], "vdim": p["vdim"], "decay": p["decay"], "rot": {"base": base, "dims": dims or 0}}

    def fn(h, ref, st):
        st = st or {"S": torch.zeros(m["heads"], m["dim"], m["vdim"], dtype=F64), "n": 0}
        if p.get("activation") == "silu":
            return plain.lightning(h, ref, "", m, p["norm_eps"], st), st
        y = plain.retention(h, ref, "", m, p["norm_eps"], list(range(st["n"], st["n"] + h.shape[0])), st)
        st["n"] += h.shape[0]
        return y, st
    return fn


def plain_delta(p):
    m = {"heads": p["num_heads"], "kv_heads": p["num_kv_heads"], "dim": p["dim"], "vdim": p["vdim"], "conv": p["conv"]}
    qk = m["kv_heads"] * m["dim"]

    def fn(h, ref, st):
        tail = lambda n: torch.zeros(m["conv"] - 1, n, dtype=F64)  # noqa: E731
        st = st or {"S": torch.zeros(m["heads"], m["dim"], m["vdim"], dtype=F64), "q": tail(qk), "k": tail(qk),
                    "v": tail(m["heads"] * m["vdim"])}
        return plain.delta(h, ref, "", m, p["norm_eps"], st), st
    return fn


def retention_params(p, dims, base=1000.0):
    return dict(p, q_scale=p["dim"] ** -0.5, position=rotation(dims, base))


def moved_by_rounding(fn, x, ref, want):
    """Per row, what rounding the projections' operands and results to bfloat16 alone does in the plain implementation,
    relative to the largest value: a read-out that is a small difference of large terms, brought to unit size by the norm
    behind it, moves far."""
    with plain.bfloat16_projections():
        rounded = fn(x.double(), ref, None)[0]
    return (rounded - want).abs().max(dim=1).values / want.abs().max()


def mixer_cases():
    yield "attention", "kept_window_attention", ATTENTION, plain_attention(ATTENTION)
    one = dict(ATTENTION, num_heads=1, num_kv_heads=1, bias={"most": 2, "rows": 2}, vdim=16)
    yield "attention, one head, two rows", "kept_window_attention", one, plain_attention(one)
    tc = dict(ATTENTION, num_heads=8, dim=32, vdim=64, bias={"most": 50, "rows": 16})
    yield "attention of sizes for the tensor cores", "kept_window_attention", tc, plain_attention(tc)
    yield "lightning", "decayed_memory", LIGHTNING, plain_memory(LIGHTNING)
    tc = dict(LIGHTNING, num_heads=2, decay=[0.0, 0.97], dim=64, vdim=32)
    yield "lightning of sizes for the tensor cores", "decayed_memory", tc, plain_memory(tc)
    one = dict(LIGHTNING, num_heads=1, decay=[1.0], dim=33, vdim=5)
    yield "lightning, one head of odd sizes that forgets nothing", "decayed_memory", one, plain_memory(one)
    yield "retention, partly rotated", "decayed_memory", retention_params(RETENTION, 10), plain_memory(RETENTION, 10)
    tc = dict(RETENTION, num_heads=2, decay=[0.9, 0.9999], dim=128, vdim=64)
    yield "retention of sizes for the tensor cores", "decayed_memory", retention_params(tc, 128), plain_memory(tc, 128)
    wide = dict(RETENTION, num_heads=1, decay=[0.95], dim=200, vdim=24)
    yield "retention, nothing rotated, wide keys", "decayed_memory", retention_params(wide, 0), plain_memory(wide, 0)
    yield "delta", "gated_delta", DELTA, plain_delta(DELTA)
    one = dict(DELTA, num_heads=3, num_kv_heads=1, conv=1, dim=17, vdim=9)
    yield "delta, one tap, odd sizes", "gated_delta", one, plain_delta(one)
    tc = dict(DELTA, num_heads=2, num_kv_heads=2, dim=64, vdim=96, conv=4)
    yield "delta of sizes for the tensor cores", "gated_delta", tc, plain_delta(tc)
    wide = dict(DELTA, num_heads=2, num_kv_heads=1, dim=300, vdim=24, conv=6)
    yield "delta, wide keys, six taps", "gated_delta", wide, plain_delta(wide)


CASES = {name: rest for name, *rest in mixer_cases()}


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("case", list(CASES))
def test_mixer_alone_whole_in_portions_and_beside_another_request(case, dtype):
    """A mixer on random rows: a request whole; then the same in portions down to two tokens and single tokens, beside
    another request whose portions start and end elsewhere, in slots and pages that were used before."""
    kind, params, fn = CASES[case]
    p = part("mixer", kind, params)
    bench = MixerBench(p, dtype, page_size=4, pages=96, max_tokens=256, seed=11)
    g = torch.Generator().manual_seed(12)
    x_of = {r: torch.randn(n, params["hidden_size"], generator=g).to(DT[dtype]) for r, n in (("a", 175), ("b", 31), ("c", 9))}
    want = {r: fn(x.double(), bench.ref, None)[0] for r, x in x_of.items()}
    call = lambda rows, ctx: p.forward(rows.cuda().contiguous(), ctx, 0, True)  # noqa: E731
    tol = None
    if dtype == "bfloat16":
        tol = max(4e-2, 3 * max(float(moved_by_rounding(fn, x, bench.ref, want[r]).max()) for r, x in x_of.items()))
        assert tol < 0.2
    close(bench.run([("c", 9)], x_of, call)["c"], want["c"], dtype, f"{case}: short request", tol)
    bench.manager.close("c")  # its slot and pages go to the next ones
    close(bench.run([("a", 175)], x_of, call)["a"], want["a"], dtype, f"{case}: whole", tol)
    bench.manager.close("a")
    got = {"a": [], "b": []}
    steps = [[("a", 2)], [("b", 5), ("a", 1)], [("a", 30), ("b", 1)], [("a", 1), ("b", 2)], [("b", 20), ("a", 102)],
             [("a", 1)], [("a", 17), ("b", 3)]] + [[("a", 1)] for _ in range(21)]
    for step in steps:
        out = bench.run(step, x_of, call)
        for r, rows in out.items():
            got[r].append(rows)
    for r in got:
        close(torch.cat(got[r]), want[r], dtype, f"{case}: request {r} in portions", tol)


@pytest.mark.parametrize("dtype", list(DT))
def test_branches_normed_one_by_one(dtype):
    """Attention and lightning attention on one input product, an output product each; what is left open is half of each
    output's unit rows times its weight."""
    from qwen3_from_scratch_b200.parts.base import PartSpec
    a, b = dict(ATTENTION), dict(LIGHTNING)
    p = part("mixer", "parallel", {"hidden_size": 40, "out_norm": {"suffix": "out", "eps": 1e-5}, "branches": [
        {"label": "left", "mixer": PartSpec("kept_window_attention", a), "scale": 0.5},
        {"label": "right", "mixer": PartSpec("decayed_memory", b), "scale": 0.5}]})
    bench = MixerBench(p, dtype, page_size=4, pages=64, max_tokens=256, seed=21)
    x = torch.randn(90, 40, generator=torch.Generator().manual_seed(22)).to(DT[dtype])
    m = {"left": {"heads": 6, "kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.25, "bias_max": 20},
         "right": {"heads": 3, "dim": 24, "vdim": 40, "decay": b["decay"]}}
    st = {"left": {"k": torch.zeros(0, 2, 24, dtype=F64), "v": torch.zeros(0, 2, 40, dtype=F64)},
          "right": {"S": torch.zeros(3, 24, 40, dtype=F64)}}
    want = plain.branches(x.double(), bench.ref, "", m, 1e-5, list(range(90)), st)

    def call(rows, ctx):
        s = p.forward(rows.cuda().contiguous(), ctx, 0, True)
        assert len(s.terms) == 2 and s.eps == 1e-5
        return sum(t.scale * plain.unit_rms(t.delta.double(), s.eps) * t.weight.double() for t in s.terms)

    tol = None if dtype == "float32" else 4e-2
    got = torch.cat([bench.run([("r", c)], {"r": x}, call)["r"] for c in (40, 2, 1, 1, 33, 2, 1, 10)])
    close(got, want, dtype, "branches", tol)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("dim,vdim,heads,kv_heads", [(16, 24, 2, 1), (32, 64, 6, 2), (64, 32, 3, 3), (128, 128, 4, 1)])
def test_every_edge_of_the_distance_buckets_shows(dim, vdim, heads, kv_heads, dtype):
    """Scores nearly equal and a bias table of large values, so that the weights are the buckets': a key counted in the
    bucket next door changes the output.  Lengths that take distances through every bucket and hundreds beyond, as a
    whole prompt, in portions (edges inside a portion, at a page's border) and at single tokens; a window's worth of keys
    beyond the last edge keeps the last row."""
    params = dict(ATTENTION, hidden_size=32, num_heads=heads, num_kv_heads=kv_heads, dim=dim, vdim=vdim, scale=1e-3,
                  bias={"most": 61, "rows": 12}, gate=True)

    def tweak(dev, ref):
        table = 2.0 * torch.randn(12, heads, generator=torch.Generator().manual_seed(5)).to(torch.bfloat16)
        dev["m.rel"], ref["rel"] = table.float().cuda(), table.double()

    p = part("mixer", "kept_window_attention", params)
    n = 330
    bench = MixerBench(p, dtype, page_size=8, pages=64, max_tokens=512, seed=31, tweak=tweak)
    x = torch.randn(n, 32, generator=torch.Generator().manual_seed(32)).to(DT[dtype])
    fn = plain_attention(params)
    want = fn(x.double(), bench.ref, None)[0]
    # what an edge one position off would do: more than the tolerance at most positions
    real = plain.bucket
    try:
        plain.bucket = lambda d, rows, most: real(d + 1 if real(d + 1, rows, most) != real(d, rows, most) else d, rows, most)
        moved = (fn(x.double(), bench.ref, None)[0] - want).abs().max(dim=1).values / want.abs().max()
    finally:
        plain.bucket = real
    tol = 2e-5 if dtype == "float32" else 2e-2
    assert float((moved > 2 * tol).float().mean()) > 0.5
    call = lambda r, ctx: p.forward(r.cuda().contiguous(), ctx, 0, True)  # noqa: E731
    close(bench.run([("r", n)], {"r": x}, call)["r"], want, dtype, "whole prompt", tol)
    bench.manager.close("r")
    cuts = [5, 1, 1, 2, 60, 1, 40] + [2] * 10 + [64, 17] + [1] * (n - 211)
    close(torch.cat([bench.run([("r", c)], {"r": x}, call)["r"] for c in cuts]), want, dtype, "portions and single tokens", tol)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("dim,vdim", [(16, 24), (64, 64)])
def test_a_key_that_stands_out_from_far_away_and_a_strong_sink(dim, vdim, dtype):
    """One key among hundreds made to stand out (its input scaled), read from far away in a prompt and in single tokens,
    the first position and a page's last among the places; one head's sink so large that the head gives almost nothing,
    another's so small that it takes nothing."""
    params = dict(ATTENTION, hidden_size=32, num_heads=4, num_kv_heads=2, dim=dim, vdim=vdim, scale=1.0, bias={"most": 40, "rows": 8})

    def tweak(dev, ref):
        for tensors, pre in ((dev, "m."), (ref, "")):
            tensors[pre + "sink"][1] = 40.0
            tensors[pre + "sink"][0] = -40.0

    p = part("mixer", "kept_window_attention", params)
    fn = plain_attention(params)
    n = 300
    for at in (0, 39, 64):
        bench = MixerBench(p, dtype, page_size=8, pages=64, max_tokens=512, seed=43, tweak=tweak)
        g = torch.Generator().manual_seed(44 + at)
        x = 0.3 * torch.randn(n, 32, generator=g)
        x[at] = 4 * torch.randn(32, generator=g)
        x = x.to(DT[dtype])
        want = fn(x.double(), bench.ref, None)[0]
        quiet = x.clone()
        quiet[at] = 0
        moved = (want - fn(quiet.double(), bench.ref, None)[0]).abs().max(dim=1).values
        assert int((moved[200:] > 0.05 * float(want[1:].abs().max())).sum()) > 5, f"token {at} is read from far away"
        call = lambda rows, ctx: p.forward(rows.cuda().contiguous(), ctx, 0, True)  # noqa: E731
        tol = None if dtype == "float32" else 3e-2
        close(bench.run([("r", n)], {"r": x}, call)["r"], want, dtype, f"{at} whole", tol)
        bench.manager.close("r")
        cuts = [36, 2, 150, 3, 2] + [1] * 40 + [n - 233]
        close(torch.cat([bench.run([("r", c)], {"r": x}, call)["r"] for c in cuts]), want, dtype, f"{at} in portions", tol)


def _carry_inputs(n, seed):
    """Rows of which the first is large and the rest tiny: what the first token writes is most of every read-out."""
    g = torch.Generator().manual_seed(seed)
    x = 0.02 * torch.randn(n, 32, generator=g)
    x[0] = 6 * torch.randn(32, generator=g)
    return x


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("kind,dim,vdim", [("retention", 24, 40), ("retention", 64, 32), ("lightning", 128, 64), ("delta", 24, 16),
                                           ("delta", 64, 64)])
def test_a_slow_decay_carries_the_first_token_to_the_end(kind, dim, vdim, dtype):
    """Decays near one and a first token that writes the memory: what it wrote is still most of the output hundreds of
    tokens later, through portions and single tokens and beside another request's tokens."""
    tweak = None
    if kind == "delta":
        params = dict(DELTA, hidden_size=32, dim=dim, vdim=vdim, conv=2)
        fn, p = plain_delta(params), part("mixer", "gated_delta", params)

        def tweak(dev, ref):
            for tensors, pre in ((dev, "m."), (ref, "")):
                tensors[pre + "A_log"].fill_(-8.0)
    elif kind == "lightning":
        params = dict(LIGHTNING, hidden_size=32, dim=dim, vdim=vdim, decay=[0.9999, 0.999, 1.0])
        fn, p = plain_memory(params), part("mixer", "decayed_memory", params)
    else:
        params = dict(RETENTION, hidden_size=32, dim=dim, vdim=vdim, decay=[0.9999, 0.999, 1.0])
        fn, p = plain_memory(params, 8), part("mixer", "decayed_memory", retention_params(params, 8))
    n = 400
    bench = MixerBench(p, dtype, page_size=8, pages=8, max_tokens=512, seed=51, tweak=tweak)
    x_of = {"r": _carry_inputs(n, 52).to(DT[dtype]), "o": torch.randn(9, 32, generator=torch.Generator().manual_seed(53)).to(DT[dtype])}
    want = fn(x_of["r"].double(), bench.ref, None)[0]
    quiet = x_of["r"].clone()
    quiet[0] = 0

    def check(got, what):
        """Without the first row, which is so much larger that it would hide the others.  bfloat16: a query that turns past
        the one stored key reads a small difference of large terms, whose sign rounding decides; one row in twenty may."""
        if dtype == "float32":
            close(got[1:], want[1:], dtype, what, 1e-4)
            return
        err = (got[1:].double().cpu() - want[1:]).abs().max(dim=1).values / want[1:].abs().max()
        assert float((err > 4e-2).float().mean()) < 0.05 and float(err.median()) < 1e-2, what

    moved = (want - fn(quiet.double(), bench.ref, None)[0])[-50:].abs().max()
    assert float(moved) > 0.3 * float(want[-50:].abs().max())
    call = lambda rows, ctx: p.forward(rows.cuda().contiguous(), ctx, 0, True)  # noqa: E731
    check(bench.run([("r", n)], x_of, call)["r"], "whole")
    bench.manager.close("r")
    got = []
    for step in ([("r", 1)], [("r", 2), ("o", 4)], [("r", 290)], [("o", 1), ("r", 1)], [("r", 2)], [("r", 64), ("o", 4)]) \
            + tuple([("r", 1)] for _ in range(40)):
        got.append(bench.run(list(step), x_of, call)["r"])
    check(torch.cat(got), "portions")


def _walk(x, rule, G, H, D, Dv, lens, act, q_scale, state, matrix):
    """One step of ``ops.memory_scan`` on rows of several requests, by the walk or in the matrix form: (o, state)."""
    from qwen3_from_scratch_b200.kernels import ops
    B, T = len(lens), sum(lens)
    q_start = torch.tensor([0] + torch.tensor(lens).cumsum(0).tolist(), dtype=torch.int32).cuda()
    slots = torch.tensor(list(range(B, 0, -1)), dtype=torch.int32).cuda()
    out, status = torch.full((T, H * Dv), float("nan"), device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    st = state.clone()
    scratch = None
    if matrix:
        alloc = lambda tag, *s, dtype: torch.full(s, float("nan"), dtype=dtype, device="cuda")  # noqa: E731
        scratch = ops.MemoryScratch(alloc, T, B, H, D, Dv, not isinstance(rule, ops.MemoryDecay))
    ops.memory_scan(x, 0, G * D, 2 * G * D, rule, q_scale, act, st, G, q_start, slots, B, out, status, max_q_len=max(lens), scratch=scratch)
    assert int(status.item()) == 0
    return out, st


@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 64, 32), (2, 2, 128, 96), (6, 3, 128, 64), (3, 1, 64, 160)])
@pytest.mark.parametrize("lens", [[64], [200], [1, 64, 65, 130, 3], [2, 500, 1, 33]])
def test_matrix_form_equals_the_walk(H, G, D, Dv, lens):
    """The tensor-core form of the three memories against the token-by-token walk on the same bfloat16 rows, from states
    that are not empty, scratch filled with NaN: portions that end inside a chunk, at its edge and just beyond, single
    tokens beside them; decays of zero and one; the delta rule with nearly parallel keys, write strengths near one and
    decays from none to strong.  They differ by float32 rounding (and what two bfloat16 halves lose: 2^-16)."""
    from qwen3_from_scratch_b200.kernels import ops
    assert ops.memory_matrix_form(torch.bfloat16, D, Dv) and not ops.memory_matrix_form(torch.float32, D, Dv)
    g = torch.Generator().manual_seed(H + D + sum(lens))
    T, B = sum(lens), len(lens)
    state = 0.3 * torch.randn(B + 1, H, Dv, D, generator=g).cuda()
    decay = ops.MemoryDecay(([0.0, 1.0, 0.97, 0.6, 0.9999, 0.5])[:H], torch.device("cuda:0"))
    rows = (0.5 * torch.randn(T, 2 * H * D + H * Dv, generator=g)).to(torch.bfloat16).cuda()
    for act, tol in (("none", 5e-5), ("silu", 1e-2)):  # silu: the matrix form's operands are rounded after it
        a, sa = _walk(rows, decay, H, H, D, Dv, lens, act, 0.25, state, False)
        b, sb = _walk(rows, decay, H, H, D, Dv, lens, act, 0.25, state, True)
        close(b, a, "float32", f"decayed, {act}", tol=tol)
        close(sb, sa, "float32", f"decayed, {act}: state", tol=tol)
    common = torch.randn(1, G, D, generator=g)
    for spread, bias_b, rate in ((1.0, 0.0, -1.0), (0.3, 3.0, -6.0), (1.0, 0.0, 2.5)):
        k = common + spread * torch.randn(T, G, D, generator=g)
        rows = torch.cat([torch.randn(T, G * D, generator=g), k.reshape(T, G * D), torch.randn(T, H * Dv, generator=g)], 1)
        rows = rows.to(torch.bfloat16).cuda()
        gates = torch.randn(T, 2 * H + 3, generator=g)
        gates[:, 2:2 + H] += bias_b
        gates = gates.to(torch.bfloat16).cuda()
        rule = ops.DeltaGates(gates, 2, 2 + H, torch.full((H,), rate).cuda(), (0.1 * torch.randn(H, generator=g)).cuda())
        rule.proj = torch.cat([gates, gates], 1).contiguous()
        a, sa = _walk(rows, rule, G, H, D, Dv, lens, "none", D ** -0.5, state, False)
        b, sb = _walk(rows, rule, G, H, D, Dv, lens, "none", D ** -0.5, state, True)
        close(b, a, "float32", f"delta {spread} {bias_b} {rate}", tol=2e-4)
        close(sb, sa, "float32", f"delta {spread} {bias_b} {rate}: state", tol=2e-4)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("W,E,top,groups,keep,ff,rows", [(40, 12, 3, 4, 2, 24, 3), (40, 12, 3, 4, 2, 24, 23), (64, 3, 3, 1, 1, 20, 40),
                                                         (128, 8, 2, 2, 1, 48, 300), (136, 40, 4, 8, 3, 16, 1100), (48, 1, 1, 1, 1, 32, 9)])
def test_experts_chosen_within_groups(W, E, top, groups, keep, ff, rows, dtype):
    """A pair at a time (few tokens, float32, inner widths that are no multiple of 16) and as grouped products."""
    from qwen3_from_scratch_b200.parts.base import Runtime
    p = part("feed_forward", "routed_experts", {"hidden_size": W, "experts": E, "top": top, "expert_ff": ff, "activation": "silu",
                                                "correction": False, "gated": True, "score": "softmax", "groups": (groups, keep),
                                                "renormalise": True})
    dev, ref = part_weights(p, dtype, seed=W + rows, scale={"router": 6.0 / W ** 0.5})
    p.setup(Runtime(torch.device("cuda:0"), DT[dtype], 1200, 2), dict(dev))
    x = torch.randn(rows, W, generator=torch.Generator().manual_seed(rows)).to(DT[dtype])
    spec = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}}
    keep_rows = min(rows, 60)
    want = plain.experts(x[:keep_rows].double(), ref, "", {"router": spec})
    got = p.forward(x.cuda())[:keep_rows]
    # a near tie of two logits may fall the other way (in float32 too, against float64); such rows are left out
    z = (x[:keep_rows].double() @ ref["router"].t()).sort(dim=1, descending=True).values
    clear = (z[:, :-1] - z[:, 1:]).min(dim=1).values > 1e-5 if E > 1 else torch.ones(keep_rows, dtype=torch.bool)
    assert clear.float().mean() > 0.9
    close(got[clear], want[clear], dtype, "experts", tol=None if dtype == "float32" else 3e-2)


# ---------------------------------------------------------------------- whole models
def tolerance(dtype, cfg, w, seqs):
    """float32: 1e-4 of the largest logit: every memory's read-out, a sum with cancellation, is brought to unit size by the
    norm behind it, which hands on the float32 rounding of the sum, and up to five layers follow one another.  bfloat16:
    three times what rounding alone does to these prompts in the plain implementation (projections' operands and results
    rounded to bfloat16), and no less than the harness's bound."""
    if dtype == "float32":
        return 1e-4
    return max(TOL[dtype], 3 * max(plain.rounding_error(cfg, w, ids) for ids in seqs.values()))


def replay(folder, dtype, seqs, schedule, **session_args):
    from qwen3_from_scratch_b200.engine.session import Session
    args = dict(page_size=8, num_pages=96, max_seqs=3, max_step_tokens=256)
    args.update(session_args)
    session = Session(folder, dtype=dtype, **args)
    r = Replayer(session, seqs)
    schedule(r)
    session.manager.check()
    assert session.manager.free_slots() == args["max_seqs"]
    return r.result()


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("key", list(CONFIGS))
def test_model_whole_decoded_and_in_portions(folders, key, dtype):
    cfg, w = plain.read_model_folder(folders[key])
    n = 90 if key != "z" else 150
    ids = tokens(cfg["vocab"], n, 51)
    want = {"a": plain.forward_logits(cfg, w, ids)}
    tol = tolerance(dtype, cfg, w, {"a": ids})

    def whole(r):
        r.step([("a", n)])

    def decoded(r):
        r.step([("a", n - 60)])
        for _ in range(60):
            r.step([("a", 1)])

    def portions(r):
        for c in [3, 2, 2, 1, 17, 2, 31, 1, 1, 2, 16, 2, 8, 2] + [n - 90] * (n > 90):
            r.step([("a", c)])

    for name, schedule in (("whole", whole), ("decoded", decoded), ("portions", portions)):
        assert_close(replay(folders[key], dtype, {"a": ids}, schedule), want, dtype, f"{key} {name}", tol=tol)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("key", ["x", "z", "w"])
def test_unequal_requests_together_equal_each_alone_with_pages_and_slots_used_again(folders, key, dtype):
    """Five requests through two state slots and a pool that holds less than their sum: portions of some beside single
    tokens of others; a slot and its pages go to the next request as soon as one ends; freed pages are filled with NaN."""
    cfg, w = plain.read_model_folder(folders[key])
    lens = {"a": 61, "b": 7, "c": 33, "d": 1, "e": 40}
    seqs = {r: tokens(cfg["vocab"], n, 60 + i) for i, (r, n) in enumerate(lens.items())}
    want = {r: plain.forward_logits(cfg, w, ids) for r, ids in seqs.items()}

    def schedule(r):
        r.step([("a", 30), ("b", 5)])
        r.step([("a", 1), ("b", 2)])             # b ends: its slot is free
        r.step([("c", 2), ("a", 1)])             # c takes b's slot
        r.step([("a", 1), ("c", 20)])
        r.step([("c", 1)])                       # a is left out of a step
        r.step([("a", 28), ("c", 10)])           # both end
        r.step([("d", 1), ("e", 9)])             # a request of a single token
        for _ in range(31):
            r.step([("e", 1)])

    got = replay(folders[key], dtype, seqs, schedule, page_size=4, num_pages=30, max_seqs=2, poison_freed_pages=True)
    assert_close(got, want, dtype, f"{key} mixed", tol=tolerance(dtype, cfg, w, seqs))


def test_long_prompt_on_the_serving_kernels(folders):
    """bfloat16 at the serving kernels' sizes with pages of 16: a prompt of 700 tokens whole and cut into long and short
    portions with single tokens between them; then a batch of a long portion beside single tokens."""
    cfg, w = plain.read_model_folder(folders["z"])
    ids, other = tokens(cfg["vocab"], 700, 77), tokens(cfg["vocab"], 90, 78)
    want = {"a": plain.forward_logits(cfg, w, ids), "b": plain.forward_logits(cfg, w, other)}
    tol = tolerance("bfloat16", cfg, w, {"a": ids, "b": other})
    for name, cuts in (("whole", [700]), ("portions", [300, 1, 250, 1, 1, 130, 17])):
        got = replay(folders["z"], "bfloat16", {"a": ids}, lambda r, cuts=cuts: [r.step([("a", n)]) for n in cuts],
                     page_size=16, num_pages=64, max_seqs=2, max_step_tokens=1024)
        assert_close(got, {"a": want["a"]}, "bfloat16", f"z long {name}", tol=tol)

    def beside(r):
        r.step([("b", 70)])
        r.step([("a", 300), ("b", 1)])
        r.step([("b", 1), ("a", 399)])
        r.step([("a", 1), ("b", 18)])

    got = replay(folders["z"], "bfloat16", {"a": ids, "b": other}, beside, page_size=16, num_pages=64, max_seqs=2,
                 max_step_tokens=1024)
    assert_close(got, want, "bfloat16", "z long beside single tokens", tol=tol)


@pytest.mark.parametrize("dtype", list(DT))
def test_long_decoding_through_graphs(folders, dtype):
    """300 single tokens after a short prompt, replayed from CUDA graphs: memories, tails and pages are carried on the
    device from step to step."""
    cfg, w = plain.read_model_folder(folders["x"])
    ids = tokens(cfg["vocab"], 310, 71)
    want = {"a": plain.forward_logits(cfg, w, ids)}

    def schedule(r):
        r.step([("a", 10)])
        for _ in range(300):
            r.step([("a", 1)])

    got = replay(folders["x"], dtype, {"a": ids}, schedule, page_size=4, num_pages=80, max_seqs=2)
    assert_close(got, want, dtype, "long decoding", tol=tolerance(dtype, cfg, w, {"a": ids}))


@pytest.mark.parametrize("key", ["x", "z"])
def test_float32_cuts_give_identical_bits(folders, key):
    """In float32 every sum has an order that depends only on the token, so a prompt whole, in portions and token by token
    gives the same bits."""
    cfg, _ = plain.read_model_folder(folders[key])
    ids = tokens(cfg["vocab"], 45, 81)
    runs = [replay(folders[key], "float32", {"a": ids}, s)["a"] for s in (
        lambda r: r.step([("a", 45)]),
        lambda r: [r.step([("a", n)]) for n in (7, 2, 1, 20, 15)],
        lambda r: [r.step([("a", 1)]) for _ in range(45)])]
    assert torch.equal(runs[0], runs[1]) and torch.equal(runs[0], runs[2])


# ---------------------------------------------------------------------- the engine's entry points
@pytest.mark.parametrize("key", ["x", "y"])
def test_greedy_generation_through_the_engine_equals_plain(folders, key):
    """Prompts of unequal length through SyncEngine.batch_generate: chunked prompts, continuous batching with fewer slots
    than requests, lookahead, CUDA graphs; float32, prompts chosen so that no step is a near tie."""
    from qwen3_from_scratch_b200.engine.engine import SyncEngine
    cfg, w = plain.read_model_folder(folders[key])
    prompts, expected = [], []
    for i, n in enumerate([1, 9, 33, 70]):
        for seed in range(100 * i, 100 * i + 50):
            prompt = tokens(cfg["vocab"], n, seed)
            out, margins = plain.greedy(cfg, w, prompt, 12)
            if min(margins) > 2e-3:
                break
        prompts.append(prompt)
        expected.append(out)
    engine = SyncEngine(folders[key], dtype="float32", block_size=8, num_pages=64, max_num_seqs=3, max_num_tokens=48,
                        chunked_prefill_size=16)
    results, batch = engine.batch_generate(prompts, max_new_tokens=12, ignore_eos=True)
    assert batch.num_requests == 4
    for want, r in zip(expected, results):
        assert r.token_ids == want and r.finish_reason == "length"
    engine.session.manager.check()
    assert engine.session.manager.free_slots() == 3


def test_preempted_request_is_recomputed_from_a_clean_state(folders):
    """A pool too small for all requests at once: the one that loses its pages starts again in a zeroed slot and still
    generates what it generates alone."""
    from qwen3_from_scratch_b200.engine.engine import SyncEngine
    cfg, _ = plain.read_model_folder(folders["y"])
    prompts = [tokens(cfg["vocab"], n, 90 + i) for i, n in enumerate([30, 28, 26])]
    alone = SyncEngine(folders["y"], dtype="float32", block_size=4, num_pages=96, max_num_seqs=4, max_num_tokens=64)
    want = [alone.generate(p, max_new_tokens=24, ignore_eos=True) for p in prompts]
    tight = SyncEngine(folders["y"], dtype="float32", block_size=4, num_pages=34, max_num_seqs=4, max_num_tokens=64)
    results, _ = tight.batch_generate(prompts, max_new_tokens=24, ignore_eos=True)
    assert [r.token_ids for r in results] == want


@pytest.mark.parametrize("dtype", list(DT))
def test_trace_replay_program_and_command_line(folders, tmp_path, dtype):
    folder = folders["x"]
    cfg, w = plain.read_model_folder(folder)
    vocab = cfg["vocab"]
    a, b = tokens(vocab, 70, 31), tokens(vocab, 50, 32)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [0, 39]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b[:2], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": a[40:41], "want": [0]},
                                {"id": "b", "tokens": b[2:50], "want": [47, 0]}], "end": ["b"]},
        {"step": 3, "entries": [{"id": "a", "tokens": a[41:70], "want": list(range(29))}], "end": ["a"]},
    ]
    out = str(tmp_path / "out")
    cmd = [sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out,
           "--max-tokens", "192", "--poison-freed-pages"]
    proc = subprocess.run(cmd, input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                          timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(4)]
    la, lb = plain.forward_logits(cfg, w, a), plain.forward_logits(cfg, w, b)
    tol = tolerance(dtype, cfg, w, {"a": a, "b": b})

    def check(step, rows):
        got = torch.from_numpy(np.fromfile(os.path.join(out, f"{step}.f32"), dtype="<f4")).view(len(rows), vocab)
        want = torch.stack(rows)
        assert float((got - want).abs().max()) <= tol * float(max(la.abs().max(), lb.abs().max()))

    check(0, [la[0], la[39]])
    check(2, [la[40], lb[49], lb[2]])
    check(3, [la[41 + i] for i in range(29)])
    if dtype == "float32":
        prompt = a[:9]
        want, margins = plain.greedy(cfg, w, prompt, 6)
        gen = [sys.executable, "-m", "qwen3_from_scratch_b200", "generate", "--model", folder, "--dtype", "float32",
               "--prompt-ids", ",".join(map(str, prompt)), "--max-new-tokens", "6", "--ignore-eos",
               "--block-size", "4", "--num-pages", "32", "--max-num-seqs", "2", "--max-num-tokens", "32"]
        proc = subprocess.run(gen, capture_output=True, text=True, cwd=ROOT, timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        if min(margins) > 1e-3:
            assert json.loads(proc.stdout.splitlines()[0])["token_ids"] == want
