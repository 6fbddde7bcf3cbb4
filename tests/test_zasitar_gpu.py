"""Zasitar on the GPU against the plain implementation (tests/plain_zasitar.py): the small kernels, each mechanism alone
through portions and batches, keys made to show just inside and outside every window, memories that carry their first token
to the end, the matrix form against the walk, then whole models in every cut, batches, reuse of pages and slots, long
decoding and greedy generation through the engine's entry point."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_zasitar as plain
from harness import Replayer, assert_close
from test_binupel_gpu import MixerBench, part_weights
from zasitar_models import CONFIGS, make_folder

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 2e-5, "bfloat16": 2e-2}
F64 = torch.float64


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {key: make_folder(str(tmp_path_factory.mktemp(f"zasitar_{key}")), config, seed)
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


def whole_output(y):
    """What a part returns, with the bias that it may have left open."""
    return y if torch.is_tensor(y) else y.delta.float() + y.bias


def ints(*values):
    return torch.tensor(values, dtype=torch.int32).cuda()


# ---------------------------------------------------------------------- the small kernels
@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("W,lens", [(48, [5]), (64, [1, 9, 2, 30]), (201, [3, 4]), (1030, [19, 1]), (5000, [2, 1])])
def test_terms_with_biases_and_mixes_with_the_token_before(W, lens, dtype):
    """A sub-layer's output with a bias, normed, weighted and scaled, into the stream: alone, with the rows copied out, and
    (single tokens) on the way to the five mixes of a token with the one before; a portion's first token reads the state,
    which then holds the portion's last row."""
    from qwen3_from_scratch_b200.kernels import ops
    g = torch.Generator().manual_seed(W + sum(lens))
    T, B, M, eps = sum(lens), len(lens), 5, 1e-3
    tight = 2e-6 if dtype == "float32" else 8e-3
    status = ints(0)
    stream0, mu = 2 * torch.randn(T, W, generator=g), torch.rand(M, W, generator=g)
    delta, bias = torch.randn(T, W, generator=g).to(DT[dtype]), torch.randn(W, generator=g)
    weight = 1 + 0.2 * torch.randn(W, generator=g)
    state0 = torch.randn(B + 2, W, generator=g)
    term = (delta.cuda(), weight.cuda(), 0.7, bias.cuda())
    total = stream0.double() + 0.7 * plain.unit_rms(delta.double() + bias.double(), eps) * weight.double()
    for want_rows in (False, True):
        stream = stream0.clone().cuda()
        out = torch.full((T, W), 7.0, dtype=DT[dtype], device="cuda") if want_rows else None
        ops.sum_norm(stream, [term], eps, None, out, 0.0)
        close(stream, total, "float32", "stream", tol=1e-6)
        if want_rows:
            close(out, total, dtype, "rows", tol=tight)

    def mixes(rows, starts, slots, term):
        stream, state = rows.clone().cuda(), state0.clone().cuda()
        n = rows.shape[0]
        out = torch.full((M, n, W), 7.0, dtype=DT[dtype], device="cuda")
        seq = [b for b in range(len(starts) - 1) for _ in range(starts[b + 1] - starts[b])]
        ops.sum_mix(stream, term, eps, mu.cuda(), state, ints(*starts), ints(*seq), ints(*slots), len(starts) - 1, out, status)
        assert int(status.item()) == 0
        return stream, state, out

    starts = [0]
    for n in lens:
        starts.append(starts[-1] + n)
    slots = list(range(B, 0, -1))
    stream, state, out = mixes(stream0, starts, slots, None)
    assert torch.equal(stream.cpu(), stream0)
    for b in range(B):
        rows = stream0[starts[b]:starts[b + 1]].double()
        before = plain.shifted(rows, state0[slots[b]].double())
        for m in range(M):
            close(out[m, starts[b]:starts[b + 1]], rows + (before - rows) * mu[m].double(), dtype, f"mix {m} of {b}", tol=tight)
        assert torch.equal(state[slots[b]].cpu(), stream0[starts[b + 1] - 1])
    assert torch.equal(state[0].cpu(), state0[0])
    stream, state, out = mixes(stream0[:B], list(range(B + 1)), slots, (delta[:B].cuda(),) + term[1:])
    close(stream, total[:B], "float32", "stream of single tokens", tol=1e-6)
    for b in range(B):
        for m in range(M):
            close(out[m, b], total[b] + (state0[slots[b]].double() - total[b]) * mu[m].double(), dtype, f"single {m}", tol=tight)
        assert torch.equal(state[slots[b]].cpu(), stream[b].cpu())


def test_a_term_does_not_go_into_a_portion_that_its_neighbours_read():
    from qwen3_from_scratch_b200.kernels import ops
    W, x = 8, torch.zeros(3, 8, device="cuda")
    args = (torch.zeros(5, W, device="cuda"), torch.zeros(2, W, device="cuda"), ints(0, 3), ints(0, 0, 0), ints(1), 1,
            torch.zeros(5, 3, W, device="cuda"), ints(0))
    with pytest.raises(ops.KernelSizeError):
        ops.sum_mix(x, (x, None, 1.0), 0.0, *args)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims,own", [(6, 2, 24, 40, 10, True), (4, 4, 17, 9, 6, True), (8, 2, 128, 64, 128, True),
                                                              (3, 1, 300, 500, 0, True), (8, 2, 128, 64, 32, False), (1, 1, 16, 8, 2, True)])
def test_biases_norms_per_head_rotation_and_pages(heads, kv_heads, dim, vdim, dims, own, dtype):
    from qwen3_from_scratch_b200.kernels import ops
    g = torch.Generator().manual_seed(heads + dim)
    T, page, pages, base, eps = 9, 4, 5, 300.0, 1e-4
    columns = heads * dim + (kv_heads * (dim + vdim) if own else 0)
    proj = torch.randn(T, columns + 8, generator=g).to(DT[dtype])
    bias = torch.randn(columns, generator=g)
    wq, wk = 1 + 0.2 * torch.randn(dim, generator=g), 1 + 0.2 * torch.randn(dim, generator=g)
    rot = {"base": base, "dims": dims, "scaling": {"factor": 4.0, "low": 0.5, "high": 6.0, "original": 60}}
    pos, table = [0, 1, 2, 3, 4, 11, 0, 1, 7], [[3, 1, 0], [2, 4, -1]]
    seq = [0] * 6 + [1] * 3
    q = torch.empty(T, heads, dim, dtype=DT[dtype], device="cuda")
    kp = torch.full((pages, kv_heads, page, dim), 9.0, dtype=DT[dtype], device="cuda")
    vp = torch.full((pages, kv_heads, page, vdim), 9.0, dtype=DT[dtype], device="cuda")
    status = ints(0)
    k_col, v_col = (4 + heads * dim, 4 + (heads + kv_heads) * dim) if own else (None, None)
    ops.head_qkv_post(proj.cuda(), 4, k_col, v_col, heads, kv_heads, dim, vdim, bias.cuda(), wq.cuda(), wk.cuda() if own else None,
                      eps, dims, plain.frequencies(rot).float().cuda(), 1.0, ints(*pos), ints(*seq), torch.tensor(table, dtype=torch.int32).cuda(),
                      q, kp, vp, status)
    assert int(status.item()) == 0
    x = proj[:, 4:4 + columns].double() + bias.double()
    tight = 1e-5 if dtype == "float32" else 8e-3
    head = lambda v, w: plain.rotate_halves(plain.unit_rms(v, eps) * w.double(), pos, rot)  # noqa: E731
    close(q, head(x[:, :heads * dim].view(T, heads, dim), wq), dtype, "queries", tol=tight)
    if not own:
        assert float(kp.float().min()) == float(vp.float().min()) == 9.0
        return
    k = head(x[:, heads * dim:(heads + kv_heads) * dim].reshape(T, kv_heads, dim), wk)
    v = x[:, (heads + kv_heads) * dim:].reshape(T, kv_heads, vdim)
    for t in range(T):
        p, at = table[seq[t]][pos[t] // page], pos[t] % page
        close(kp[p, :, at], k[t], dtype, f"key {t}", tol=tight)
        close(vp[p, :, at], v[t], dtype, f"value {t}", tol=tight)
    assert int((kp.float() == 9.0).all(dim=3).all(dim=1).sum()) == pages * page - T


class Batch:
    """The parts of a step's context that an attention kernel reads: requests with (earlier tokens, tokens of the step), those
    with a single token first."""

    def __init__(self, portions):
        self.num_seqs, self.num_decode = len(portions), sum(n == 1 for _, n in portions)
        self.max_q_len, self.max_kv_len = max(n for _, n in portions), max(past + n for past, n in portions)
        self.q_start = ints(*([0] + torch.tensor([n for _, n in portions]).cumsum(0).tolist()))
        self.kv_len = ints(*[past + n for past, n in portions])


@pytest.mark.parametrize("H,G,D,page", [(8, 2, 64, 16), (4, 1, 128, 16), (3, 3, 64, 64), (6, 2, 128, 32)])
@pytest.mark.parametrize("window", [1, 37, 128, 129, 300, 0x7fffffff])
def test_windowed_attention_of_single_tokens_and_whole_query_tiles(H, G, D, page, window):
    """The TMA-fed decode kernel and the tcgen05 portion kernel: windows that start inside a tile, at its edge and just beyond
    it, of the token itself and of everything; portions that start at the request's first token and far behind it, beside single
    tokens (the first one among them) and alone.  Pages before the windows have been given back (holes in the table),
    everything that is not a live key is NaN.  Sinks that take nearly all and nothing, or none."""
    from qwen3_from_scratch_b200.kernels import ops
    portions = [(1000, 1), (0, 1), (431, 1), (0, 300), (517, 131), (64, 64), (255, 2)]
    g = torch.Generator().manual_seed(H + D + page)
    per = -(-1001 // page)
    total = per * len(portions) + 3
    k_pages = torch.full((total, G, page, D), float("nan"), dtype=torch.bfloat16)
    v_pages = k_pages.clone()
    table = torch.full((len(portions), per), -1, dtype=torch.int32)
    ids = torch.randperm(total, generator=g).tolist()
    T = sum(n for _, n in portions)
    q = torch.randn(T, H, D, generator=g).to(torch.bfloat16)
    sink = torch.randn(H, generator=g)
    sink[0], sink[-1] = 9.0, -60.0
    scale, at = 1.7 / D ** 0.5, 0
    want = {True: torch.zeros(T, H, D, dtype=F64), False: torch.zeros(T, H, D, dtype=F64)}
    for b, (past, n) in enumerate(portions):
        k, v = (torch.randn(past + n, G, D, generator=g).to(torch.bfloat16) for _ in range(2))
        for j in range(past + n):
            if (j // page + 1) * page > past - window + 1:  # the page still holds something that the first query reads
                if table[b, j // page] < 0:
                    table[b, j // page] = ids.pop()
                k_pages[table[b, j // page], :, j % page], v_pages[table[b, j // page], :, j % page] = k[j], v[j]
        back = torch.arange(past, past + n)[:, None] - torch.arange(past + n)[None, :]
        seen = (back >= 0) & (back < window)
        for h in range(H):
            s = (q[at:at + n, h].double() @ k[:, h * G // H].double().t() * scale).masked_fill(~seen, -float("inf"))
            for taken in (True, False):
                extra = sink[h].double() if taken else torch.tensor(-float("inf"), dtype=F64)
                top = torch.maximum(s.max(dim=1).values, extra)[:, None]
                e = torch.exp(s - top)
                want[taken][at:at + n, h] = e @ v[:, h * G // H].double() / (e.sum(1, keepdim=True) + torch.exp(extra - top))
        at += n
    kd, vd, td = k_pages.cuda(), v_pages.cuda(), table.cuda()
    partial = torch.full((ops.decode_partial_numel(len(portions), H, D),), float("nan"), device="cuda")
    singles = sum(n == 1 for _, n in portions)
    for rows, keep in ((slice(0, len(portions)), slice(0, T)), (slice(0, singles), slice(0, singles)),
                       (slice(singles, len(portions)), slice(singles, T))):
        ctx, qd = Batch(portions[rows]), q[keep].contiguous().cuda()
        for taken in (True, False):
            out = torch.full((qd.shape[0], H * D), 7.0, dtype=torch.bfloat16, device="cuda")
            status = ints(0)
            assert ops.window_attention_takes(qd, kd, vd, out, ctx, scale)
            ops.window_attention(qd, kd, vd, out, ctx, td[rows].contiguous(), window, scale, sink.cuda() if taken else None, status, partial)
            assert int(status.item()) == 0
            expected = want[taken][keep]
            close(out, expected.reshape(-1, H * D), "bfloat16", f"attention {rows} {taken}", tol=1e-2)
            close(out.view(-1, H, D)[:, 0], expected[:, 0], "bfloat16", "a head whose sink takes nearly all", tol=1e-2)
    short = Batch([(9, 1), (5, 128 * G // H - 1)])
    assert not ops.window_attention_takes(qd, kd, vd, out, short, scale) and not ops.window_attention_takes(qd, kd, vd, out, ctx, -scale)
    assert not ops.window_attention_takes(qd.float(), kd, vd, out, ctx, scale)


@pytest.mark.parametrize("W,E,top,shared", [(2048, 16, 3, True), (40, 7, 2, False), (72, 8, 8, True), (256, 39, 4, True), (136, 1, 1, False),
                                            (33, 12, 3, True), (64, 60, 5, True)])
@pytest.mark.parametrize("rows", [1, 16, 70, 600])
@pytest.mark.parametrize("dtype", list(DT))
def test_router_with_a_bias_and_the_shared_experts_row(W, E, top, shared, rows, dtype):
    """Logits with a bias, a softmax over the chosen ones, the shared expert's share from one more row: on the tensor cores in
    bfloat16 (weights with all the bits of a float32), otherwise lane by lane; a token's result bit for bit the same whatever
    else is in the step."""
    from qwen3_from_scratch_b200.kernels import ops
    g = torch.Generator().manual_seed(W + E + rows)
    h = torch.randn(rows, W, generator=g).to(DT[dtype])
    router, bias = torch.randn(E + shared, W, generator=g) * (3.0 / W ** 0.5), torch.randn(E, generator=g)
    rd, bd = router.cuda(), bias.cuda()

    def route(x):
        n = x.shape[0]
        ids, wts = torch.full((n, top), -1, dtype=torch.int32, device="cuda"), torch.zeros(n, top, device="cuda")
        share = torch.zeros(n, device="cuda") if shared else None
        ops.moe_route(x.contiguous().cuda(), rd, None, ids, wts, 1.0, "softmax", 1, 1, True, logit_bias=bd, share=share)
        return ids.cpu(), wts.cpu(), share.cpu() if shared else torch.zeros(n)

    ids, wts, share = route(h)
    z = h.double() @ router[:E].double().t() + bias.double()
    clear = 0
    for t in range(min(rows, 100)):
        s = z[t].sort(descending=True).values
        if E > 1 and float((s[:-1] - s[1:]).min()) < 1e-5:
            continue
        clear += 1
        chosen, weights = plain.route(z[t], top)
        assert ids[t].tolist() == chosen, t
        close(wts[t], weights, "float32", f"weights of row {t}", tol=2e-5)
    assert clear > 0.8 * min(rows, 100)
    if shared:
        close(share, plain.sigmoid(h.double() @ router[E].double()), "float32", "shares", tol=1e-5)
    for lo, hi in ((0, 1), (rows // 2, rows // 2 + 2)):
        assert all(torch.equal(a, b[lo:hi]) for a, b in zip(route(h[lo:hi]), (ids, wts, share)))


@pytest.mark.parametrize("T,C,R", [(1, 24, 5), (7, 72, 1), (33, 130, 37), (3, 2048, 64), (100, 64, 96), (700, 200, 64)])
def test_decays_of_a_low_rank_projection(T, C, R):
    from qwen3_from_scratch_b200.kernels import ops
    g = torch.Generator().manual_seed(C)
    low, w2, w0 = torch.randn(T, R + 3, generator=g), torch.randn(C, R, generator=g), 3 * torch.randn(C, generator=g)
    w0[0], w0[1] = 30.0, -30.0  # gone at once; kept for good
    out = torch.empty(T, C, device="cuda")
    ops.low_rank_decay(low.cuda(), w2.t().contiguous().cuda(), w0.cuda(), out)
    want = -torch.exp(torch.tanh(low[:, :R].double()) @ w2.double().t() + w0.double())
    assert torch.allclose(out.cpu().double(), want.clamp(min=-104.0), rtol=1e-4, atol=0)


@pytest.mark.parametrize("activation", ["gelu_tanh", "limited", "silu", "relu"])
@pytest.mark.parametrize("bias", [True, False])
@pytest.mark.parametrize("width,ff,rows", [(40, 20, 5), (64, 72, 3), (64, 72, 16), (136, 40, 90), (256, 384, 300), (512, 1024, 1100)])
@pytest.mark.parametrize("dtype", list(DT))
def test_gated_feed_forward_with_biases(width, ff, rows, activation, bias, dtype):
    """Few rows, the tcgen05 products' epilogues (single and by pairs), the library's product and the gate's kernel; the
    last bias is left open."""
    from qwen3_from_scratch_b200.parts.base import Runtime
    if dtype == "float32" and rows > 100:
        rows = 60
    names = {"gate": "gate", "up": "up", "down": "down", "gate_bias": "gate.b", "up_bias": "up.b", "down_bias": "down.b"}
    p = part("feed_forward", "gated_mlp", {"hidden_size": width, "intermediate_size": ff, "activation": activation, "bias": bias,
                                           "limit": 0.8, "names": names})
    dev, ref = part_weights(p, dtype, seed=width + rows)
    p.setup(Runtime(torch.device("cuda:0"), DT[dtype], 1200, 2), dict(dev))
    x = torch.randn(rows, width, generator=torch.Generator().manual_seed(rows)).to(DT[dtype])
    h = x.double()
    gate, up = (plain.linear(h, ref[s], ref.get(s + ".b")) for s in ("gate", "up"))
    if activation == "limited":
        gate, up = gate.clamp(max=0.8), up.clamp(-0.8, 0.8)
        mid = gate * plain.sigmoid(1.702 * gate) * (up + 1)
    else:
        mid = {"gelu_tanh": plain.gelu_tanh, "silu": plain.silu, "relu": lambda z: z.clamp(min=0)}[activation](gate) * up
    want = plain.linear(mid, ref["down"], ref.get("down.b"))
    got = p.forward(x.cuda())
    assert torch.is_tensor(got) != bias
    close(whole_output(got), want, dtype, activation, tol=None if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("rows", [1, 7, 16, 40])
@pytest.mark.parametrize("sizes,width", [([48, 48, 48, 48], 64), ([24, 24], 40), ([32, 16, 8], 72)])
def test_projections_side_by_side(sizes, width, rows, dtype):
    from qwen3_from_scratch_b200.parts.base import Runtime
    from qwen3_from_scratch_b200.parts.linear import GroupedLinear
    g = torch.Generator().manual_seed(width + rows)
    weights = [(torch.randn(n, width, generator=g) / width ** 0.5).to(DT[dtype]) for n in sizes]
    layer = GroupedLinear([w.cuda() for w in weights], Runtime(torch.device("cuda:0"), DT[dtype], 64, 2), "t")
    x = torch.randn(len(sizes), rows, width, generator=g).to(DT[dtype])
    want = torch.cat([x[i].double() @ w.double().t() for i, w in enumerate(weights)], dim=1)
    close(layer(x.cuda()), want, dtype, "side by side", tol=2e-6 if dtype == "float32" else 8e-3)


# ---------------------------------------------------------------------- each mechanism alone
ATTENTION = {"hidden_size": 40, "num_heads": 6, "num_kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.3, "window": 13, "gate": False,
             "fixed_sink": 0.0, "proj_bias": True, "qk_norm_eps": 1e-5}
MIXING = {"hidden_size": 40, "num_heads": 3, "dim": 24, "norm_eps": 1e-5, "rank": 6}
SCALING = {"factor": 4.0, "low": 0.5, "high": 6.0, "original": 60}


def rotated(p, dims, base=500.0, scaling=SCALING, **more):
    from qwen3_from_scratch_b200.parts.base import PartSpec
    return dict(p, position=PartSpec("rotary_banded", {"dims": dims, "base": base, "scaling": scaling}), **more)


def attention_config(p):
    pos = p["position"].params
    return {"heads": p["num_heads"], "kv_heads": p["num_kv_heads"], "dim": p["dim"], "vdim": p["vdim"], "scale": p["scale"],
            "mask": {"size": p["window"]}, "rot": {"base": pos["base"], "dims": pos["dims"], "scaling": pos["scaling"]}}


def plain_attention(p):
    m = attention_config(p)

    def fn(h, ref, st):
        st = st or {"k": torch.zeros(0, m["kv_heads"], m["dim"], dtype=F64), "v": torch.zeros(0, m["kv_heads"], m["vdim"], dtype=F64)}
        start = st["k"].shape[0]
        return plain.attention(h, ref, "", m, p["qk_norm_eps"], list(range(start, start + h.shape[0])), st), st
    return fn


def plain_mixing(p):
    H, D = p["num_heads"], p["dim"]

    def fn(h, ref, st):
        st = st or {"S": torch.zeros(H, D, D, dtype=F64), "h": torch.zeros(p["hidden_size"], dtype=F64)}
        return plain.time_mixing(h, ref, "", {"heads": H, "dim": D}, p["norm_eps"], st), st
    return fn


def decays(low, high):
    """A tweak: the decays' offsets spread evenly between two numbers (log(-log w))."""
    def tweak(dev, ref):
        n = ref["w0"].numel()
        w0 = torch.linspace(low, high, n)[torch.randperm(n, generator=torch.Generator().manual_seed(1))].to(torch.bfloat16)
        dev["m.w0"], ref["w0"] = w0.float().cuda(), w0.double()
    return tweak


def mixer_cases():
    for name, p in (("attention, partly rotated", rotated(ATTENTION, 10)),
                    ("attention, one head, a window of the token itself", rotated(dict(ATTENTION, num_heads=1, num_kv_heads=1, window=1, vdim=16), 0)),
                    ("attention, one head, odd sizes, a window of two", rotated(dict(ATTENTION, num_heads=1, num_kv_heads=1, dim=17, vdim=9, window=2), 4, scaling=None)),
                    ("attention of sizes for the tensor cores", rotated(dict(ATTENTION, num_heads=8, dim=64, vdim=32, window=50, scale=0.2), 64)),
                    ("attention over everything there is", rotated(dict(ATTENTION, num_heads=4, dim=32, vdim=64, window=1000, scale=0.2), 16))):
        yield name, "kept_window_attention", p, plain_attention(p), None
    for name, p, tweak in (("time mixing", dict(MIXING), decays(-6.0, 0.5)),
                           ("time mixing, one head of an odd size, rank one", dict(MIXING, num_heads=1, dim=17, rank=1), decays(-3.0, 1.0)),
                           ("time mixing of wide keys", dict(MIXING, num_heads=2, dim=200, rank=40), decays(-7.0, 0.0)),
                           ("time mixing of heads of 32", dict(MIXING, num_heads=4, dim=32), decays(-7.0, 2.0)),
                           ("time mixing of heads of 64", dict(MIXING, num_heads=2, dim=64), decays(-7.0, 3.5)),
                           ("time mixing of heads of 128", dict(MIXING, num_heads=1, dim=128), decays(-8.0, 1.0))):
        yield name, "time_mixing", p, plain_mixing(p), tweak


CASES = {name: rest for name, *rest in mixer_cases()}


def moved_by_rounding(fn, x, ref, want):
    """What rounding the projections' operands and results to bfloat16 alone does in the plain implementation, relative to
    the largest value."""
    with plain.bfloat16_projections():
        rounded = fn(x.double(), ref, None)[0]
    return float((rounded - want).abs().max() / want.abs().max())


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("case", list(CASES))
def test_mixer_alone_whole_in_portions_and_beside_another_request(case, dtype):
    """A mixer on random rows: a request whole; then the same in portions down to two tokens and single tokens, beside
    another request whose portions start and end elsewhere, in slots and pages that were used before."""
    kind, params, fn, tweak = CASES[case]
    p = part("mixer", kind, params)
    bench = MixerBench(p, dtype, page_size=4, pages=96, max_tokens=256, seed=11, tweak=tweak)
    g = torch.Generator().manual_seed(12)
    x_of = {r: torch.randn(n, params["hidden_size"], generator=g).to(DT[dtype]) for r, n in (("a", 175), ("b", 31), ("c", 9))}
    want = {r: fn(x.double(), bench.ref, None)[0] for r, x in x_of.items()}
    call = lambda rows, ctx: whole_output(p.forward(rows.cuda().contiguous(), ctx, 0, True))  # noqa: E731
    tol = None
    if dtype == "bfloat16":
        tol = max(3e-2, 3 * max(moved_by_rounding(fn, x, bench.ref, want[r]) for r, x in x_of.items()))
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
@pytest.mark.parametrize("dim,vdim,heads,kv_heads,window", [(16, 24, 2, 1, 9), (32, 64, 6, 2, 64), (64, 32, 3, 3, 37), (128, 128, 4, 1, 130),
                                                            (64, 64, 12, 3, 101)])
def test_a_key_just_inside_and_just_outside_the_window_shows(dim, vdim, heads, kv_heads, window, dtype):
    """One token whose key answers every query and whose value stands out: the last position that its window reaches still
    gives its value, the next one nothing of it; a window one longer or shorter would be far off.  Tokens at a page's first and
    last place and the request's first among them; as a whole prompt, with portions that end at the edge, and decoded."""
    params = rotated(dict(ATTENTION, hidden_size=32, num_heads=heads, num_kv_heads=kv_heads, dim=dim, vdim=vdim, scale=1.5 / dim,
                          window=window), 0)

    def tweak(dev, ref):  # queries and keys from the biases alone but for the first feature, which turns a key towards them
        for tensors, pre in ((dev, "m."), (ref, "")):
            one = lambda n: torch.where(torch.arange(n) % dim < dim // 2, 1.0, -1.0)  # noqa: E731
            tensors[pre + "q"].zero_(), tensors[pre + "k"].zero_()
            tensors[pre + "q.b"].copy_(one(heads * dim)), tensors[pre + "k.b"].copy_(-one(kv_heads * dim))
            tensors[pre + "k"][:, 0] = 2 * one(kv_heads * dim).to(tensors[pre + "k"])
            tensors[pre + "q.norm"].fill_(2.0), tensors[pre + "k.norm"].fill_(1.5)

    p = part("mixer", "kept_window_attention", params)
    fn = plain_attention(params)
    n = window + 40
    for at in (0, 7, 16):
        bench = MixerBench(p, dtype, page_size=8, pages=64, max_tokens=256, seed=31, tweak=tweak)
        x = 0.3 * torch.randn(n, 32, generator=torch.Generator().manual_seed(32 + at))
        x[:, 0] = 0
        x[at] = 3 * torch.randn(32, generator=torch.Generator().manual_seed(33))
        x[at, 0] = 1.0
        x = x.to(DT[dtype])
        want = fn(x.double(), bench.ref, None)[0]
        tol = 2e-5 if dtype == "float32" else 2e-2
        for other in (window - 1, window + 1):
            moved = (plain_attention(dict(params, window=other))(x.double(), bench.ref, None)[0] - want).abs().max(dim=1).values
            edge = at + min(window, other)
            assert float(moved[edge]) > 5 * tol * float(want.abs().max()), "the edge shows"
        call = lambda r, ctx: whole_output(p.forward(r.cuda().contiguous(), ctx, 0, True))  # noqa: E731
        close(bench.run([("r", n)], {"r": x}, call)["r"], want, dtype, f"{at} whole", tol)
        bench.manager.close("r")
        for cuts in ([at + window - 1, 2, n - at - window - 1], [at + window, 1, 2] + [1] * (n - at - window - 3),
                     [at + 1] + [1] * (n - at - 1)):
            close(torch.cat([bench.run([("r", c)], {"r": x}, call)["r"] for c in cuts]), want, dtype, f"{at} in {cuts[:3]}", tol)
            bench.manager.close("r")


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("dim,vdim", [(16, 24), (64, 64)])
def test_the_one_in_the_denominator(dim, vdim, dtype):
    """Scores far below zero: the sink takes nearly everything; near zero: its share of one among the window's tokens; the
    first token, alone in its window, gives e^s / (1 + e^s) of its value."""
    for scale in (-3.0, 0.0, 0.5):
        params = rotated(dict(ATTENTION, hidden_size=32, num_heads=4, num_kv_heads=2, dim=dim, vdim=vdim, scale=scale, window=20), 0)

        def tweak(dev, ref):  # every query and key the same: the score is scale * dim at every pair
            for tensors, pre in ((dev, "m."), (ref, "")):
                for t in ("q", "k"):
                    tensors[pre + t].zero_(), tensors[pre + t + ".b"].fill_(2.0), tensors[pre + t + ".norm"].fill_(1.0 / dim ** 0.5)

        p = part("mixer", "kept_window_attention", params)
        bench = MixerBench(p, dtype, page_size=4, pages=32, max_tokens=64, seed=3, tweak=tweak)
        x = torch.randn(50, 32, generator=torch.Generator().manual_seed(4)).to(DT[dtype])
        want = plain_attention(params)(x.double(), bench.ref, None)[0]
        v = plain.linear(x.double(), bench.ref["v"], bench.ref["v.b"]).view(50, 2, vdim)[0].repeat_interleave(2, dim=0).reshape(1, -1)
        first = v / (1 + np.exp(-scale)) @ bench.ref["o"].t() + bench.ref["o.b"]
        assert torch.allclose(want[:1], first, atol=1e-4 * float(first.abs().max()))
        call = lambda r, ctx: whole_output(p.forward(r.cuda().contiguous(), ctx, 0, True))  # noqa: E731
        for cuts in ([50], [1, 2, 20, 1, 26]):
            close(torch.cat([bench.run([("r", c)], {"r": x}, call)["r"] for c in cuts]), want, dtype, f"{scale} {cuts}")
            bench.manager.close("r")


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("dim", [24, 32, 64, 128])
def test_a_slow_decay_carries_the_first_token_to_the_end(dim, dtype):
    """Decays near one and a first token that writes the memory: what it wrote is still most of the output hundreds of
    tokens later, through portions and single tokens and beside another request's tokens."""
    params = dict(MIXING, hidden_size=32, num_heads=2, dim=dim)
    fn, p = plain_mixing(params), part("mixer", "time_mixing", params)

    def tweak(dev, ref):
        for tensors, pre in ((dev, "m."), (ref, "")):
            tensors[pre + "w0"].fill_(-8.0), tensors[pre + "w2"].mul_(0.1)
            for s in "rkvgw":
                tensors[pre + "mu." + s].mul_(0.2)

    n = 400
    bench = MixerBench(p, dtype, page_size=8, pages=8, max_tokens=512, seed=51, tweak=tweak)
    g = torch.Generator().manual_seed(52)
    x = 0.02 * torch.randn(n, 32, generator=g)
    x[0] = 6 * torch.randn(32, generator=g)
    x_of = {"r": x.to(DT[dtype]), "o": torch.randn(9, 32, generator=g).to(DT[dtype])}
    want = fn(x_of["r"].double(), bench.ref, None)[0]
    quiet = x_of["r"].clone()
    quiet[0] = 0
    moved = (want - fn(quiet.double(), bench.ref, None)[0])[-50:].abs().max()
    assert float(moved) > 0.3 * float(want[-50:].abs().max())

    def check(got, what):
        """Without the first rows, which are so much larger that they would hide the others.  bfloat16: a receptance that turns
        past the stored key reads a small difference of large terms, whose sign rounding decides; one row in twenty may."""
        if dtype == "float32":
            close(got[2:], want[2:], dtype, what, 1e-4)
            return
        err = (got[2:].double().cpu() - want[2:]).abs().max(dim=1).values / want[2:].abs().max()
        assert float((err > 4e-2).float().mean()) < 0.05 and float(err.median()) < 1e-2, what

    call = lambda rows, ctx: p.forward(rows.cuda().contiguous(), ctx, 0, True)  # noqa: E731
    check(bench.run([("r", n)], x_of, call)["r"], "whole")
    bench.manager.close("r")
    got = []
    for step in ([("r", 1)], [("r", 2), ("o", 4)], [("r", 290)], [("o", 1), ("r", 1)], [("r", 2)], [("r", 64), ("o", 4)]) \
            + tuple([("r", 1)] for _ in range(40)):
        got.append(bench.run(list(step), x_of, call)["r"])
    check(torch.cat(got), "portions")


def _memory(rows, logw, bonus, H, D, lens, state, matrix):
    """One step of ``ops.channel_memory_scan`` on rows of several requests, by the walk or in the matrix form: (o, state)."""
    from qwen3_from_scratch_b200.kernels import ops
    B, T = len(lens), sum(lens)
    q_start = torch.tensor([0] + torch.tensor(lens).cumsum(0).tolist(), dtype=torch.int32).cuda()
    out, status = torch.full((T, H * D), float("nan"), device="cuda"), ints(0)
    st, scratch = state.clone(), None
    if matrix:
        alloc = lambda tag, *s, dtype: torch.full(s, float("nan"), dtype=dtype, device="cuda")  # noqa: E731
        scratch = ops.ChannelScratch(alloc, T, B, H, D)
    ops.channel_memory_scan(rows, 0, H * D, 2 * H * D, ops.ChannelDecay(logw, bonus), st, q_start, ints(*range(B, 0, -1)), B, out,
                            status, max_q_len=max(lens), scratch=scratch)
    assert int(status.item()) == 0
    return out, st


@pytest.mark.parametrize("H,D", [(3, 32), (2, 64), (2, 128), (5, 64)])
@pytest.mark.parametrize("lens", [[64], [200], [1, 64, 65, 130, 3], [2, 500, 1, 33, 16, 17]])
def test_matrix_form_equals_the_walk_and_the_walk_the_plain_recurrence(H, D, lens):
    """The tensor-core form against the token-by-token walk on the same bfloat16 rows, from states that are not empty, scratch
    filled with NaN: portions that end inside a chunk or one of its parts, at an edge and just beyond, single tokens beside
    them; decays from none to total, slow ones right behind total ones in the same channel.  They differ by float32 rounding
    and what two bfloat16 halves lose (2^-16)."""
    from qwen3_from_scratch_b200.kernels import ops
    assert ops.channel_matrix_form(torch.bfloat16, D, D) and not ops.channel_matrix_form(torch.float32, D, D)
    assert not ops.channel_matrix_form(torch.bfloat16, 48, 48)
    g = torch.Generator().manual_seed(H + D + sum(lens))
    T, B = sum(lens), len(lens)
    state = 0.3 * torch.randn(B + 1, H, D, D, generator=g).cuda()
    rows = (0.5 * torch.randn(T, 3 * H * D + 8, generator=g)).to(torch.bfloat16).cuda()
    bonus = torch.randn(H, D, generator=g).cuda()
    for low, high, sudden in ((-9.0, -2.0, 0.0), (-4.0, 2.0, 0.0), (-7.0, -4.0, 0.1), (0.0, 4.6, 0.0)):
        logw = -torch.exp(low + (high - low) * torch.rand(T, H * D, generator=g))
        logw = torch.where(torch.rand(T, H * D, generator=g) < sudden, torch.tensor(-104.0), logw).clamp(min=-104.0).cuda()
        a, sa = _memory(rows, logw, bonus, H, D, lens, state, False)
        b, sb = _memory(rows, logw, bonus, H, D, lens, state, True)
        close(b, a, "float32", f"{low} {high} {sudden}", tol=5e-5)
        close(sb, sa, "float32", f"{low} {high} {sudden}: state", tol=5e-5)
        at = 0
        for i, n in enumerate(lens[:3]):
            r, k, v = (rows[at:at + n, s * H * D:(s + 1) * H * D].double().cpu().view(n, H, D) for s in range(3))
            o, S = plain.time_mixing_memory(r, k, v, logw[at:at + n].double().cpu().view(n, H, D), bonus.double().cpu(),
                                            state[B - i].double().cpu().transpose(1, 2))
            close(a[at:at + n], o.reshape(n, H * D), "float32", f"walk {i}", tol=1e-5)
            close(sa[B - i].transpose(1, 2), S, "float32", f"walk {i}: state", tol=1e-5)
            at += n


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("W,E,top,ff,shared,rows", [(40, 12, 3, 24, (40, 0.9), 3), (40, 12, 3, 24, None, 23), (64, 3, 3, 20, (16, 0.5), 40),
                                                    (128, 8, 2, 48, (64, 1.2), 300), (136, 40, 4, 16, (8, 0.7), 1100), (48, 1, 1, 32, (24, 1.0), 9),
                                                    (33, 5, 2, 16, (9, 0.8), 6)])
def test_limited_experts_beside_a_gated_shared_one(W, E, top, ff, shared, rows, dtype):
    """A pair at a time (few tokens, float32, inner widths that are no multiple of 16) and as grouped products; a biased
    router, a softmax over the chosen logits, the shared expert's share per token."""
    from qwen3_from_scratch_b200.parts.base import PartSpec, Runtime
    names = {"gate": "gate", "up": "up", "down": "down"}
    spec = None if shared is None else PartSpec("gated_mlp", {"hidden_size": W, "intermediate_size": shared[0], "activation": "limited",
                                                              "limit": shared[1], "names": names})
    p = part("feed_forward", "routed_experts", {
        "hidden_size": W, "experts": E, "top": top, "expert_ff": ff, "activation": "limited", "limit": 0.8, "correction": False,
        "gated": True, "score": "softmax", "renormalise": True, "router_bias": True, "shared": spec, "shared_gate": shared is not None})
    dev, ref = part_weights(p, dtype, seed=W + rows, scale={"router": 4.0 / W ** 0.5})
    p.setup(Runtime(torch.device("cuda:0"), DT[dtype], 1200, 2), dict(dev))
    x = torch.randn(rows, W, generator=torch.Generator().manual_seed(rows)).to(DT[dtype])
    mlp = {"router": {"experts": E, "top": top}, "expert": {"limit": 0.8}}
    if shared is not None:
        mlp["shared"] = {"ff": shared[0], "limit": shared[1]}
    keep_rows = min(rows, 60)
    want = plain.experts(x[:keep_rows].double(), ref, "", mlp)
    got = p.forward(x.cuda())[:keep_rows]
    # a near tie of two logits may fall the other way (in float32 too, against float64); such rows are left out
    z = (x[:keep_rows].double() @ ref["router"].t() + ref["router.b"]).sort(dim=1, descending=True).values
    clear = (z[:, :-1] - z[:, 1:]).min(dim=1).values > 1e-5 if E > 1 else torch.ones(keep_rows, dtype=torch.bool)
    assert clear.float().mean() > 0.9
    close(got[clear], want[clear], dtype, "experts", tol=None if dtype == "float32" else 3e-2)


@pytest.mark.parametrize("dtype", list(DT))
def test_two_layers_on_the_keys_of_one(dtype):
    """A layer with keys of its own and one with queries, a scale and a wider window of its own that reads them: the pages
    are kept as far back as the reader looks, and the reader writes none."""
    from qwen3_from_scratch_b200.engine.model import shared_need
    params = rotated(dict(ATTENTION, window=10), 8)
    reading = rotated(dict(ATTENTION, window=33, scale=0.45), 8, shares_kv=True)
    a, b = part("mixer", "kept_window_attention", params), part("mixer", "kept_window_attention", reading)
    assert not any(".k" in s.name or ".v" in s.name for s in b.weight_specs())
    a.cache_spec = lambda own=a.cache_spec: shared_need(own(), b.cache_spec())
    bench = MixerBench(a, dtype, page_size=4, pages=20, max_tokens=64, seed=61, max_seqs=1)
    dev, ref = part_weights(b, dtype, 62)
    b.setup(bench.rt, dict(dev))
    n = 120
    x = torch.randn(n, 40, generator=torch.Generator().manual_seed(63)).to(DT[dtype])
    st = {"k": torch.zeros(0, 2, 24, dtype=F64), "v": torch.zeros(0, 2, 40, dtype=F64)}
    eps, pos = 1e-5, list(range(n))
    want = torch.cat([plain.attention(x.double(), bench.ref, "", attention_config(params), eps, pos, st),
                      plain.attention(x.double(), ref, "", dict(attention_config(reading), kv_from=0), eps, pos, st)], dim=1)

    def call(rows, ctx):
        h = rows.cuda().contiguous()
        first = whole_output(a.forward(h, ctx, 0, True)).clone()
        with pytest.raises(ValueError, match="of its own to write"):
            b.forward(h, ctx, 0, True)
        return torch.cat([first, whole_output(b.forward(h, ctx, 0, False))], dim=1)

    got = torch.cat([bench.run([("r", c)], {"r": x}, call)["r"] for c in [20, 1, 2, 15, 1, 1, 30] + [1] * 50])
    close(got, want, dtype, "both", tol=None if dtype == "float32" else 3e-2)


# ---------------------------------------------------------------------- whole models
def check_logits(got, want, dtype, what):
    """float32: every position within 1e-4 of the largest logit: every memory's read-out, a sum with cancellation, is brought
    to unit size by the norm behind it, and so is every sub-layer's output, which hands on the float32 rounding of the sums.
    bfloat16: half of a request's positions within 2e-2, nine in ten (or all but three) within 5e-2.  At the others rounding
    alone goes farther in the plain implementation too (up to 0.2: a read-out that is a small difference of large terms, a
    choice of experts that turns over, and what follows one in the memories); a wrong key, state or page moves far more
    positions than those."""
    if dtype == "float32":
        assert_close(got, want, dtype, what, tol=1e-4)
        return
    for req, w in want.items():
        g = got[req].double()
        assert g.shape == w.shape and torch.isfinite(g).all(), f"{what}: request {req}"
        err = (g - w).abs().max(dim=-1).values / float(w.abs().max())
        over = (err > 5e-2).nonzero().flatten().tolist()
        assert float(err.median()) <= 2e-2, f"{what}: request {req}: median error {float(err.median()):.3g}"
        assert len(over) <= max(3, 0.1 * len(err)), f"{what}: request {req}: beyond 5e-2 at {over}"
        assert float(err.max()) < 0.6, f"{what}: request {req}: {float(err.max()):.3g} at {int(err.argmax())}"


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
    n = 90 if key != "z" else 180
    ids = tokens(cfg["vocab"], n, 51)
    want = {"a": plain.forward_logits(cfg, w, ids)}

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
        check_logits(replay(folders[key], dtype, {"a": ids}, schedule), want, dtype, f"{key} {name}")


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
    check_logits(got, want, dtype, f"{key} mixed")


def test_long_prompt_on_the_serving_kernels(folders):
    """bfloat16 at the serving kernels' sizes with pages of 16: a prompt of 700 tokens whole and cut into long and short
    portions with single tokens between them; then a batch of a long portion beside single tokens."""
    cfg, w = plain.read_model_folder(folders["z"])
    ids, other = tokens(cfg["vocab"], 700, 77), tokens(cfg["vocab"], 90, 78)
    want = {"a": plain.forward_logits(cfg, w, ids), "b": plain.forward_logits(cfg, w, other)}
    for name, cuts in (("whole", [700]), ("portions", [300, 1, 250, 1, 1, 130, 17])):
        got = replay(folders["z"], "bfloat16", {"a": ids}, lambda r, cuts=cuts: [r.step([("a", n)]) for n in cuts],
                     page_size=16, num_pages=64, max_seqs=2, max_step_tokens=1024)
        check_logits(got, {"a": want["a"]}, "bfloat16", f"z long {name}")

    def beside(r):
        r.step([("b", 70)])
        r.step([("a", 300), ("b", 1)])
        r.step([("b", 1), ("a", 399)])
        r.step([("a", 1), ("b", 18)])

    got = replay(folders["z"], "bfloat16", {"a": ids, "b": other}, beside, page_size=16, num_pages=64, max_seqs=2,
                 max_step_tokens=1024)
    check_logits(got, want, "bfloat16", "z long beside single tokens")


@pytest.mark.parametrize("dtype", list(DT))
def test_long_decoding_through_graphs(folders, dtype):
    """300 single tokens after a short prompt, replayed from CUDA graphs: memories, last inputs and pages are carried on the
    device from step to step, every window passed many times over."""
    cfg, w = plain.read_model_folder(folders["x"])
    ids = tokens(cfg["vocab"], 310, 71)
    want = {"a": plain.forward_logits(cfg, w, ids)}

    def schedule(r):
        r.step([("a", 10)])
        for _ in range(300):
            r.step([("a", 1)])

    got = replay(folders["x"], dtype, {"a": ids}, schedule, page_size=4, num_pages=80, max_seqs=2, poison_freed_pages=True)
    check_logits(got, want, dtype, "long decoding")


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
    cfg, _ = plain.read_model_folder(folders["x"])
    prompts = [tokens(cfg["vocab"], n, 90 + i) for i, n in enumerate([30, 28, 26])]
    alone = SyncEngine(folders["x"], dtype="float32", block_size=4, num_pages=96, max_num_seqs=4, max_num_tokens=64)
    want = [alone.generate(p, max_new_tokens=24, ignore_eos=True) for p in prompts]
    tight = SyncEngine(folders["x"], dtype="float32", block_size=4, num_pages=22, max_num_seqs=4, max_num_tokens=64)
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

    def check(step, rows):
        got = torch.from_numpy(np.fromfile(os.path.join(out, f"{step}.f32"), dtype="<f4")).view(len(rows), vocab)
        check_logits({step: got}, {step: torch.stack(rows)}, dtype, "replayed")

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
