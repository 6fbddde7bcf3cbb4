"""Domelix without a GPU: its configuration, what the model asks of the weights and of the cache, the distance buckets, and
the plain implementation against itself (a prompt whole, in portions and token by token through the explicit caches and
states) and on values worked by hand."""

import copy
import math

import pytest
import torch

import plain_domelix as plain
from domelix_models import BIAS_ROWS, CONFIGS, DOMELIX_X, DOMELIX_Y, DOMELIX_Z, make_folder, tensor_shapes

F64 = plain.F64


def model_of(config):
    from qwen3_from_scratch_b200.engine.model import Model
    from qwen3_from_scratch_b200.registry import build_model_spec, config_from_dict
    return Model(build_model_spec(config_from_dict(config)))


@pytest.mark.parametrize("key", list(CONFIGS))
def test_the_model_asks_for_the_tensors_the_design_names(key):
    """Names and shapes, but for the rows of a distance bias's table, which the folder decides."""
    config = CONFIGS[key][0]
    want = tensor_shapes(config)
    specs = {s.name: s for s in model_of(config).weight_specs()}
    assert set(specs) == set(want)
    for name, shape in want.items():
        assert specs[name].takes(shape), (name, shape, specs[name].shape)
        if name.endswith(".rel"):
            assert specs[name].free_dims == (0,) and specs[name].takes((5, shape[1])) and not specs[name].takes((8, shape[1] + 1))
        else:
            assert tuple(specs[name].shape) == shape


def test_a_table_of_another_width_is_refused_and_any_number_of_rows_loads(tmp_path):
    from qwen3_from_scratch_b200.weights.loader import WeightsError, load_weights
    specs = model_of(DOMELIX_Y).weight_specs()

    def load(rows, heads):
        def tweak(t):
            t["l1.mix.left.rel"] = torch.zeros(rows, heads, dtype=torch.bfloat16)
        folder = make_folder(str(tmp_path / f"{rows}x{heads}"), DOMELIX_Y, 1, tweak)
        return load_weights(folder, specs, device="cpu", compute_dtype=torch.bfloat16)

    assert tuple(load(2, 1)["l1.mix.left.rel"].shape) == (2, 1) and tuple(load(50, 1)["l1.mix.left.rel"].shape) == (50, 1)
    with pytest.raises(WeightsError, match="l1.mix.left.rel"):
        load(2, 2)


def test_configuration_round_trip():
    from qwen3_from_scratch_b200.registry import config_from_dict
    cfg = config_from_dict(DOMELIX_X)
    assert cfg.architecture == "Domelix" and (cfg.vocab, cfg.width, cfg.norm_eps) == (211, 64, 1e-5)
    d, par, ret = cfg.layers[0], cfg.layers[1], cfg.layers[2]
    assert (d.type, d.mixer.heads, d.mixer.kv_heads, d.mixer.dim, d.mixer.vdim, d.mixer.conv) == ("delta", 4, 2, 24, 16, 3)
    left, right = par.mixer.left, par.mixer.right
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.scale, left.bias_max) == (6, 2, 24, 40, 0.2, 20)
    assert (right.heads, right.dim, right.vdim, right.decay) == (3, 16, 24, (0.0, 0.6, 1.0))
    assert (ret.mixer.rot_base, ret.mixer.rot_dims, ret.mixer.decay) == (1000.0, 12, (0.5, 0.93, 0.999)) and ret.mlp is None
    assert (d.mlp.experts, d.mlp.top, d.mlp.groups, d.mlp.keep, d.mlp.expert_ff) == (12, 3, 4, 2, 24)
    assert config_from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == DOMELIX_X


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0].update(type="hyena"), "not built"),
    (lambda c: c["layers"][0].update(mlp={"kind": "dense", "ff": 8}), "moe"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("bias_max"), "bias_max"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 0.6, 1.5]), "decay"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=22), "dims"),
    (lambda c: c["layers"][2]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=5), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].pop("groups"), "groups"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_configuration_errors_name_the_key(change, message):
    from qwen3_from_scratch_b200.config.model_config import ConfigError
    from qwen3_from_scratch_b200.registry import config_from_dict
    config = copy.deepcopy(DOMELIX_X)
    change(config)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(config)


def test_cache_needs():
    """The attention keeps pages of keys and values for good, a memory a float32 state kept column by column, the delta
    rule also the tail of its convolutions (none with a single tap)."""
    from qwen3_from_scratch_b200.parts.base import StateSpec
    layout = model_of(DOMELIX_X).cache_layout()
    groups = {tuple((p.name, p.heads, p.width) for p in g.spec.planes): (g.cache_ids, g.spec.window) for g in layout.groups}
    assert groups == {(("k", 2, 24), ("v", 2, 40)): ([(1, "left")], None), (("k", 4, 16), ("v", 4, 8)): ([(3, "left")], None)}
    assert layout.states[(0, "state")] == StateSpec((4, 16, 24), "float32")
    assert layout.states[(0, "conv")] == StateSpec((2, 2 * 48 + 64), "float32")
    assert layout.states[(1, "right")] == StateSpec((3, 24, 16), "float32")
    assert layout.states[2] == StateSpec((3, 36, 20), "float32")
    assert set(model_of(DOMELIX_Y).cache_layout().states) == {0, (1, "right"), (2, "state")}


def test_random_model_folder_through_the_framework_writer(tmp_path):
    from qwen3_from_scratch_b200.registry import config_from_dict
    from qwen3_from_scratch_b200.weights import write_random_model
    folder = write_random_model(str(tmp_path / "m"), config_from_dict(DOMELIX_Z), seed=1)
    config, w = plain.read_model_folder(folder)
    shapes = {k: tuple(v.shape) for k, v in w.items()}
    want = tensor_shapes(DOMELIX_Z)
    assert {k: v for k, v in shapes.items() if not k.endswith(".rel")} == {k: v for k, v in want.items() if not k.endswith(".rel")}
    logits = plain.forward_logits(config, w, [5, 17, 3, 250, 9])
    assert logits.shape == (5, 300) and torch.isfinite(logits).all()


@pytest.mark.parametrize("rows,most", [(8, 20), (2, 2), (16, 60), (30, 77), (32, 128), (16, 1000), (4, 2.5), (6, 3), (64, 40)])
def test_distance_buckets(rows, most):
    """The engine's table of rows by distance ends where all further distances read the last row, and says what the
    formula says up to there and beyond."""
    from qwen3_from_scratch_b200.parts.attention import distance_buckets
    table = distance_buckets(rows, most)
    assert table[0] == 0 and table[-1] == rows - 1 and (len(table) == 1 or table[-2] < rows - 1)
    assert all(a <= b for a, b in zip(table, table[1:]))
    for n in range(2 * len(table) + 50):
        if most > rows // 2:
            assert plain.bucket(n, rows, most) == table[min(n, len(table) - 1)], n
    # exactly at a boundary: most = half * 2^(rows - half) puts the edge between rows half + k and half + k - 1 at half * 2^k
    exact = distance_buckets(8, 4 * 2 ** 4)
    assert [exact.index(b) for b in range(8)] == [0, 1, 2, 3, 4, 8, 16, 32] and len(exact) == 33


@pytest.mark.parametrize("key", list(CONFIGS))
def test_plain_whole_prompt_equals_plain_in_portions_and_token_by_token(tmp_path, key):
    config, seed = CONFIGS[key]
    cfg, w = plain.read_model_folder(make_folder(str(tmp_path / key), config, seed))
    ids = torch.randint(0, cfg["vocab"], (70,), generator=torch.Generator().manual_seed(7)).tolist()
    whole = plain.forward_logits(cfg, w, ids)
    for cuts in ([30, 2, 1, 37], [1] * 70, [2] * 35):
        state, rows, at = plain.new_state(cfg), [], 0
        for c in cuts:
            rows.append(plain.forward(cfg, w, ids[at:at + c], state))
            at += c
        assert float((torch.cat(rows) - whole).abs().max()) < 1e-9 * float(whole.abs().max())


@pytest.mark.parametrize("key", list(CONFIGS))
def test_every_tensor_moves_the_logits(tmp_path, key):
    """The test weights hide nothing: whatever tensor is disturbed, the logits change (an expert's only if it is chosen)."""
    config, seed = CONFIGS[key]
    cfg, w = plain.read_model_folder(make_folder(str(tmp_path / key), config, seed))
    ids = torch.randint(0, cfg["vocab"], (24,), generator=torch.Generator().manual_seed(8)).tolist()
    base = plain.forward_logits(cfg, w, ids)
    for name in w:
        if ".mlp.e" in name or (name.endswith("router") and w[name].shape[0] == 1):
            continue
        if name.endswith("sink") and w[name].numel() == 1:  # a single head's share is undone by the norm behind it
            continue
        changed = dict(w)
        noise = torch.randn(w[name].shape, generator=torch.Generator().manual_seed(len(name)), dtype=F64)
        changed[name] = w[name] * (1 + 0.5 * noise) + (0.3 if w[name].dim() == 1 else 0.0)
        assert float((plain.forward_logits(cfg, changed, ids) - base).abs().max()) > 1e-4, name


def test_attention_by_hand_bias_sink_and_gate():
    """All scores equal but for the bias: weights are e^rel of the distance's row, the sink takes its share and gives
    nothing, the gate of a zero matrix halves the output; the scale does not touch the bias."""
    W, n, rows = 4, 30, 6
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 1, "scale": 7.0, "bias_max": 12}
    rel = torch.tensor([[0.3], [-0.2], [0.9], [0.1], [-0.7], [0.4]], dtype=F64)
    w = {"q": torch.zeros(2, W, dtype=F64), "k": torch.zeros(2, W, dtype=F64), "v": torch.zeros(1, W, dtype=F64), "rel": rel,
         "sink": torch.tensor([0.25], dtype=F64), "g": torch.zeros(1, W, dtype=F64), "o": torch.ones(1, 1, dtype=F64)}
    w["v"][0, 0] = 1.0
    h = torch.zeros(n, W, dtype=F64)
    h[:, 0] = torch.arange(n, dtype=F64) + 1
    st = {"k": torch.zeros(0, 1, 2, dtype=F64), "v": torch.zeros(0, 1, 1, dtype=F64)}
    got = plain.attention(h, w, "", m, list(range(n)), st)[:, 0]
    # half = 3; beyond it 3 + floor(3 ln(n / 3) / ln 4): 3, 4 -> 3; 5, 6, 7 -> 4; from 8 on (n / 3 > 4^(2/3) = 2.52) -> 5
    row = lambda d: d if d < 3 else (3 if d < 5 else (4 if d < 8 else 5))  # noqa: E731
    for i in range(n):
        e = [math.exp(float(rel[row(i - j), 0])) for j in range(i + 1)]
        want = 0.5 * sum(x * (j + 1) for j, x in enumerate(e)) / (sum(e) + math.exp(0.25))
        assert abs(float(got[i]) - want) < 1e-12, i


def test_memories_by_hand():
    """One head, keys and values of one number: the recurrences written out."""
    W = 2
    h = torch.tensor([[1.0, 2.0], [-1.0, 0.5], [2.0, -3.0]], dtype=F64)
    w = {k: torch.zeros(1, W, dtype=F64) for k in ("q", "k", "v", "g")}
    w["q"][0, 0] = w["k"][0, 0] = w["v"][0, 1] = 1.0
    w["o"] = torch.tensor([[1.0], [0.0]], dtype=F64)
    sg = lambda z: 1 / (1 + math.exp(-z))  # noqa: E731
    # lightning: silu on everything, a weight, a sigmoid gate of zero
    w["norm"] = torch.tensor([3.0], dtype=F64)
    got = plain.lightning(h, w, "", {"heads": 1, "dim": 1, "vdim": 1, "decay": [0.5]}, 1e-6, {"S": torch.zeros(1, 1, 1, dtype=F64)})
    S, want = 0.0, []
    for a, b in h.tolist():
        k, v = a * sg(a), b * sg(b)
        S = 0.5 * S + k * v
        o = S * k
        want.append(o / math.sqrt(o * o + 1e-6) * 3.0 * 0.5)
    assert torch.allclose(got[:, 0], torch.tensor(want, dtype=F64), atol=1e-12)
    # the delta rule: one tap of a factor, a second one on the token before; b, a read the first input
    w.update({"q.conv": torch.tensor([[0.5, 1.0]], dtype=F64), "k.conv": torch.tensor([[-0.3, 0.8]], dtype=F64),
              "v.conv": torch.tensor([[0.2, 1.1]], dtype=F64), "b": torch.tensor([[0.7, 0.0]], dtype=F64),
              "a": torch.tensor([[-0.4, 0.0]], dtype=F64), "A_log": torch.tensor([-0.5], dtype=F64),
              "dt_bias": torch.tensor([0.1], dtype=F64), "g": torch.tensor([[0.0, 1.0]], dtype=F64)})
    st = {"S": torch.zeros(1, 1, 1, dtype=F64), **{x: torch.zeros(1, 1, dtype=F64) for x in "qkv"}}
    got = plain.delta(h, w, "", {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "conv": 2}, 1e-6, st)
    S, want, before = 0.0, [], (0.0, 0.0)
    for a, b in h.tolist():
        q, k, v = a + 0.5 * before[0], 0.8 * a - 0.3 * before[0], 1.1 * b + 0.2 * before[1]
        before = (a, b)
        q, k, v = q * sg(q), k * sg(k), v * sg(v)
        q, k = q / math.sqrt(q * q + 1e-6), k / math.sqrt(k * k + 1e-6)
        g = math.exp(-math.exp(-0.5) * math.log1p(math.exp(-0.4 * a + 0.1)))
        S = g * S
        u = sg(0.7 * a) * (v - S * k)
        S += k * u
        o = S * q
        want.append(o / math.sqrt(o * o + 1e-6) * 3.0 * b * sg(b))
    assert torch.allclose(got[:, 0], torch.tensor(want, dtype=F64), atol=1e-12)
    assert abs(float(st["S"]) - S) < 1e-12
    # retention: a rotation of the pair (value 0, value 1) by the position, the factor 2^-1/2 on the keys
    w2 = {"q": torch.eye(2, dtype=F64), "k": torch.eye(2, dtype=F64), "v": torch.tensor([[0.0, 1.0]], dtype=F64),
          "g": torch.tensor([[1.0, 0.0]], dtype=F64), "o": torch.ones(1, 1, dtype=F64)}
    m = {"heads": 1, "dim": 2, "vdim": 1, "decay": [0.75], "rot": {"base": 10.0, "dims": 2}}
    got = plain.retention(h, w2, "", m, 1e-6, [0, 1, 2], {"S": torch.zeros(1, 2, 1, dtype=F64)})
    S, want = [0.0, 0.0], []
    for p, (a, b) in enumerate(h.tolist()):
        r = (a * math.cos(p) - b * math.sin(p), b * math.cos(p) + a * math.sin(p))
        S = [0.75 * s + x / math.sqrt(2) * b for s, x in zip(S, r)]
        o = S[0] * r[0] + S[1] * r[1]
        want.append(o / math.sqrt(o * o + 1e-6) * a * sg(a))
    assert torch.allclose(got[:, 0], torch.tensor(want, dtype=F64), atol=1e-12)


def test_the_router_chooses_within_the_best_groups():
    z = torch.tensor([2.0, 0.0, 1.9, 1.8, 1.0, -5.0, 1.7, 1.6], dtype=F64)  # groups of two: best members 2, 1.9, 1, 1.7
    chosen, weights = plain.route(z, {"experts": 8, "top": 3, "groups": {"count": 4, "keep": 2}})
    assert chosen == [0, 2, 3]  # not 6 (1.7 > 0): its group is not among the two best
    e = [math.exp(v) for v in (2.0, 1.9, 1.8)]
    assert torch.allclose(weights, torch.tensor([x / sum(e) for x in e], dtype=F64))
    assert plain.route(z, {"experts": 8, "top": 3, "groups": {"count": 1, "keep": 1}})[0] == [0, 2, 3]
    assert plain.route(z, {"experts": 8, "top": 4, "groups": {"count": 4, "keep": 3}})[0] == [0, 2, 3, 6]
    assert plain.route(z, {"experts": 8, "top": 2, "groups": {"count": 4, "keep": 1}})[0] == [0, 1]
    tie = torch.tensor([1.0, 2.0, 2.0, 2.0], dtype=F64)
    assert plain.route(tie, {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 1}})[0] == [1, 0]


def test_both_sub_layers_read_the_same_stream(tmp_path):
    """One layer: the stream after it is x + mixer(norm1 x) + experts(norm2 x), the feed-forward blind to the mixer."""
    config = copy.deepcopy(DOMELIX_Y)
    config["layers"] = config["layers"][:1]
    cfg, w = plain.read_model_folder(make_folder(str(tmp_path / "m"), config, 9))
    ids = [3, 14, 15, 92, 65]
    layers = []
    plain.forward(cfg, w, ids, layers_out=layers)
    x = w["embed"][torch.tensor(ids)]
    entry, eps = cfg["layers"][0], 1e-6
    n1 = x / torch.sqrt((x * x).mean(1, keepdim=True) + eps) * (1 + w["l0.norm1"])
    n2 = x / torch.sqrt((x * x).mean(1, keepdim=True) + eps) * (1 + w["l0.norm2"])
    mix = plain.retention(n1, w, "l0.mix.", entry["mixer"], eps, list(range(5)), plain.new_state(cfg)[0])
    assert torch.allclose(layers[0], x + mix + plain.experts(n2, w, "l0.mlp.", entry["mlp"]), atol=1e-12)


def test_pending_sums():
    from qwen3_from_scratch_b200.parts.base import PendingSum, PendingTerm
    a, b, w = torch.ones(2, 3), torch.zeros(2, 3), torch.ones(3)
    s = PendingSum.of(PendingSum((PendingTerm(a, w, 0.5), PendingTerm(b, w, 0.5)), 1e-3), a)
    assert [t.weight is w for t in s.terms] == [True, True, False] and s.eps == 1e-3 and s.terms[2].delta is a
    assert PendingSum.of(a).eps == 0.0
    with pytest.raises(ValueError, match="epsilon"):
        PendingSum.of(s, PendingSum((PendingTerm(a, w, 1.0),), 1e-5))


def test_bias_rows_are_even_and_known():
    assert all(r % 2 == 0 for r in BIAS_ROWS.values()) and {c["vocab"] for c, _ in CONFIGS.values()} == set(BIAS_ROWS)
