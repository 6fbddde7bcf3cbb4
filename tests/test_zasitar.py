"""Zasitar without a GPU: its configuration, what the model asks of the weights and of the cache, the stretched frequencies,
and the plain implementation against itself (a prompt whole, in portions and token by token through the explicit caches and
states) and on values worked by hand."""

import copy
import math

import pytest
import torch

import plain_zasitar as plain
from zasitar_models import CONFIGS, ZASITAR_X, ZASITAR_Y, ZASITAR_Z, make_folder, tensor_shapes

F64 = plain.F64


def model_of(config):
    from qwen3_from_scratch_b200.engine.model import Model
    from qwen3_from_scratch_b200.registry import build_model_spec, config_from_dict
    return Model(build_model_spec(config_from_dict(config)))


@pytest.mark.parametrize("key", list(CONFIGS))
def test_the_model_asks_for_the_tensors_the_design_names(key):
    """Names and shapes, but for the rank of the decays' projection, which the folder decides."""
    config = CONFIGS[key][0]
    want = tensor_shapes(config)
    specs = {s.name: s for s in model_of(config).weight_specs()}
    assert set(specs) == set(want)
    for name, shape in want.items():
        assert specs[name].takes(shape), (name, shape, specs[name].shape)
        if name.endswith((".w1", ".w2")):
            assert specs[name].free_dims == ((0,) if name.endswith("w1") else (1,))
        else:
            assert tuple(specs[name].shape) == shape


def test_a_layer_without_feed_forward_may_still_carry_its_norm_and_scale(tmp_path):
    from qwen3_from_scratch_b200.weights.loader import WeightsError, load_weights
    model = model_of(ZASITAR_X)

    def load(extra):
        def tweak(t):
            t.update({name: torch.ones(64, dtype=torch.bfloat16) for name in extra})
        folder = make_folder(str(tmp_path / str(len(extra))), ZASITAR_X, 1, tweak)
        return load_weights(folder, model.weight_specs(), device="cpu", compute_dtype=torch.bfloat16,
                            ignorable=model.spec.ignorable_weights)

    load(["l2.norm2", "l2.ls2", "l5.ls2"])
    with pytest.raises(WeightsError, match="l4.mix.k"):
        load(["l2.norm2", "l2.ls2", "l5.ls2", "l4.mix.k"])


def test_configuration_round_trip():
    from qwen3_from_scratch_b200.registry import config_from_dict
    cfg = config_from_dict(ZASITAR_X)
    assert cfg.architecture == "Zasitar" and (cfg.vocab, cfg.width, cfg.norm_eps) == (211, 64, 1e-5)
    a, b = cfg.layers[1], cfg.layers[4]
    assert (cfg.layers[0].type, cfg.layers[0].mixer.heads, cfg.layers[0].mixer.dim) == ("wkv", 3, 24)
    assert (a.mixer.heads, a.mixer.kv_heads, a.mixer.dim, a.mixer.vdim, a.mixer.scale, a.mixer.window) == (6, 2, 24, 40, 0.3, 13)
    assert (a.mixer.rot_base, a.mixer.rot_dims, a.mixer.kv_from, a.mlp.ff) == (1000.0, 16, None, 72)
    s = a.mixer.rot_scaling
    assert (s.factor, s.low, s.high, s.original) == (4.0, 0.5, 6.0, 90) and cfg.layers[3].mixer.rot_scaling is None
    assert (b.mixer.kv_from, b.mixer.window) == (1, 30) and cfg.layers[2].mlp is None
    e = cfg.layers[0].mlp
    assert (e.experts, e.top, e.expert.ff, e.expert.limit, e.shared.ff, e.shared.limit) == (12, 3, 24, 0.7, 40, 1.1)
    assert cfg.layers[3].mlp.shared is None
    for config in (ZASITAR_X, ZASITAR_Y, ZASITAR_Z):
        cfg = config_from_dict(config)
        assert config_from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == config


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][0].update(type="mamba"), "not built"),
    (lambda c: c["layers"][0].update(mlp={"kind": "sparse"}), "dense"),
    (lambda c: c["layers"][0]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("high"), "high"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(low=6.0), "exceed"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=1), "earlier"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=0), "earlier"),
    (lambda c: c["layers"][5]["mixer"].update(kv_from=4), "of its own"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=-1), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=3), "layer 3"),
    (lambda c: c["layers"][4]["mixer"]["rot"].update(base=999.0), "layer 1"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=13), "top"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0.0), "limit"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_errors_name_the_key(change, message):
    from qwen3_from_scratch_b200.config.model_config import ConfigError
    from qwen3_from_scratch_b200.registry import config_from_dict
    config = copy.deepcopy(ZASITAR_X)
    change(config)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(config)


def test_cache_needs():
    """A layer with keys of its own keeps pages over the widest window that it and the layers that read it look back; those
    keep nothing; time mixing keeps a matrix per head and the last input, both float32."""
    from qwen3_from_scratch_b200.parts.base import StateSpec
    model = model_of(ZASITAR_X)
    layout = model.cache_layout()
    groups = {tuple((p.name, p.heads, p.width) for p in g.spec.planes): (g.cache_ids, g.spec.window) for g in layout.groups}
    assert groups == {(("k", 2, 24), ("v", 2, 40)): ([1], 30), (("k", 4, 16), ("v", 4, 8)): ([3], 21)}
    assert layout.states == {(0, "shift"): StateSpec((64,)), (0, "state"): StateSpec((3, 24, 24)), (2, "shift"): StateSpec((64,)),
                             (2, "state"): StateSpec((2, 40, 40)), (6, "shift"): StateSpec((64,)), (6, "state"): StateSpec((1, 16, 16))}
    assert [(c.layer, c.cache, c.write_cache) for c in model.spec.order] == [
        (0, 0, True), (1, 1, True), (2, 2, True), (3, 3, True), (4, 1, False), (5, 1, False), (6, 6, True)]


def test_what_two_layers_on_one_cache_need():
    from qwen3_from_scratch_b200.engine.model import shared_need
    from qwen3_from_scratch_b200.parts.base import CachePlane, KVCacheSpec, PagedCacheSpec, StateSpec
    assert shared_need(KVCacheSpec(2, 8, 5), KVCacheSpec(2, 8, 9)) == KVCacheSpec(2, 8, 9)
    assert shared_need(KVCacheSpec(2, 8, 5), KVCacheSpec(2, 8)) == shared_need(KVCacheSpec(2, 8), KVCacheSpec(2, 8, 5)) == KVCacheSpec(2, 8)
    planes = (CachePlane("k", 1, 4),)
    assert shared_need(PagedCacheSpec(planes, 4, keep_first=3), PagedCacheSpec(planes, 9)) == PagedCacheSpec(planes, 9, keep_first=3)
    assert shared_need(KVCacheSpec(2, 8, 5), KVCacheSpec(2, 16, 5)) is None
    assert shared_need(KVCacheSpec(2, 8, 5), StateSpec((3,))) is None and shared_need(StateSpec((3,)), StateSpec((3,))) == StateSpec((3,))


def test_random_model_folder_through_the_framework_writer(tmp_path):
    from qwen3_from_scratch_b200.registry import config_from_dict
    from qwen3_from_scratch_b200.weights import write_random_model
    folder = write_random_model(str(tmp_path / "m"), config_from_dict(ZASITAR_Z), seed=1)
    config, w = plain.read_model_folder(folder)
    shapes, want = {k: tuple(v.shape) for k, v in w.items()}, tensor_shapes(ZASITAR_Z)
    rank = lambda d: {k: v for k, v in d.items() if not k.endswith((".w1", ".w2"))}  # noqa: E731
    assert rank(shapes) == rank(want) and set(shapes) == set(want)
    logits = plain.forward_logits(config, w, [5, 17, 3, 250, 9])
    assert logits.shape == (5, 300) and torch.isfinite(logits).all()


@pytest.mark.parametrize("dims,base,scaling", [(16, 1000.0, (4.0, 0.5, 6.0, 90)), (32, 20000.0, (8.0, 1.0, 4.0, 256)),
                                               (2, 10.0, (3.0, 1.0, 2.0, 5)), (64, 500.0, (2.0, 0.1, 10.0, 100)), (8, 100.0, None)])
def test_stretched_frequencies(dims, base, scaling):
    """The engine's position part against the plain frequencies, and those against the three bands written out."""
    from qwen3_from_scratch_b200.parts.base import PartSpec
    from qwen3_from_scratch_b200.registry import create_part
    s = None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling))
    part = create_part("position", PartSpec("rotary_banded", {"dims": dims, "base": base, "scaling": s}), name="p")
    want = plain.frequencies({"dims": dims, "base": base, "scaling": s})
    assert torch.allclose(torch.tensor(part._freq, dtype=F64), want, rtol=1e-12) and part.magnitude == 1.0
    bands = set()
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if s is None:
            assert abs(float(want[i]) - f) < 1e-15
            continue
        length = 2 * math.pi / f
        if length < s["original"] / s["high"]:
            bands.add("kept")
            assert abs(float(want[i]) - f) < 1e-12 * f
        elif length > s["original"] / s["low"]:
            bands.add("stretched")
            assert abs(float(want[i]) - f / s["factor"]) < 1e-12 * f
        else:
            bands.add("between")
            assert f / s["factor"] - 1e-12 <= float(want[i]) <= f + 1e-12
    if dims in (16, 32, 64):
        assert bands == {"kept", "stretched", "between"}


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
        if ".mlp.e" in name or (".router" in name and w[name].shape[0] == 1):
            continue
        changed = dict(w)
        noise = torch.randn(w[name].shape, generator=torch.Generator().manual_seed(len(name)), dtype=F64)
        changed[name] = w[name] * (1 + 0.5 * noise) + (0.3 if w[name].dim() == 1 else 0.0)
        assert float((plain.forward_logits(cfg, changed, ids) - base).abs().max()) > 1e-4, name


def test_attention_by_hand_window_sink_and_shared_keys():
    """Queries and keys that their biases make, so that every score is the scale (times a norm's weight): the weights are
    e^s / (1 + n e^s) over the window's n tokens; a second layer reads the first one's values through its own window."""
    W, n = 3, 12
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 1, "scale": 0.35, "mask": {"size": 4}, "rot": {"base": 10.0, "dims": 0}}
    zero = lambda *s: torch.zeros(*s, dtype=F64)  # noqa: E731
    one = lambda *v: torch.tensor(v, dtype=F64)  # noqa: E731
    w = {"q": zero(2, W), "q.b": one(5.0, 5.0), "q.norm": one(1.0, 1.0), "k": zero(2, W), "k.b": one(0.2, 0.2), "k.norm": one(2.0, 1.0),
         "v": zero(1, W), "v.b": one(10.0), "o": torch.ones(1, 1, dtype=F64), "o.b": one(-1.0)}
    w["v"][0, 0] = 1.0
    h = zero(n, W)
    h[:, 0] = torch.arange(n, dtype=F64)
    st = {"k": zero(0, 1, 2), "v": zero(0, 1, 1)}
    got = plain.attention(h, w, "", m, 0.0, list(range(n)), st)[:, 0]
    # both heads are normed to (1, 1), the key's weights are (2, 1): q . k = 3
    e = math.exp(3 * 0.35)

    def want(i, window):
        seen = range(max(0, i - window + 1), i + 1)
        return sum(10.0 + j for j in seen) * e / (1 + len(seen) * e) - 1.0

    for i in range(n):
        assert abs(float(got[i]) - want(i, 4)) < 1e-12, i
    reader = dict(m, kv_from=0, mask={"size": 7})
    own = {k: w[k] for k in ("q", "q.b", "q.norm", "o", "o.b")}
    got = plain.attention(h, own, "", reader, 0.0, list(range(n)), st)[:, 0]
    for i in range(n):
        assert abs(float(got[i]) - want(i, 7)) < 1e-12, i


def test_time_mixing_by_hand():
    """One head with keys and values of one number: the mixes with the token before, the decay, the bonus and the gate
    written out."""
    W = 2
    h = torch.tensor([[1.0, 2.0], [-1.0, 0.5], [2.0, -3.0]], dtype=F64)
    mu = {"r": (0.1, 0.9), "k": (0.2, 0.8), "v": (0.3, 0.7), "g": (0.4, 0.6), "w": (0.5, 0.25)}
    w = {f"mu.{s}": torch.tensor(v, dtype=F64) for s, v in mu.items()}
    w.update({"r": torch.tensor([[1.0, 0.0]], dtype=F64), "k": torch.tensor([[0.0, 1.0]], dtype=F64),
              "v": torch.tensor([[0.5, 0.5]], dtype=F64), "g": torch.tensor([[1.0, -1.0]], dtype=F64),
              "w1": torch.tensor([[0.3, 0.2], [-0.5, 0.1]], dtype=F64), "w2": torch.tensor([[0.7, -0.4]], dtype=F64),
              "w0": torch.tensor([-0.3], dtype=F64), "u": torch.tensor([[1.7]], dtype=F64), "norm": torch.tensor([3.0], dtype=F64),
              "o": torch.tensor([[1.0], [0.0]], dtype=F64)})
    st = {"S": torch.zeros(1, 1, 1, dtype=F64), "h": torch.zeros(W, dtype=F64)}
    got = plain.time_mixing(h, w, "", {"heads": 1, "dim": 1}, 1e-2, st)[:, 0]
    S, before, want = 0.0, (0.0, 0.0), []
    for x in h.tolist():
        mix = {s: [x[i] + (before[i] - x[i]) * mu[s][i] for i in range(2)] for s in mu}
        before = x
        r, k, v = mix["r"][0], mix["k"][1], 0.5 * (mix["v"][0] + mix["v"][1])
        a = mix["w"]
        decay = math.exp(-math.exp(0.7 * math.tanh(0.3 * a[0] + 0.2 * a[1]) - 0.4 * math.tanh(-0.5 * a[0] + 0.1 * a[1]) - 0.3))
        o = (S + 1.7 * k * v) * r
        S = decay * S + k * v
        g = mix["g"][0] - mix["g"][1]
        want.append(o / math.sqrt(o * o + 1e-2) * 3.0 * g / (1 + math.exp(-g)))
    assert torch.allclose(got, torch.tensor(want, dtype=F64), atol=1e-12)
    assert abs(float(st["S"]) - S) < 1e-12 and st["h"].tolist() == [2.0, -3.0]


def test_limited_experts_and_the_router_by_hand():
    eye = torch.eye(4, dtype=F64)
    x = torch.tensor([[-3.0, -0.4, 0.4, 3.0]], dtype=F64)
    got = plain.limited_expert(x, {"gate": eye, "up": eye, "down": eye}, "", 0.5)[0]
    for v, y in zip(x[0].tolist(), got.tolist()):
        g, u = min(v, 0.5), max(-0.5, min(v, 0.5))
        assert abs(y - g / (1 + math.exp(-1.702 * g)) * (u + 1)) < 1e-12
    chosen, weights = plain.route(torch.tensor([1.0, 3.0, -2.0, 2.5, 3.0], dtype=F64), 3)
    assert chosen == [1, 4, 3]
    e = [math.exp(v) for v in (3.0, 3.0, 2.5)]
    assert torch.allclose(weights, torch.tensor([v / sum(e) for v in e], dtype=F64))
    # the bias of the logits decides and weighs; the shared expert's share is one number per token
    mlp = {"router": {"experts": 2, "top": 1}, "expert": {"limit": 9.0}, "shared": {"limit": 9.0}}
    w = {"router": torch.zeros(2, 4, dtype=F64), "router.b": torch.tensor([0.0, 1.0], dtype=F64), "shared.sg": 0.5 * torch.ones(1, 4, dtype=F64)}
    for i, pre in enumerate(("e0.", "e1.", "shared.")):
        w.update({pre + "gate": eye, pre + "up": eye, pre + "down": (i + 1) * eye})
    one = plain.limited_expert(x, w, "e0.", 9.0)[0]
    share = 1 / (1 + math.exp(-0.5 * float(x.sum())))
    assert torch.allclose(plain.experts(x, w, "", mlp)[0], (2 + 3 * share) * one, atol=1e-12)


def test_norms_stand_behind_the_sub_layers_only(tmp_path):
    """One layer: the mixer reads the embedding as it is, the feed-forward what the mixer left; each output is normed,
    weighted and scaled on its way into the stream."""
    config = copy.deepcopy(ZASITAR_X)
    config["layers"] = config["layers"][1:2]
    cfg, w = plain.read_model_folder(make_folder(str(tmp_path / "m"), config, 9))
    ids = [3, 14, 15, 92, 65]
    layers = []
    logits = plain.forward(cfg, w, ids, layers_out=layers)
    unit = lambda y: y / torch.sqrt((y * y).mean(1, keepdim=True) + 1e-5)  # noqa: E731
    x = w["embed"][torch.tensor(ids)]
    a = plain.attention(x, w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5, list(range(5)), plain.new_state(cfg)[0])
    x = x + unit(a) * w["l0.norm1"] * w["l0.ls1"]
    x = x + unit(plain.dense(x, w, "l0.mlp.")) * w["l0.norm2"] * w["l0.ls2"]
    assert torch.allclose(layers[0], x, atol=1e-12)
    assert torch.allclose(logits, (unit(x) * w["final.norm"]) @ w["head"].t(), atol=1e-12)


def test_open_terms_carry_a_bias():
    from qwen3_from_scratch_b200.parts.base import PendingSum, PendingTerm
    a, b, w = torch.ones(2, 3), torch.full((3,), 2.0), torch.ones(3)
    s = PendingSum.of(PendingTerm(a, bias=b), a)
    assert s.kernel_terms()[0][3] is b and s.kernel_terms()[1][3] is None and s.eps == 0.0
    with pytest.raises(ValueError, match="PendingSum"):
        PendingSum.of(PendingTerm(a, w))
