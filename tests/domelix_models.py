"""Small Domelix configurations and model folders for the tests: the configuration dicts, the tensors the design names
for them (names and shapes restated here from the design, not asked of the engine) and random weights strong enough that
every mechanism moves the logits."""

from __future__ import annotations

import json
import os
from typing import Dict

import torch
from safetensors.torch import save_file


def attention(heads, kv_heads, dim, vdim, scale, bias_max):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max}


def lightning(dim, vdim, decay):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay}


def parallel(left, right):
    return {"type": "parallel", "mixer": {"left": left, "right": right}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def retention(dim, vdim, decay, base, dims):
    return {"type": "retention", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay,
                                           "rot": {"base": base, "dims": dims}}}


def moe(experts, top, groups, keep, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top,
                                                            "groups": {"count": groups, "keep": keep}}}


def with_mlp(entry, mlp):
    return dict(entry, mlp=mlp)


# X: every layer with sizes of its own: three query heads per key head, a bias table of eight rows that widen up to 20
# positions, keys narrower and wider than values, decays of 0 and 1 beside others, a partly rotated retention, two value
# heads per query/key head, three taps, a layer without feed-forward, experts in groups of which some are kept, in one
# group, and in groups that are all kept.
DOMELIX_X = {
    "architecture": "Domelix", "vocab": 211, "width": 64, "norm": {"eps": 1e-5},
    "layers": [with_mlp(delta(4, 2, 24, 16, 3), moe(12, 3, 4, 2, 24)),
               with_mlp(parallel(attention(6, 2, 24, 40, 0.2, 20), lightning(16, 24, [0.0, 0.6, 1.0])), moe(5, 2, 1, 1, 32)),
               with_mlp(retention(20, 36, [0.5, 0.93, 0.999], 1000.0, 12), None),
               with_mlp(parallel(attention(4, 4, 16, 8, 0.3, 9.5), lightning(40, 8, [0.97])), moe(6, 4, 3, 3, 16)),
               with_mlp(delta(3, 3, 40, 24, 5), moe(6, 1, 3, 1, 40))]}
# Y: one of everything: a single head everywhere, a single tap (no tail to keep), nothing rotated, a bias table of two
# rows, every expert chosen; one expert alone.
DOMELIX_Y = {
    "architecture": "Domelix", "vocab": 173, "width": 48, "norm": {"eps": 1e-6},
    "layers": [with_mlp(retention(16, 24, [0.9], 10000.0, 0), moe(3, 3, 1, 1, 40)),
               with_mlp(parallel(attention(1, 1, 32, 24, 0.18, 2), lightning(8, 16, [0.8])), moe(4, 2, 2, 1, 24)),
               with_mlp(delta(1, 1, 16, 8, 1), moe(1, 1, 1, 1, 56))]}
# Z: sizes in the manner of the serving kernels, small: heads of 64 and 128, slow decays, experts in multiples of 16.
DOMELIX_Z = {
    "architecture": "Domelix", "vocab": 300, "width": 128, "norm": {"eps": 1e-6},
    "layers": [with_mlp(parallel(attention(8, 2, 64, 64, 0.11, 60), lightning(64, 128, [0.9, 0.99, 0.9995])), moe(24, 3, 6, 2, 48)),
               with_mlp(delta(4, 2, 128, 64, 4), moe(8, 2, 2, 1, 64)),
               with_mlp(retention(128, 32, [0.97, 0.995], 50000.0, 64), moe(10, 4, 5, 4, 32)),
               with_mlp(delta(2, 2, 64, 96, 2), moe(24, 3, 6, 2, 48))]}
# W: more experts than a warp has lanes; five heads, keys of 80 and 128, values of 112 and 96, a table of 30 rows, six
# taps (beyond the convolution kernels that are compiled per number of taps).
DOMELIX_W = {
    "architecture": "Domelix", "vocab": 400, "width": 160, "norm": {"eps": 1e-6},
    "layers": [with_mlp(retention(128, 96, [0.98, 0.9, 0.5], 20000.0, 128), moe(40, 5, 8, 3, 16)),
               with_mlp(parallel(attention(5, 5, 80, 112, 0.1, 77), lightning(24, 56, [0.6, 0.7, 0.8, 0.9, 0.999])), moe(6, 2, 3, 2, 48)),
               with_mlp(delta(6, 2, 72, 40, 6), moe(36, 2, 2, 1, 24))]}
CONFIGS = {"x": (DOMELIX_X, 3), "y": (DOMELIX_Y, 4), "z": (DOMELIX_Z, 5), "w": (DOMELIX_W, 6)}
BIAS_ROWS = {211: 8, 173: 2, 300: 16, 400: 30}  # by vocabulary: a table's rows stand in no configuration


def tensor_shapes(config: dict) -> Dict[str, tuple]:
    W, V = config["width"], config["vocab"]
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, entry in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", entry["mixer"], entry["mlp"]
        shapes[p + "norm1"] = (W,)

        def memory(pre, m, norm):
            H, D, Dv = m["heads"], m["dim"], m["vdim"]
            shapes.update({pre + "q": (H * D, W), pre + "k": (H * D, W), pre + "v": (H * Dv, W), pre + "g": (H * Dv, W),
                           pre + "o": (W, H * Dv)})
            if norm:
                shapes[pre + "norm"] = (H * Dv,)

        if entry["type"] == "parallel":
            a, pre = m["left"], p + "mix.left."
            H, G, D, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            shapes.update({pre + "q": (H * D, W), pre + "k": (G * D, W), pre + "v": (G * Dv, W), pre + "g": (H * Dv, W),
                           pre + "rel": (BIAS_ROWS[V], H), pre + "sink": (H,), pre + "o": (W, H * Dv), pre + "out": (W,),
                           p + "mix.right.out": (W,)})
            memory(p + "mix.right.", m["right"], True)
        elif entry["type"] == "retention":
            memory(p + "mix.", m, False)
        else:
            H, G, D, Dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            pre = p + "mix."
            for x, n in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                shapes.update({pre + x: (n, W), pre + x + ".conv": (n, K)})
            shapes.update({pre + "b": (H, W), pre + "a": (H, W), pre + "A_log": (H,), pre + "dt_bias": (H,), pre + "norm": (Dv,),
                           pre + "g": (H * Dv, W), pre + "o": (W, H * Dv)})
        if mlp is not None:
            E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            shapes.update({p + "norm2": (W,), p + "mlp.router": (E, W)})
            for e in range(E):
                shapes.update({f"{p}mlp.e{e}.gate": (F, W), f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    return shapes


def random_tensor(name: str, shape: tuple, g: torch.Generator) -> torch.Tensor:
    r = lambda: torch.randn(shape, generator=g)  # noqa: E731
    leaf = name.rsplit(".", 1)[-1]
    if leaf in ("norm1", "norm2") or name == "final.norm":  # stored around zero
        t = 0.2 * r()
    elif leaf in ("norm", "out"):
        t = 1.0 + 0.2 * r()
    elif leaf in ("sink", "rel"):  # of the size of the scores: a visible share of the weight
        t = 1.0 * r()
    elif leaf == "A_log":
        t = torch.log(0.02 + 0.5 * torch.rand(shape, generator=g))
    elif leaf == "dt_bias":
        t = 0.5 * r()
    elif leaf == "conv":
        t = r() * (1.0 / shape[-1] ** 0.5)
    elif name == "embed":
        t = 0.7 * r()
    elif leaf == "router":  # scores spread out, so that few choices are near ties
        t = r() * (3.0 / shape[-1] ** 0.5)
    elif leaf == "down":  # a choice of experts that rounding turns over must not move a bfloat16 run's logits by more than
        t = r() * (0.2 / shape[-1] ** 0.5)  # other rounding does
    else:  # a matrix [out, in]: outputs of order one for inputs of order one
        t = r() * (1.3 / shape[-1] ** 0.5)
    return t.to(torch.bfloat16)


def make_folder(folder: str, config: dict, seed: int, tweak=None) -> str:
    """config.json and model.safetensors (bfloat16) in ``folder``.  ``tweak(tensors)`` may change them first."""
    os.makedirs(folder, exist_ok=True)
    g = torch.Generator().manual_seed(seed)
    tensors = {name: random_tensor(name, shape, g) for name, shape in sorted(tensor_shapes(config).items())}
    if tweak is not None:
        tweak(tensors)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(folder, "model.safetensors"))
    return folder
