"""Small Zasitar configurations and model folders for the tests: the configuration dicts, the tensors the design names
for them (names and shapes restated here from the design, not asked of the engine) and random weights strong enough that
every mechanism moves the logits."""

from __future__ import annotations

import json
import os
from typing import Dict

import torch
from safetensors.torch import save_file


def wkv(heads, dim, mlp):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, scale, window, base, dims, mlp, scaling=None, kv_from=None):
    rot = {"base": base, "dims": dims}
    if scaling is not None:
        factor, low, high, original = scaling
        rot["scaling"] = {"factor": factor, "low": low, "high": high, "original": original}
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}, "rot": rot}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        d["shared"] = {"ff": shared[0], "limit": shared[1]}
    return d


# X: every layer with sizes of its own: three query heads per key head, keys narrower than values, a partly rotated head with
# all three bands of the frequency scaling, two layers that read one layer's keys (over a wider and a narrower window, with
# other scales) with another attention layer between, time mixing first and last, every kind of feed-forward and none.
ZASITAR_X = {
    "architecture": "Zasitar", "vocab": 211, "width": 64, "norm": {"eps": 1e-5},
    "layers": [wkv(3, 24, moe(12, 3, 24, 0.7, (40, 1.1))),
               attention(6, 2, 24, 40, 0.3, 13, 1000.0, 16, dense(72), (4.0, 0.5, 6.0, 90)),
               wkv(2, 40, None),
               attention(4, 4, 16, 8, 0.35, 21, 500.0, 16, moe(5, 2, 32, 0.9)),
               attention(6, 2, 24, 40, 0.25, 30, 1000.0, 16, moe(6, 6, 16, 1.4, (24, 0.5)), (4.0, 0.5, 6.0, 90), kv_from=1),
               attention(6, 2, 24, 40, 0.4, 7, 1000.0, 16, None, (4.0, 0.5, 6.0, 90), kv_from=1),
               wkv(1, 16, dense(20))]}
# Y: one of everything: a single head everywhere, a window of the token itself, nothing rotated, one expert alone, every
# expert chosen, a decay projection of rank one.
ZASITAR_Y = {
    "architecture": "Zasitar", "vocab": 173, "width": 48, "norm": {"eps": 1e-6},
    "layers": [attention(1, 1, 16, 24, 0.5, 1, 10000.0, 0, moe(1, 1, 40, 0.8, (16, 0.9))),
               attention(1, 1, 32, 32, 0.2, 9, 10000.0, 32, None, (8.0, 1.0, 4.0, 64)),
               wkv(1, 32, moe(3, 3, 24, 2.0)),
               attention(1, 1, 16, 24, 0.4, 5, 10000.0, 0, dense(56), kv_from=0)]}
# Z: sizes in the manner of the serving kernels, small: heads of 32, 64 and 128, experts in multiples of 16.
ZASITAR_Z = {
    "architecture": "Zasitar", "vocab": 300, "width": 128, "norm": {"eps": 1e-6},
    "layers": [wkv(2, 64, dense(256)),
               attention(8, 2, 64, 64, 0.15, 70, 20000.0, 32, moe(16, 4, 48, 1.2, (80, 0.8)), (8.0, 1.0, 4.0, 256)),
               wkv(4, 32, moe(10, 2, 32, 0.6, (64, 1.6))),
               attention(8, 2, 64, 64, 0.12, 130, 20000.0, 32, dense(128), (8.0, 1.0, 4.0, 256), kv_from=1),
               attention(2, 1, 128, 32, 0.1, 64, 20000.0, 128, dense(192), (2.0, 1.0, 2.0, 100)),
               wkv(1, 128, moe(8, 3, 64, 1.0, (32, 1.0)))]}
# W: more experts than a warp has lanes, sizes that no tensor-core kernel takes.
ZASITAR_W = {
    "architecture": "Zasitar", "vocab": 400, "width": 160, "norm": {"eps": 1e-6},
    "layers": [attention(5, 5, 80, 112, 0.12, 50, 3000.0, 40, moe(40, 5, 20, 1.3, (36, 0.7)), (3.0, 0.8, 3.0, 200)),
               wkv(2, 72, moe(36, 2, 24, 0.9, (8, 1.0))),
               attention(5, 5, 80, 112, 0.1, 50, 3000.0, 40, dense(100), (3.0, 0.8, 3.0, 200), kv_from=0)]}
CONFIGS = {"x": (ZASITAR_X, 3), "y": (ZASITAR_Y, 4), "z": (ZASITAR_Z, 5), "w": (ZASITAR_W, 6)}
RANKS = {211: 5, 173: 1, 300: 16, 400: 37}  # by vocabulary: the rank of the decay's projection stands in no configuration


def tensor_shapes(config: dict) -> Dict[str, tuple]:
    W, V = config["width"], config["vocab"]
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, entry in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", entry["mixer"], entry["mlp"]
        shapes.update({p + "norm1": (W,), p + "ls1": (W,)})
        if entry["type"] == "wkv":
            n = m["heads"] * m["dim"]
            shapes.update({f"{p}mix.mu.{s}": (W,) for s in "rkvgw"})
            shapes.update({f"{p}mix.{s}": (n, W) for s in "rkvg"})
            shapes.update({p + "mix.w1": (RANKS[V], W), p + "mix.w2": (n, RANKS[V]), p + "mix.w0": (n,),
                           p + "mix.u": (m["heads"], m["dim"]), p + "mix.norm": (n,), p + "mix.o": (W, n)})
        else:
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            shapes.update({p + "mix.q": (H * D, W), p + "mix.q.b": (H * D,), p + "mix.q.norm": (D,), p + "mix.o": (W, H * Dv),
                           p + "mix.o.b": (W,)})
            if m.get("kv_from") is None:
                shapes.update({p + "mix.k": (G * D, W), p + "mix.k.b": (G * D,), p + "mix.k.norm": (D,), p + "mix.v": (G * Dv, W),
                               p + "mix.v.b": (G * Dv,)})
        if mlp is None:
            continue
        shapes.update({p + "norm2": (W,), p + "ls2": (W,)})

        def ff(pre, F, bias):
            for s, shape in (("gate", (F, W)), ("up", (F, W)), ("down", (W, F))):
                shapes[pre + s] = shape
                if bias:
                    shapes[f"{pre}{s}.b"] = shape[:1]

        if mlp["kind"] == "dense":
            ff(p + "mlp.", mlp["ff"], True)
            continue
        E = mlp["router"]["experts"]
        shapes.update({p + "mlp.router": (E, W), p + "mlp.router.b": (E,)})
        for e in range(E):
            ff(f"{p}mlp.e{e}.", mlp["expert"]["ff"], False)
        if mlp.get("shared"):
            ff(p + "mlp.shared.", mlp["shared"]["ff"], False)
            shapes[p + "mlp.shared.sg"] = (1, W)
    return shapes


def random_tensor(name: str, shape: tuple, g: torch.Generator) -> torch.Tensor:
    r = lambda: torch.randn(shape, generator=g)  # noqa: E731
    leaf = name.rsplit(".", 1)[-1]
    if leaf in ("norm", "norm1", "norm2"):
        t = 1.0 + 0.2 * r()
    elif leaf == "ls1":
        t = 0.8 + 0.2 * r()
    elif leaf == "ls2":  # a choice of experts that rounding turns over must not move a bfloat16 run's logits by much more
        t = 0.4 + 0.1 * r()  # than other rounding does
    elif leaf == "b":
        t = 0.3 * r()
    elif ".mu." in name:
        t = torch.rand(shape, generator=g)
    elif leaf == "w0":  # decays from next to none to strong ones
        t = -6.0 + 6.5 * torch.rand(shape, generator=g)
    elif leaf == "w2":
        t = r() * (0.6 / shape[-1] ** 0.5)
    elif leaf == "u":
        t = 0.8 + 0.3 * r()
    elif name == "embed":
        t = 0.8 * r()
    elif leaf == "router":  # logits spread out, so that few choices are near ties
        t = r() * (4.0 / shape[-1] ** 0.5)
    else:  # a matrix [out, in]: outputs of order one for inputs of order one
        t = r() * (1.2 / shape[-1] ** 0.5)
    return t.to(torch.bfloat16)


def make_folder(folder: str, config: dict, seed: int, tweak=None) -> str:
    """config.json and model.safetensors (bfloat16) in ``folder``.  ``tweak(tensors)`` may change them first."""
    os.makedirs(folder, exist_ok=True)
    g = torch.Generator().manual_seed(seed)
    tensors = {name: random_tensor(name, shape, g) for name, shape in sorted(tensor_shapes(config).items())}
    for name in tensors:  # receptances that lean towards the keys: a read-out is then seldom a small difference of large
        if name.endswith(".mix.r"):  # terms, which the norm behind it would blow up together with its rounding
            tensors[name] = (0.6 * tensors[name].float() + 0.9 * tensors[name[:-1] + "k"].float()).to(torch.bfloat16)
    if tweak is not None:
        tweak(tensors)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(folder, "model.safetensors"))
    return folder
