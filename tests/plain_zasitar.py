"""A plain, slow statement of the Zasitar design in float64 on the CPU: one function per mechanism, written from the
mechanism's equations, sharing no code with the engine.  Whatever is carried from token to token (the keys and values of
the attention layers that have their own, the matrix states of the time mixing and the input it saw last) is taken and
returned explicitly, so that a prompt can run whole, in portions or token by token through the same functions.

Notation: T tokens, W the stream's width, H heads.  ``w`` maps tensor names to float64 tensors.
"""

from __future__ import annotations

import json
import math
import os
from typing import List, Optional, Sequence

import torch
from safetensors import safe_open

F64 = torch.float64

# What a projection does to its operand and its result: nothing, or (inside ``bfloat16_projections()``) rounding
# both to bfloat16, which is where a bfloat16 run rounds.
_round = [lambda t: t]


class bfloat16_projections:
    def __enter__(self):
        _round.append(lambda t: t.to(torch.bfloat16).to(F64))

    def __exit__(self, *exc):
        _round.pop()


def linear(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x W^T (+ b) for a weight stored [out, in]."""
    r = _round[-1]
    y = r(x) @ weight.t()
    return r(y if bias is None else y + bias)


def read_model_folder(folder: str):
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    w = {}
    with safe_open(os.path.join(folder, "model.safetensors"), framework="pt") as f:
        for name in f.keys():
            t = f.get_tensor(name)
            w[name] = t.to(F64) if t.is_floating_point() else t
    return config, w


# ---------------------------------------------------------------------- small functions
def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


# ---------------------------------------------------------------------- rotation with stretched slow frequencies
def frequencies(rot: dict) -> torch.Tensor:
    """One frequency per pair: kept where its wavelength is short beside the original context, divided by ``factor`` where
    it is long, and a blend of the two in between."""
    s, out = rot.get("scaling"), []
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        if s is not None:
            turns = s["original"] * f / (2.0 * math.pi)  # how often the pair turns within the original context
            if turns < s["low"]:
                f = f / s["factor"]
            elif turns <= s["high"]:
                share = (turns - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - share) * f / s["factor"] + share * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_halves(v: torch.Tensor, positions: Sequence[int], rot: dict) -> torch.Tensor:
    """v [T, heads, D]: of the first ``dims`` values, value i turns with value i + dims / 2."""
    half = rot["dims"] // 2
    a = torch.tensor(list(positions), dtype=F64)[:, None] * frequencies(rot)[None, :]
    cos, sin = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    out = v.clone()
    u, s = v[..., :half], v[..., half:2 * half]
    out[..., :half] = u * cos - s * sin
    out[..., half:2 * half] = s * cos + u * sin
    return out


# ---------------------------------------------------------------------- windowed attention
def new_keys(h: torch.Tensor, w, pre: str, m: dict, eps: float, positions: Sequence[int]):
    """What a layer with keys of its own adds to its cache: (keys [T, G, D] normed and rotated, values [T, G, Dv])."""
    T, G, D, Dv = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    k = unit_rms(linear(h, w[pre + "k"], w[pre + "k.b"]).view(T, G, D), eps) * w[pre + "k.norm"]
    return _round[-1](rotate_halves(k, positions, m["rot"])), linear(h, w[pre + "v"], w[pre + "v.b"]).view(T, G, Dv)


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, positions: Sequence[int], scale: float, window: int):
    """q [T, H, D] at ``positions``, all keys k [n, G, D] and values v [n, G, Dv] of the request: softmax over the last
    ``window`` positions with a one in the denominator.  Returns [T, H, Dv]."""
    T, H, _ = q.shape
    n, G, Dv = v.shape
    out = torch.zeros(T, H, Dv, dtype=F64)
    back = torch.tensor(list(positions))[:, None] - torch.arange(n)[None, :]
    seen = (back >= 0) & (back < window)
    for head in range(H):
        g = head // (H // G)
        s = torch.where(seen, q[:, head] @ k[:, g].t() * scale, torch.tensor(-math.inf, dtype=F64))
        top = s.max(dim=1).values.clamp(min=0.0)[:, None]
        e = torch.exp(s - top)
        out[:, head] = e @ v[:, g] / (e.sum(1, keepdim=True) + torch.exp(-top))
    return out


def attention(h: torch.Tensor, w, pre: str, m: dict, eps: float, positions: Sequence[int], st: dict) -> torch.Tensor:
    """``st``: the keys and values this layer reads; a layer with ``kv_from`` is handed the other layer's."""
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = unit_rms(linear(h, w[pre + "q"], w[pre + "q.b"]).view(T, H, D), eps) * w[pre + "q.norm"]
    q = _round[-1](rotate_halves(q, positions, m["rot"]))
    if m.get("kv_from") is None:
        k, v = new_keys(h, w, pre, m, eps, positions)
        st["k"], st["v"] = torch.cat([st["k"], k]), torch.cat([st["v"], v])
    o = attend(q, st["k"], st["v"], positions, float(m["scale"]), int(m["mask"]["size"]))
    return linear(o.reshape(T, H * Dv), w[pre + "o"], w[pre + "o.b"])


# ---------------------------------------------------------------------- time mixing
def shifted(h: torch.Tensor, before: torch.Tensor) -> torch.Tensor:
    """h [T, W] moved back by one token; ``before`` [W] is the input ahead of the first one."""
    return torch.cat([before[None], h])[:-1]


def log_decay(mix: torch.Tensor, w, pre: str) -> torch.Tensor:
    return -torch.exp(torch.tanh(_round[-1](mix) @ w[pre + "w1"].t()) @ w[pre + "w2"].t() + w[pre + "w0"])


def time_mixing_memory(r, k, v, logw, u, S):
    """r, k, logw [T, H, D], v [T, H, Dv], u [H, D], S [H, D, Dv]: the output reads the state before the token, the token
    itself with the bonus; then the state takes the decay of every key channel and the token.  (o [T, H, Dv], S)."""
    out = []
    for t in range(r.shape[0]):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(((S + u[:, :, None] * kv) * r[t][:, :, None]).sum(1))
        S = torch.exp(logw[t])[:, :, None] * S + kv
    return torch.stack(out), S


def time_mixing(h: torch.Tensor, w, pre: str, m: dict, eps: float, st: dict) -> torch.Tensor:
    T, H, D = h.shape[0], m["heads"], m["dim"]
    step = shifted(h, st["h"]) - h
    mixes = {s: h + step * w[pre + "mu." + s] for s in "rkvgw"}
    st["h"] = h[-1]
    r, k, v = (linear(mixes[s], w[pre + s]).view(T, H, D) for s in "rkv")
    logw = log_decay(mixes["w"], w, pre).view(T, H, D)
    o, st["S"] = time_mixing_memory(r, k, v, logw, w[pre + "u"], st["S"])
    o = unit_rms(o, eps).reshape(T, H * D) * w[pre + "norm"] * silu(linear(mixes["g"], w[pre + "g"]))
    return linear(o, w[pre + "o"])


# ---------------------------------------------------------------------- feed-forwards
def dense(h: torch.Tensor, w, pre: str) -> torch.Tensor:
    p = {s: linear(h, w[pre + s], w[pre + s + ".b"]) for s in ("gate", "up")}
    return linear(gelu_tanh(p["gate"]) * p["up"], w[pre + "down"], w[pre + "down.b"])


def limited_expert(h: torch.Tensor, w, pre: str, limit: float) -> torch.Tensor:
    """Gate and up values held back by ``limit`` (the gate from above only); the gate's sigmoid is steeper than silu's and
    the up value is moved by one."""
    g = linear(h, w[pre + "gate"]).clamp(max=limit)
    u = linear(h, w[pre + "up"]).clamp(min=-limit, max=limit)
    return linear(g * sigmoid(1.702 * g) * (u + 1.0), w[pre + "down"])


def route(z: torch.Tensor, top: int):
    """Logits of one token -> (the chosen experts, their weights: a softmax over the chosen logits)."""
    chosen = sorted(range(z.numel()), key=lambda e: (-float(z[e]), e))[:top]
    s = torch.exp(z[chosen] - z[chosen].max())
    return chosen, s / s.sum()


def experts(h: torch.Tensor, w, pre: str, mlp: dict) -> torch.Tensor:
    r = _round[-1]
    z = r(h) @ w[pre + "router"].t() + w[pre + "router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        x = h[t:t + 1]
        for e, s in zip(*route(z[t], mlp["router"]["top"])):
            out[t] += s * limited_expert(x, w, f"{pre}e{e}.", float(mlp["expert"]["limit"]))[0]
    if mlp.get("shared"):
        share = sigmoid(r(h) @ w[pre + "shared.sg"].t())
        out = out + share * limited_expert(h, w, pre + "shared.", float(mlp["shared"]["limit"]))
    return out


# ---------------------------------------------------------------------- a request's states and the whole model
def new_state(config: dict) -> List[dict]:
    states = []
    for entry in config["layers"]:
        m, z = entry["mixer"], lambda *s: torch.zeros(*s, dtype=F64)
        if entry["type"] == "wkv":
            st = {"S": z(m["heads"], m["dim"], m["dim"]), "h": z(config["width"])}
        elif m.get("kv_from") is None:
            st = {"k": z(0, m["kv_heads"], m["dim"]), "v": z(0, m["kv_heads"], m["vdim"])}
        else:
            st = {}
        st["length"] = 0
        states.append(st)
    return states


def forward(config: dict, w, tokens: Sequence[int], state: Optional[List[dict]] = None,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of a request's next ``tokens``; ``state`` (``new_state``) carries what earlier portions left."""
    if state is None:
        state = new_state(config)
    eps = float(config["norm"]["eps"])
    start = state[0]["length"]
    positions = list(range(start, start + len(tokens)))
    x = w["embed"][torch.tensor(list(tokens))].clone()
    for i, entry in enumerate(config["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        if entry["type"] == "wkv":
            y = time_mixing(x, w, p + "mix.", m, eps, state[i])
        else:
            source = i if m.get("kv_from") is None else m["kv_from"]
            y = attention(x, w, p + "mix.", m, eps, positions, state[source])
        x = x + unit_rms(y, eps) * w[p + "norm1"] * w[p + "ls1"]
        mlp = entry["mlp"]
        if mlp is not None:
            y = dense(x, w, p + "mlp.") if mlp["kind"] == "dense" else experts(x, w, p + "mlp.", mlp)
            x = x + unit_rms(y, eps) * w[p + "norm2"] * w[p + "ls2"]
        state[i]["length"] = start + len(tokens)
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(unit_rms(x, eps) * w["final.norm"], w["head"])


def forward_logits(config: dict, w, ids: Sequence[int]) -> torch.Tensor:
    return forward(config, w, ids)


def rounding_error(config: dict, w, ids: Sequence[int]) -> float:
    """The largest difference that rounding every projection's operand and result to bfloat16 makes to a logit of this
    prompt, relative to the largest logit."""
    exact = forward(config, w, ids)
    with bfloat16_projections():
        rounded = forward(config, w, ids)
    return float((rounded - exact).abs().max()) / float(exact.abs().max())


def greedy(config: dict, w, prompt: Sequence[int], new_tokens: int):
    """(generated ids, gap between the two largest logits at every step), token by token through the states."""
    state = new_state(config)
    logits = forward(config, w, prompt, state)
    out, margins = [], []
    for _ in range(new_tokens):
        top = torch.topk(logits[-1], 2).values
        margins.append(float(top[0] - top[1]))
        out.append(int(torch.argmax(logits[-1])))
        logits = forward(config, w, [out[-1]], state)
    return out, margins
