"""A plain, slow statement of the Domelix design in float64 on the CPU: one function per mechanism, written from the
mechanism's equations, sharing no code with the engine.  Whatever is carried from token to token (the keys and values
of the attention, the matrix states of the three linear memories, the tails of the short convolutions) is taken and
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


def linear(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """x W^T for a weight stored [out, in]."""
    r = _round[-1]
    return r(r(x) @ weight.t())


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


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.logaddexp(torch.zeros_like(z), z)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def norm_one_plus(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * (1.0 + weight)


def unit_length(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).sum(dim=-1, keepdim=True) + 1e-6)


def rotate_halves(v: torch.Tensor, positions: Sequence[int], base: float, dims: int) -> torch.Tensor:
    """v [T, heads, D]: of the first ``dims`` values, value i turns with value i + dims / 2."""
    if dims == 0:
        return v
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    a = torch.tensor(list(positions), dtype=F64)[:, None] * freq[None, :]
    cos, sin = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    half = dims // 2
    out = v.clone()
    u, s = v[..., :half], v[..., half:dims]
    out[..., :half] = u * cos - s * sin
    out[..., half:dims] = s * cos + u * sin
    return out


# ---------------------------------------------------------------------- attention with a distance bias and a sink
def bucket(n: int, rows: int, most: float) -> int:
    """Which row of a bias table of ``rows`` rows a distance of n tokens reads: one row per distance below rows / 2,
    then rows that widen with the logarithm of the distance, the last one from ``most`` on (or a little before)."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(most / half) * (rows - half)))


def attention(h: torch.Tensor, w, pre: str, m: dict, positions: Sequence[int], st: dict) -> torch.Tensor:
    """Grouped-query heads without rotation; every earlier token is read.  ``st["k"]`` [n, G, D], ``st["v"]`` [n, G, Dv]."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = linear(h, w[pre + "q"]).view(T, H, D)
    st["k"] = torch.cat([st["k"], linear(h, w[pre + "k"]).view(T, G, D)])
    st["v"] = torch.cat([st["v"], linear(h, w[pre + "v"]).view(T, G, Dv)])
    rel, sink = w[pre + "rel"], w[pre + "sink"]
    longest = max(positions)
    rows = torch.tensor([bucket(n, rel.shape[0], float(m["bias_max"])) for n in range(longest + 1)])
    out = torch.zeros(T, H, Dv, dtype=F64)
    n = st["k"].shape[0]
    back = torch.tensor(positions)[:, None] - torch.arange(n)[None, :]  # how far back a key is; negative: not yet there
    for head in range(H):
        g = head // (H // G)
        s = q[:, head] @ st["k"][:, g].t() * float(m["scale"]) + rel[rows[back.clamp(min=0)], head]
        s = torch.where(back >= 0, s, torch.tensor(-math.inf, dtype=F64))
        top = torch.maximum(s.max(dim=1).values, sink[head])[:, None]
        e = torch.exp(s - top)
        out[:, head] = e @ st["v"][:, g] / (e.sum(1) + torch.exp(sink[head] - top[:, 0]))[:, None]
    gated = out.reshape(T, H * Dv) * sigmoid(linear(h, w[pre + "g"]))
    return linear(gated, w[pre + "o"])


# ---------------------------------------------------------------------- memories with a decay per head
def decayed_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay, S: torch.Tensor):
    """q, k [T, H, D], v [T, H, Dv], S [H, D, Dv]: S <- decay_h S + k v^T; o = S^T q.  Returns (o [T, H, Dv], S)."""
    g = torch.tensor(list(decay), dtype=F64)[:, None, None]
    out = []
    for t in range(q.shape[0]):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def lightning(h: torch.Tensor, w, pre: str, m: dict, eps: float, st: dict) -> torch.Tensor:
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    r = _round[-1]
    q, k = r(silu(linear(h, w[pre + "q"]))).view(T, H, D), r(silu(linear(h, w[pre + "k"]))).view(T, H, D)
    v = r(silu(linear(h, w[pre + "v"]))).view(T, H, Dv)
    o, st["S"] = decayed_memory(q, k, v, m["decay"], st["S"])
    o = unit_rms(o.reshape(T, H * Dv), eps) * w[pre + "norm"]
    return linear(o * sigmoid(linear(h, w[pre + "g"])), w[pre + "o"])


def retention(h: torch.Tensor, w, pre: str, m: dict, eps: float, positions: Sequence[int], st: dict) -> torch.Tensor:
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    r = _round[-1]
    q = r(rotate_halves(linear(h, w[pre + "q"]).view(T, H, D), positions, base, dims))
    k = r(rotate_halves(linear(h, w[pre + "k"]).view(T, H, D), positions, base, dims)) * D ** -0.5
    v = linear(h, w[pre + "v"]).view(T, H, Dv)
    o, st["S"] = decayed_memory(q, k, v, m["decay"], st["S"])
    o = unit_rms(o, eps).reshape(T, H * Dv)
    return linear(o * silu(linear(h, w[pre + "g"])), w[pre + "o"])


# ---------------------------------------------------------------------- the gated delta rule
def short_conv(x: torch.Tensor, taps: torch.Tensor, tail: torch.Tensor):
    """x [T, C], taps [C, K], tail [K - 1, C] the inputs before: y_t[c] = sum_j taps[c, j] x_(t - K + 1 + j)[c].
    Returns (y, the new tail)."""
    K = taps.shape[1]
    seen = torch.cat([tail, x])
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(K):
            y[t] += taps[:, j] * seen[t + j]
    return y, seen[seen.shape[0] - (K - 1):]


def delta(h: torch.Tensor, w, pre: str, m: dict, eps: float, st: dict) -> torch.Tensor:
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    r = _round[-1]
    parts = {}
    for x in ("q", "k", "v"):
        y, st[x] = short_conv(linear(h, w[pre + x]), w[pre + x + ".conv"], st[x])
        parts[x] = r(silu(y))
    q = unit_length(parts["q"].view(T, G, D)) * D ** -0.5
    k = unit_length(parts["k"].view(T, G, D))
    v = parts["v"].view(T, H, Dv)
    beta = sigmoid(linear(h, w[pre + "b"]))
    g = torch.exp(-torch.exp(w[pre + "A_log"]) * softplus(linear(h, w[pre + "a"]) + w[pre + "dt_bias"]))
    S, out = st["S"], []
    of = torch.arange(H) // (H // G)
    for t in range(T):
        kt, qt = k[t][of], q[t][of]
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (S * kt[:, :, None]).sum(1))
        S = S + kt[:, :, None] * u[:, None, :]
        out.append((S * qt[:, :, None]).sum(1))
    st["S"] = S
    o = unit_rms(torch.stack(out), eps) * w[pre + "norm"]
    return linear(o.reshape(T, H * Dv) * silu(linear(h, w[pre + "g"])), w[pre + "o"])


# ---------------------------------------------------------------------- routed experts
def route(z: torch.Tensor, router: dict):
    """Logits of one token -> (the chosen experts, their weights)."""
    E, top = router["experts"], router["top"]
    groups, keep = router["groups"]["count"], router["groups"]["keep"]
    s = torch.exp(z - z.max())
    s = s / s.sum()
    per = E // groups
    best = sorted(range(groups), key=lambda n: (-float(s[n * per:(n + 1) * per].max()), n))[:keep]
    allowed = [e for e in range(E) if e // per in best]
    chosen = sorted(allowed, key=lambda e: (-float(s[e]), e))[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20)


def experts(h: torch.Tensor, w, pre: str, mlp: dict) -> torch.Tensor:
    r = _round[-1]
    z = r(h) @ w[pre + "router"].t()
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, weights = route(z[t], mlp["router"])
        x = h[t:t + 1]
        for e, s in zip(chosen, weights):
            p = f"{pre}e{e}."
            out[t] += s * linear(silu(linear(x, w[p + "gate"])) * linear(x, w[p + "up"]), w[p + "down"])[0]
    return out


# ---------------------------------------------------------------------- a request's states and the whole model
def new_state(config: dict) -> List[dict]:
    states = []
    for entry in config["layers"]:
        m, z = entry["mixer"], lambda *s: torch.zeros(*s, dtype=F64)
        if entry["type"] == "parallel":
            a, b = m["left"], m["right"]
            st = {"left": {"k": z(0, a["kv_heads"], a["dim"]), "v": z(0, a["kv_heads"], a["vdim"])},
                  "right": {"S": z(b["heads"], b["dim"], b["vdim"])}}
        elif entry["type"] == "delta":
            qk = m["kv_heads"] * m["dim"]
            st = {"S": z(m["heads"], m["dim"], m["vdim"]), "q": z(m["conv"] - 1, qk), "k": z(m["conv"] - 1, qk),
                  "v": z(m["conv"] - 1, m["heads"] * m["vdim"])}
        else:
            st = {"S": z(m["heads"], m["dim"], m["vdim"])}
        st["length"] = 0
        states.append(st)
    return states


def branches(h: torch.Tensor, w, pre: str, m: dict, eps: float, positions: Sequence[int], st: dict) -> torch.Tensor:
    """Two mixers side by side on the same input: half the sum of their outputs, each normed over the width."""
    a = attention(h, w, pre + "left.", m["left"], positions, st["left"])
    b = lightning(h, w, pre + "right.", m["right"], eps, st["right"])
    return 0.5 * (unit_rms(a, eps) * w[pre + "left.out"] + unit_rms(b, eps) * w[pre + "right.out"])


def mixer(h: torch.Tensor, w, pre: str, entry: dict, eps: float, positions: Sequence[int], st: dict) -> torch.Tensor:
    if entry["type"] == "parallel":
        return branches(h, w, pre, entry["mixer"], eps, positions, st)
    if entry["type"] == "delta":
        return delta(h, w, pre, entry["mixer"], eps, st)
    return retention(h, w, pre, entry["mixer"], eps, positions, st)


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
        p = f"l{i}."
        y = mixer(norm_one_plus(x, w[p + "norm1"], eps), w, p + "mix.", entry, eps, positions, state[i])
        if entry["mlp"] is not None:
            y = y + experts(norm_one_plus(x, w[p + "norm2"], eps), w, p + "mlp.", entry["mlp"])
        x = x + y
        state[i]["length"] = start + len(tokens)
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(norm_one_plus(x, w["final.norm"], eps), w["head"])


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
