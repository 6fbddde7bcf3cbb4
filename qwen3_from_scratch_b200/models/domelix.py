"""Domelix as a model specification: blocks whose mixer and feed-forward read the same stream side by side, each behind an
RMS norm whose weight is stored around zero; per layer one of three mixers (softmax attention with a distance bias, a
sink and output gates beside lightning attention, each output normed, half their sum; the gated delta rule behind short
convolutions; retention with a rotation); a feed-forward of routed gated experts, chosen by softmax within the best groups
and weighted by their renormalised scores, or none.

Tensor names: ``embed``, ``head``, ``final.norm``, per layer ``l<i>.norm1`` / ``norm2``, ``l<i>.mix.*`` (parallel:
``left.{q,k,v,g,rel,sink,o,out}`` and ``right.{q,k,v,g,norm,o,out}``; delta: ``q, q.conv, k, k.conv, v, v.conv, b, a, A_log,
dt_bias, g, norm, o``; retention: ``q, k, v, g, o``), ``l<i>.mlp.{router, e<n>.{gate,up,down}}``.
"""

from __future__ import annotations

from ..config.domelix_config import ARCHITECTURE, DomelixConfig, DomelixLayer
from ..parts.base import LayerCall, ModelSpec, PartSpec
from ..registry import register_architecture

# constants of the design (what config.json cannot change)
EXPERT_ACTIVATION = "silu"  # experts: W_down (silu(W_gate h) * (W_up h))
BRANCH_SHARE = 0.5          # the parallel mixer: half the sum of the two normed outputs
RANDOM_BIAS_ROWS = 32       # rows of a distance bias's table where weights are made up (a folder's table has its own)
_BLOCK_NAMES = {"norm1": "norm1", "mixer": "mix", "norm2": "norm2", "feed_forward": "mlp"}


def _mixer(layer: DomelixLayer, cfg: DomelixConfig) -> PartSpec:
    m = layer.mixer
    if layer.type == "delta":
        return PartSpec("gated_delta", {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads,
                                        "dim": m.dim, "vdim": m.vdim, "conv": m.conv, "norm_eps": cfg.norm_eps})
    if layer.type == "retention":
        return PartSpec("decayed_memory", {
            "hidden_size": cfg.width, "num_heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": m.decay,
            "norm_eps": cfg.norm_eps, "norm": "heads", "gate": "silu",
            # the keys' factor dim^-1/2 on the queries instead: the same read-out, the state without the factor
            "q_scale": m.dim ** -0.5,
            "position": PartSpec("rotary_stretched", {"dims": m.rot_dims, "base": m.rot_base})})
    a, b = m.left, m.right
    left = PartSpec("kept_window_attention", {
        "hidden_size": cfg.width, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim,
        "scale": a.scale, "gate": True, "sink": True, "bias": {"most": a.bias_max, "rows": RANDOM_BIAS_ROWS}})
    right = PartSpec("decayed_memory", {
        "hidden_size": cfg.width, "num_heads": b.heads, "dim": b.dim, "vdim": b.vdim, "decay": b.decay,
        "norm_eps": cfg.norm_eps, "activation": "silu", "norm": "row", "norm_weight": True, "gate": "sigmoid"})
    return PartSpec("parallel", {"hidden_size": cfg.width, "out_norm": {"suffix": "out", "eps": cfg.norm_eps}, "branches": [
        {"label": "left", "mixer": left, "scale": BRANCH_SHARE}, {"label": "right", "mixer": right, "scale": BRANCH_SHARE}]})


def _feed_forward(layer: DomelixLayer, cfg: DomelixConfig):
    e = layer.mlp
    if e is None:
        return None
    return PartSpec("routed_experts", {"hidden_size": cfg.width, "experts": e.experts, "top": e.top, "expert_ff": e.expert_ff,
                                       "activation": EXPERT_ACTIVATION, "correction": False, "gated": True,
                                       "score": "softmax", "groups": (e.groups, e.keep), "renormalise": True})


@register_architecture(ARCHITECTURE, DomelixConfig)
def domelix_spec(cfg: DomelixConfig) -> ModelSpec:
    norm = PartSpec("rms_norm", {"dim": cfg.width, "eps": cfg.norm_eps, "suffix": "", "one_plus": True})
    layers, ignorable = [], []
    for i, layer in enumerate(cfg.layers):
        ff = _feed_forward(layer, cfg)
        if ff is None:  # a folder may still carry the norm in front of a feed-forward that is not there
            ignorable.append(f"l{i}.norm2")
        layers.append((f"l{i}", PartSpec("parallel_pre_norm", {"norm1": norm, "mixer": _mixer(layer, cfg),
                                                               "norm2": norm if ff else None, "feed_forward": ff,
                                                               "names": _BLOCK_NAMES})))
    return ModelSpec(
        embedding=("embed", PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "suffix": ""})),
        layers=layers, order=[LayerCall(layer=i, cache=i) for i in range(len(layers))],
        final_norm=("final.norm", norm),
        head=("head", PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "suffix": ""})),
        vocab_size=cfg.vocab,
        max_positions=1 << 30,  # nothing in the design depends on a longest position
        ignorable_weights=tuple(ignorable),
        eos_token_id=cfg.eos_token_id,
    )
