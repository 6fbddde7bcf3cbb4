"""Zasitar as a model specification: blocks whose sub-layers read the residual stream itself, with an RMS norm and a scale per
feature on their outputs; per layer RWKV-style time mixing, or attention over a sliding window with biases on its
projections, a norm per head, a rotation whose slow frequencies are stretched and a one in the softmax's denominator, which
may read the keys and values of an earlier layer; a dense feed-forward with biases, routed experts beside a shared one with
a gate of its own, or none.

Tensor names: ``embed``, ``head``, ``final.norm``, per layer ``l<i>.norm1`` / ``norm2`` / ``ls1`` / ``ls2``, ``l<i>.mix.*`` (wkv:
``mu.{r,k,v,g,w}, r, k, v, g, w1, w2, w0, u, norm, o``; attention: ``q, q.b, q.norm, k, k.b, k.norm, v, v.b, o, o.b``, without
those of k and v where the layer reads another's), ``l<i>.mlp.*`` (dense: ``{gate,up,down}`` and ``.b`` of each; experts:
``router, router.b, e<n>.{gate,up,down}, shared.{gate,up,down,sg}``).
"""

from __future__ import annotations

from ..config.zasalix_config import DenseFF
from ..config.zasitar_config import ARCHITECTURE, LimitedFF, ZasitarConfig, ZasitarLayer
from ..parts.base import LayerCall, ModelSpec, PartSpec
from ..registry import register_architecture

# constants of the design (what config.json cannot change)
DENSE_ACTIVATION = "gelu_tanh"    # dense: W_down (gelu(W_gate h) * (W_up h)), the tanh form
EXPERT_ACTIVATION = "limited"     # experts: gate and up value held back by the limit, g sigmoid(1.702 g) (u + 1)
SINK_LOGIT = 0.0                  # attention: a one in the softmax's denominator
RANDOM_DECAY_RANK = 64            # rank of the decay's projection where weights are made up (a folder's tensors have their own)
_BLOCK_NAMES = {"norm1": "norm1", "mixer": "mix", "norm2": "norm2", "feed_forward": "mlp", "scale1": "ls1", "scale2": "ls2"}
_MLP_NAMES = {"gate": "gate", "up": "up", "down": "down", "gate_bias": "gate.b", "up_bias": "up.b", "down_bias": "down.b"}


def _mixer(layer: ZasitarLayer, cfg: ZasitarConfig) -> PartSpec:
    m = layer.mixer
    if layer.type == "wkv":
        return PartSpec("time_mixing", {"hidden_size": cfg.width, "num_heads": m.heads, "dim": m.dim, "norm_eps": cfg.norm_eps,
                                        "rank": RANDOM_DECAY_RANK})
    s = m.rot_scaling
    scaling = None if s is None else {"factor": s.factor, "low": s.low, "high": s.high, "original": s.original}
    return PartSpec("kept_window_attention", {
        "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim,
        "scale": m.scale, "window": m.window, "gate": False, "fixed_sink": SINK_LOGIT, "proj_bias": True,
        "qk_norm_eps": cfg.norm_eps, "shares_kv": m.kv_from is not None,
        "position": PartSpec("rotary_banded", {"dims": m.rot_dims, "base": m.rot_base, "scaling": scaling})})


def _feed_forward(layer: ZasitarLayer, cfg: ZasitarConfig):
    e = layer.mlp
    if e is None:
        return None
    if isinstance(e, DenseFF):
        return PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": e.ff, "activation": DENSE_ACTIVATION,
                                      "bias": True, "names": _MLP_NAMES})

    def shared(s: LimitedFF) -> PartSpec:
        return PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": s.ff, "activation": EXPERT_ACTIVATION,
                                      "limit": s.limit, "names": _MLP_NAMES})

    return PartSpec("routed_experts", {
        "hidden_size": cfg.width, "experts": e.experts, "top": e.top, "expert_ff": e.expert.ff, "activation": EXPERT_ACTIVATION,
        "limit": e.expert.limit, "correction": False, "gated": True, "score": "softmax", "renormalise": True,
        "router_bias": True, "shared": shared(e.shared) if e.shared else None, "shared_gate": e.shared is not None})


@register_architecture(ARCHITECTURE, ZasitarConfig)
def zasitar_spec(cfg: ZasitarConfig) -> ModelSpec:
    norm = PartSpec("rms_norm", {"dim": cfg.width, "eps": cfg.norm_eps, "suffix": ""})
    layers, order, ignorable = [], [], []
    for i, layer in enumerate(cfg.layers):
        ff = _feed_forward(layer, cfg)
        if ff is None:  # a folder may still carry the norm and the scale of a feed-forward that is not there
            ignorable += [f"l{i}.norm2", f"l{i}.ls2"]
        layers.append((f"l{i}", PartSpec("output_norm", {
            "width": cfg.width, "norm1": norm, "mixer": _mixer(layer, cfg), "norm2": norm if ff else None, "feed_forward": ff,
            "layer_scale": True, "names": _BLOCK_NAMES})))
        source = layer.mixer.kv_from if layer.type == "attention" else None
        order.append(LayerCall(layer=i, cache=i if source is None else source, write_cache=source is None))
    return ModelSpec(
        embedding=("embed", PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "suffix": ""})),
        layers=layers, order=order,
        final_norm=("final.norm", norm),
        head=("head", PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "suffix": ""})),
        vocab_size=cfg.vocab,
        max_positions=1 << 30,  # nothing in the design depends on a longest position
        ignorable_weights=tuple(ignorable),
        eos_token_id=cfg.eos_token_id,
    )
