"""Attention mixers over a paged cache: grouped-query softmax attention (with optional per-head RMSNorm of q and
k, an optional position encoding and an optional sliding window), sigmoid attention whose values are its keys,
softmax attention through a latent (one latent vector and one rotated key part per token, shared by the heads; with
optional output gates and an optional sink in the softmax), softmax attention over a window and pooled blocks, and
softmax attention over a window that also keeps a request's first tokens, or over all tokens with a bias by distance and
a sink (or with biases on the projections, a norm per head, a fixed sink, the keys and values of another layer).

Reference: models/self_attn.py:300-386 (packed [T, hidden] input, merged QKV, head norm then
rotation, keys/values written to pages, causal attention over the cache, output projection),
models/attn.py:388-499 (scale = head_dim^-0.5, q head h reads kv head h // (Hq / Hkv)).
The window (a query at position p reads keys p - window < n <= p) is what config.json's
``sliding_window`` asks of a layer; the reference itself never reads that key.
In a step where every row brings one token the decode attention kernel does the head norm, the
rotation and the page write itself, from the raw QKV projection.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

from ..kernels import ops
from ..registry import create_part, register_part
from .base import (CachePlane, KVCacheSpec, Mixer, PagedCacheSpec, PartSpec, PendingTerm, Runtime, StepContext, WeightSpec)
from .linear import Linear


@register_part("mixer", "gqa_attention")
class GQAAttention(Mixer):
    graph_capturable = True

    def __init__(self, name: str, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int,
                 qk_norm_eps: Optional[float] = None, position: Optional[PartSpec] = None,
                 window: Optional[int] = None):
        super().__init__(name)
        self.hidden_size = int(hidden_size)
        self.num_heads, self.num_kv_heads, self.head_dim = int(num_heads), int(num_kv_heads), int(head_dim)
        if self.num_heads % self.num_kv_heads:
            raise ValueError(f"{self.num_heads} query heads are not a multiple of {self.num_kv_heads} kv heads")
        self.qk_norm_eps = None if qk_norm_eps is None else float(qk_norm_eps)
        self.window = None if window is None else int(window)
        self.position = create_part("position", position, name=f"{name}.position") if position else None
        self.scale = float(self.head_dim) ** -0.5

    # ------------------------------------------------------------------ declarations
    def weight_specs(self) -> List[WeightSpec]:
        h, d = self.hidden_size, self.head_dim
        specs = [WeightSpec(f"{self.name}.q_proj.weight", (self.num_heads * d, h)),
                 WeightSpec(f"{self.name}.k_proj.weight", (self.num_kv_heads * d, h)),
                 WeightSpec(f"{self.name}.v_proj.weight", (self.num_kv_heads * d, h)),
                 WeightSpec(f"{self.name}.o_proj.weight", (h, self.num_heads * d))]
        if self.qk_norm_eps is not None:
            specs += [WeightSpec(f"{self.name}.q_norm.weight", (d,), kind="vector", init="one_plus_normal"),
                      WeightSpec(f"{self.name}.k_norm.weight", (d,), kind="vector", init="one_plus_normal")]
        if self.position is not None:
            specs += self.position.weight_specs()
        return specs

    def cache_spec(self) -> KVCacheSpec:
        return KVCacheSpec(self.num_kv_heads, self.head_dim, self.window)

    # ------------------------------------------------------------------ device side
    def setup(self, rt: Runtime, weights: Dict[str, torch.Tensor]) -> None:
        super().setup(rt, weights)
        q = weights.pop(f"{self.name}.q_proj.weight")
        k = weights.pop(f"{self.name}.k_proj.weight")
        v = weights.pop(f"{self.name}.v_proj.weight")
        dtype = torch.float32 if torch.float32 in (q.dtype, k.dtype, v.dtype) else q.dtype
        merged = torch.cat([q.to(dtype), k.to(dtype), v.to(dtype)], dim=0)  # rows ordered q, k, v
        del q, k, v
        self.qkv = Linear(merged, rt, tag="attn.qkv")
        self.o_proj = Linear(weights.pop(f"{self.name}.o_proj.weight"), rt, tag="attn.o_proj")
        self.q_norm_weight = self.k_norm_weight = None
        if self.qk_norm_eps is not None:
            self.q_norm_weight = weights[f"{self.name}.q_norm.weight"]
            self.k_norm_weight = weights[f"{self.name}.k_norm.weight"]
        if self.position is not None:
            self.position.setup(rt, weights)
        self._q = rt.shared("attn.q", rt.max_tokens, self.num_heads, self.head_dim)
        self._o = rt.shared("attn.o", rt.max_tokens, self.num_heads, self.head_dim)
        self._partial = None
        if ops.fast_attention_takes(rt.dtype, self.num_heads, self.num_kv_heads, self.head_dim):
            self._partial = rt.shared("attn.partial", ops.decode_partial_numel(rt.max_seqs, self.num_heads,
                                                                               self.head_dim), dtype=torch.float32)

    fuses_stream = True

    def can_fuse_stream(self, rows: int) -> bool:
        return self.qkv.takes_stream_norm(rows) and self.o_proj.can_add_into_stream(rows)

    def forward(self, x, ctx: StepContext, cache_id: Optional[int], write_cache: bool, into_stream=None,
                next_norm_weight=None):
        """``x``: the normed activations, or a ``StreamNorm`` that the QKV product applies itself.
        ``into_stream``: the output projection adds into this stream and its ``StreamStats`` are returned
        (with the rows times ``next_norm_weight`` if that is given)."""
        T = x.shape[0]
        hq, hkv, d = self.num_heads, self.num_kv_heads, self.head_dim
        k_pages, v_pages, table = ctx.kv(cache_id)
        q = self._q[:T]
        eps = self.qk_norm_eps if self.qk_norm_eps is not None else 0.0
        fused = self.position.fused_rotary() if self.position is not None else None
        out = self._o[:T]
        whole_rotation = fused is None or fused[1] == d
        if ((self.position is None or fused is not None) and whole_rotation
                and ops.decode_takes_raw_qkv(self.rt.dtype, hq, hkv, d, k_pages.shape[2], T, ctx.num_seqs, ctx.num_decode)):
            # every row decodes: the attention kernel norms and rotates its own query and the new key itself
            # (the step's angles are made before the projection, so that the kernel may fetch them early)
            cos_sin = self.position.step_table(ctx) if fused is not None else None
            qkv = self.qkv(x)
            raw = (qkv, self.q_norm_weight, self.k_norm_weight, eps, cos_sin, write_cache)
            self.attend(q, k_pages, v_pages, table, ctx, out, raw_qkv=raw)
            if into_stream is not None:
                return self.o_proj.into_stream(out.view(T, hq * d), into_stream, next_norm_weight)
            return self.o_proj(out.view(T, hq * d))
        if ((self.position is None or fused is not None) and torch.is_tensor(x)
                and ops.gemm_tc_qkv_takes(T, x, self.qkv.weight, d, fused[1] if fused is not None else 0)
                and ops.gemm_tc_qkv_pays(T, self.qkv.weight)):
            # a prompt portion: the projection's own epilogue norms, rotates and writes the pages
            cos_sin = self.position.step_table(ctx) if fused is not None else None
            ops.gemm_tc_qkv(x, self.qkv.weight, q, k_pages, v_pages, self.q_norm_weight, self.k_norm_weight, eps,
                            cos_sin, ctx.positions, ctx.tok_seq, table, hq, hkv, d, write_cache, self.rt.status,
                            pair=ops.gemm_tc_qkv_pays(T, self.qkv.weight) == "pair")
            self.attend(q, k_pages, v_pages, table, ctx, out)
            if into_stream is not None:
                return self.o_proj.into_stream(out.view(T, hq * d), into_stream, next_norm_weight)
            return self.o_proj(out.view(T, hq * d))
        qkv = self.qkv(x)
        if self.position is None or fused is not None:
            inv_freq, rotary_dim = fused if fused is not None else (None, 0)
            cos_sin = self.position.step_table(ctx) if fused is not None else None
            ops.qkv_post(qkv, q, k_pages, v_pages, self.q_norm_weight, self.k_norm_weight, eps, inv_freq,
                         rotary_dim, ctx.positions, ctx.tok_seq, table, hq, hkv, d, write_cache, self.rt.status,
                         cos_sin=cos_sin)
        else:
            # a position encoding the kernel does not know: norm, encode, then scatter, as separate steps
            heads = qkv.view(T, hq + 2 * hkv, d)
            qh = heads[:, :hq].contiguous()
            kh = heads[:, hq:hq + hkv].contiguous()
            if self.qk_norm_eps is not None:
                qn, kn = torch.empty_like(qh), torch.empty_like(kh)
                ops.rmsnorm(qh, self.q_norm_weight, qn, eps)
                ops.rmsnorm(kh, self.k_norm_weight, kn, eps)
                qh, kh = qn, kn
            heads[:, :hq].copy_(self.position.apply(qh, ctx.positions))
            heads[:, hq:hq + hkv].copy_(self.position.apply(kh, ctx.positions))
            ops.qkv_post(qkv, q, k_pages, v_pages, None, None, 0.0, None, 0, ctx.positions, ctx.tok_seq, table,
                         hq, hkv, d, write_cache, self.rt.status)
        self.attend(q, k_pages, v_pages, table, ctx, out)
        if into_stream is not None:
            return self.o_proj.into_stream(out.view(T, hq * d), into_stream, next_norm_weight)
        return self.o_proj(out.view(T, hq * d))

    def attend(self, q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, table: torch.Tensor,
               ctx: StepContext, out: torch.Tensor, raw_qkv=None) -> None:
        """Causal attention of this step's queries over the pages (keys of this step included)."""
        ops.paged_attention(q, k_pages, v_pages, out, ctx.q_start, ctx.kv_len, ctx.tok_seq, table, ctx.num_seqs,
                            ctx.num_decode, ctx.max_q_len, ctx.max_kv_len, self.scale, self.window or 0,
                            self.rt.status, self._partial, raw_qkv=raw_qkv)


@register_part("mixer", "sigmoid_attention")
class SigmoidAttention(Mixer):
    """Grouped-query causal attention whose weights are not normalised over the keys: a visible key n gets
    sigmoid(q . k_n * scale + b_h), b_h one learned number per head, and the weighted values are summed as they
    are.  The values are the keys as projected (there is no value projection): the cache holds the normed key in
    plane ``k`` and the key before its norm in plane ``v``.  q and k are RMS-normed per head with one weight per
    kind, shared by the heads; there is no rotation, positions enter through the causal mask and, optionally,
    through a temperature on the query, tau(p) = 1 + coef * ln(floor((p + 1) / every) + 1).  Each head's output
    is multiplied by sigmoid(W_g h)_h, a gate read from the mixer's input, before the output projection.
    Scores, weights, norms, the temperature and the gate are float32 in every run.

    One product gives q, k and the gates (``names``: the tensors' names after the part's own)."""

    graph_capturable = True
    NAMES = {"q": "q", "k": "k", "q_norm": "q.norm", "k_norm": "k.norm", "head_bias": "pb", "gate": "g", "out": "o"}

    def __init__(self, name: str, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, scale: float,
                 qk_norm_eps: float, temp_coef: float = 0.0, temp_every: int = 0,
                 names: Optional[Dict[str, str]] = None):
        super().__init__(name)
        self.hidden_size = int(hidden_size)
        self.num_heads, self.num_kv_heads, self.head_dim = int(num_heads), int(num_kv_heads), int(head_dim)
        if self.num_heads % self.num_kv_heads:
            raise ValueError(f"{self.num_heads} query heads are not a multiple of {self.num_kv_heads} kv heads")
        self.scale, self.qk_norm_eps = float(scale), float(qk_norm_eps)
        self.temp_coef, self.temp_every = float(temp_coef), int(temp_every)
        n = dict(self.NAMES)
        n.update(names or {})
        self.tensors = {k: f"{name}.{v}" for k, v in n.items()}

    def weight_specs(self) -> List[WeightSpec]:
        t, h, d = self.tensors, self.hidden_size, self.head_dim
        return [WeightSpec(t["q"], (self.num_heads * d, h)), WeightSpec(t["k"], (self.num_kv_heads * d, h)),
                WeightSpec(t["q_norm"], (d,), kind="vector", init="one_plus_normal"),
                WeightSpec(t["k_norm"], (d,), kind="vector", init="one_plus_normal"),
                WeightSpec(t["head_bias"], (self.num_heads,), kind="vector", init="normal"),
                WeightSpec(t["gate"], (self.num_heads, h)),
                WeightSpec(t["out"], (h, self.num_heads * d))]

    def cache_spec(self) -> KVCacheSpec:
        return KVCacheSpec(self.num_kv_heads, self.head_dim)

    def setup(self, rt: Runtime, weights: Dict[str, torch.Tensor]) -> None:
        super().setup(rt, weights)
        t = self.tensors
        q, k, g = weights.pop(t["q"]), weights.pop(t["k"]), weights.pop(t["gate"])
        dtype = torch.float32 if torch.float32 in (q.dtype, k.dtype, g.dtype) else q.dtype
        self.proj = Linear(torch.cat([q.to(dtype), k.to(dtype), g.to(dtype)], dim=0), rt, tag="sattn.proj")
        del q, k, g
        self.o_proj = Linear(weights.pop(t["out"]), rt, tag="sattn.o_proj")
        self.q_norm_weight, self.k_norm_weight = weights[t["q_norm"]], weights[t["k_norm"]]
        self.head_bias = weights[t["head_bias"]]
        self._q = rt.shared("attn.q", rt.max_tokens, self.num_heads, self.head_dim)
        self._o = rt.shared("attn.o", rt.max_tokens, self.num_heads, self.head_dim)
        self._gate = rt.shared("sattn.gate", rt.max_tokens, self.num_heads, dtype=torch.float32)
        self._partial = None
        if ops.sigmoid_attention_fast(rt.dtype, self.num_heads, self.num_kv_heads, self.head_dim):
            self._partial = rt.shared("sattn.partial", ops.sigmoid_partial_numel(rt.max_seqs, self.num_heads,
                                                                                  self.head_dim), dtype=torch.float32)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache_id: Optional[int], write_cache: bool) -> torch.Tensor:
        T, hq, hkv, d = x.shape[0], self.num_heads, self.num_kv_heads, self.head_dim
        k_pages, v_pages, table = ctx.kv(cache_id)
        q, out, gate = self._q[:T], self._o[:T], self._gate[:T]
        ops.qk_gate_post(self.proj(x), q, k_pages, v_pages, self.q_norm_weight, self.k_norm_weight, self.qk_norm_eps,
                         self.temp_coef, self.temp_every, ctx.positions, ctx.tok_seq, table, hq, hkv, d, gate, write_cache,
                         self.rt.status)
        ops.sigmoid_attention(q, k_pages, v_pages, out, self.head_bias, gate, ctx.q_start, ctx.kv_len, ctx.tok_seq, table,
                              ctx.num_seqs, ctx.num_decode, ctx.max_q_len, ctx.max_kv_len, self.scale, self.rt.status,
                              partial=self._partial)
        return self.o_proj(out.view(T, hq * d))


@register_part("mixer", "latent_attention")
class LatentAttention(Mixer):
    """Causal softmax attention whose keys and values are made from one latent vector per token (the multi-head
    latent attention of DeepSeek-V2).  With h the input:

        c_q = rmsnorm(W_dq h) w_q;   q = W_uq c_q, per head [dim plain | rot_dim rotated]
        W_dkv h = [kv_rank values | rot_dim values]:  c = rmsnorm(first part) w_kv;  r = the rest, rotated, one for all heads
        score(head) = (q_plain . W_uk,head c + q_rot . r) * scale;   value(head) = W_uv,head c
        out = W_o concat_heads(sigmoid(W_g h)_head * softmax(scores) values)

    ``gate=False``: no W_g, the heads' outputs go to W_o as they are.  ``sink=True``: a learned logit per head
    (``<name>.sink``) that takes part in the softmax's denominator only, weights = exp(s_j) / (sum_j exp(s_j) + exp(sink)):
    nothing is scored for it, nothing is weighted by it, and ``scale`` is not applied to it.
    ``pairing``: which values of a rotated part turn together, "halves" (i with i + dims / 2) or "neighbours" (2i with
    2i + 1); the frequencies are the position part's either way.

    Per token the cache holds only c (plane ``c``) and r (plane ``r``), one "head" each.  Keys and values are never
    formed: the plain query is taken through W_uk once (q' = W_uk,head^T q_plain, ``kv_rank`` values), the kernels
    attend over the latents themselves, and the result goes through W_uv,head afterwards.  ``scale`` is used as given.
    Norms, angles, scores, weights and the gate are float32 in every run.  ``position``: a part with
    ``frequencies()`` (``rotary_stretched``); ``names``: the tensors' names after the part's own."""

    graph_capturable = True
    NAMES = {"dq": "dq", "dq_norm": "dq.norm", "uq": "uq", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv",
             "gate": "g", "out": "o", "sink": "sink"}

    def __init__(self, name: str, hidden_size: int, num_heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int,
                 q_rank: int, scale: float, norm_eps: float, position: PartSpec, names: Optional[Dict[str, str]] = None,
                 gate: bool = True, sink: bool = False, pairing: str = "halves"):
        super().__init__(name)
        self.has_gate, self.has_sink, self.pairing = bool(gate), bool(sink), str(pairing)
        ops.rotary_pairing(self.pairing)
        self.hidden_size, self.num_heads = int(hidden_size), int(num_heads)
        self.dim, self.rot_dim, self.vdim = int(dim), int(rot_dim), int(vdim)
        self.kv_rank, self.q_rank = int(kv_rank), int(q_rank)
        self.scale, self.norm_eps = float(scale), float(norm_eps)
        self.position = create_part("position", position, name=f"{name}.position")
        n = dict(self.NAMES)
        n.update(names or {})
        self.tensors = {k: f"{name}.{v}" for k, v in n.items()}

    def weight_specs(self) -> List[WeightSpec]:
        t, w, H = self.tensors, self.hidden_size, self.num_heads
        return [WeightSpec(t["dq"], (self.q_rank, w)),
                WeightSpec(t["dq_norm"], (self.q_rank,), kind="vector", init="one_plus_normal"),
                WeightSpec(t["uq"], (H * (self.dim + self.rot_dim), self.q_rank)),
                WeightSpec(t["dkv"], (self.kv_rank + self.rot_dim, w)),
                WeightSpec(t["dkv_norm"], (self.kv_rank,), kind="vector", init="one_plus_normal"),
                WeightSpec(t["uk"], (H * self.dim, self.kv_rank)),
                WeightSpec(t["uv"], (H * self.vdim, self.kv_rank))] + (
                    [WeightSpec(t["gate"], (H, w))] if self.has_gate else []) + (
                    [WeightSpec(t["sink"], (H,), kind="vector", init="normal")] if self.has_sink else []) + [
                WeightSpec(t["out"], (w, H * self.vdim))] + self.position.weight_specs()

    def cache_spec(self) -> PagedCacheSpec:
        return PagedCacheSpec((CachePlane("c", 1, self.kv_rank), CachePlane("r", 1, self.rot_dim)))

    def setup(self, rt: Runtime, weights: Dict[str, torch.Tensor]) -> None:
        super().setup(rt, weights)
        t, H = self.tensors, self.num_heads
        dq, dkv = weights.pop(t["dq"]), weights.pop(t["dkv"])
        g = weights.pop(t["gate"]) if self.has_gate else dq[:0]
        self.sink = weights[t["sink"]] if self.has_sink else None
        dtype = torch.float32 if torch.float32 in (dq.dtype, dkv.dtype, g.dtype) else dq.dtype
        # one product reads the input: query latent, kv latent with the shared key part, gates (padded to whole
        # groups of eight rows so that the few-rows product takes it)
        rows = self.q_rank + self.kv_rank + self.rot_dim + g.shape[0]
        pad = torch.zeros((-rows) % 8, dq.shape[1], dtype=dtype, device=dq.device)
        self.down = Linear(torch.cat([dq.to(dtype), dkv.to(dtype), g.to(dtype), pad], dim=0), rt, tag="lattn.down")
        del dq, dkv, g
        self.kv_col, self.gate_col = self.q_rank, self.q_rank + self.kv_rank + self.rot_dim
        self.q_norm, self.kv_norm = weights[t["dq_norm"]], weights[t["dkv_norm"]]
        self.up_q = Linear(weights.pop(t["uq"]), rt, tag="lattn.uq")
        uk, uv = weights.pop(t["uk"]), weights.pop(t["uv"])
        # per head: W_uk^T [kv_rank, dim] takes the plain query into the latent's space, W_uv [vdim, kv_rank] brings
        # the attended latent out; both in the compute dtype (a float32 run: float32)
        self.uk_t = uk.view(H, self.dim, self.kv_rank).transpose(1, 2).to(rt.dtype).contiguous()
        self.uv = uv.view(H, self.vdim, self.kv_rank).to(rt.dtype).contiguous()
        del uk, uv
        self.o_proj = Linear(weights.pop(t["out"]), rt, tag="lattn.o_proj")
        self.position.setup(rt, weights)
        T = rt.max_tokens
        self._cq = rt.shared("lattn.cq", T, self.q_rank)
        self._gate = rt.shared("lattn.gate", T, H, dtype=torch.float32) if self.has_gate else None
        self._q_plain = rt.shared("lattn.q_plain", T, H * self.dim)
        self._q_rot = rt.shared("lattn.q_rot", T, H, self.rot_dim)
        self._q_abs = rt.shared("lattn.q_abs", H * T * self.kv_rank, dtype=torch.float32)
        self._o_lat = rt.shared("lattn.o_lat", T, H * self.kv_rank)
        self._o_heads = rt.shared("lattn.o_heads", H * T * self.vdim, dtype=torch.float32)
        self._o = rt.shared("lattn.o", T, H * self.vdim)
        self._partial = None
        if ops.latent_attention_fast(rt.dtype, self.kv_rank, self.rot_dim):
            self._partial = rt.shared("lattn.partial", ops.latent_partial_numel(rt.max_seqs, H, self.kv_rank),
                                      dtype=torch.float32)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache_id: Optional[int], write_cache: bool) -> torch.Tensor:
        T, H, rank, rot = x.shape[0], self.num_heads, self.kv_rank, self.rot_dim
        planes, table = ctx.pages(cache_id)
        c_pages, r_pages = planes["c"], planes["r"]
        freq, mag, dims = self.position.frequencies()
        status = self.rt.status
        cq, gate = self._cq[:T], (self._gate[:T] if self.has_gate else None)
        ops.latent_kv_post(self.down(x), self.q_rank, self.kv_col, rank, rot, dims, self.gate_col, H, self.q_norm,
                           self.kv_norm, self.norm_eps, freq, mag, ctx.positions, ctx.tok_seq, table, c_pages, r_pages, cq,
                           gate, write_cache, status, pairing=self.pairing)
        q_plain, q_rot = self._q_plain[:T], self._q_rot[:T]
        ops.latent_q_post(self.up_q(cq), H, self.dim, rot, dims, freq, mag, ctx.positions, q_plain, q_rot,
                          pairing=self.pairing)
        q_abs = self._q_abs[: H * T * rank].view(H, T, rank)
        ops.block_diag(q_plain, self.uk_t, q_abs)
        o_lat = self._o_lat[:T]
        ops.latent_attention(q_abs, q_rot, c_pages, r_pages, ctx, table, o_lat, self.scale, status, partial=self._partial,
                             sink=self.sink)
        o_heads = self._o_heads[: H * T * self.vdim].view(H, T, self.vdim)
        ops.block_diag(o_lat, self.uv, o_heads)
        out = self._o[:T]
        ops.gate_heads(o_heads, gate, out)
        return self.o_proj(out)


@register_part("mixer", "pooled_window_attention")
class PooledWindowAttention(Mixer):
    """Grouped-query softmax attention over a sliding window of tokens and, before the window, one pooled key and
    value per block of ``pool`` tokens.  With h the input, H heads on G key/value heads (head n reads key/value head
    n // (H / G)), keys of ``dim`` and values of ``vdim`` values:

        q = rmsnorm_all(W_q h) w_q;  k = rmsnorm_all(W_k h) w_k;  v = W_v h      (one mean over the whole projection)
        q, k rotated by ``position`` (a part with ``frequencies()``: the first ``dims`` values of every head)
        score = q . k * scale;  score <- softcap * tanh(score / softcap) if a cap is given
        position i reads the tokens j with 0 <= i - j < window and block b (tokens b pool .. b pool + pool - 1) once
        b pool + pool - 1 <= i - window; a block's key is the mean of its keys as the cache holds them, its value the
        mean of its values; tokens and blocks share one softmax
        out = W_o concat_heads(softmax(scores) values)

    Two caches per run: pages with one entry per token (planes ``k`` and ``v``; the manager keeps the pages that the
    last max(window, pool) tokens touch, so that a block's tokens are still there when its last one arrives) and pages
    with one entry per block (``pooled``: planes ``pk`` and ``pv``).  ``scale`` is used as given.  Norms, angles, scores
    and weights are float32 in every run.  ``names``: the tensors' names after the part's own."""

    graph_capturable = True
    splittable = True
    NAMES = {"q": "q", "k": "k", "v": "v", "q_norm": "q.norm", "k_norm": "k.norm", "out": "o"}

    def __init__(self, name: str, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float,
                 window: int, pool: int, norm_eps: float, position: PartSpec, softcap: Optional[float] = None,
                 names: Optional[Dict[str, str]] = None):
        super().__init__(name)
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        if self.num_heads % self.num_kv_heads:
            raise ValueError(f"{self.num_heads} query heads are not a multiple of {self.num_kv_heads} kv heads")
        self.dim, self.vdim = int(dim), int(vdim)
        self.scale, self.norm_eps = float(scale), float(norm_eps)
        self.softcap = None if softcap is None else float(softcap)
        self.window, self.pool = int(window), int(pool)
        if self.window < 1 or self.pool < 1:
            raise ValueError(f"attention {name}: window {self.window} and pool {self.pool} must be positive")
        self.position = create_part("position", position, name=f"{name}.position")
        n = dict(self.NAMES)
        n.update(names or {})
        self.tensors = {k: f"{name}.{v}" for k, v in n.items()}

    def weight_specs(self) -> List[WeightSpec]:
        t, w, H, G, D, Dv = self.tensors, self.hidden_size, self.num_heads, self.num_kv_heads, self.dim, self.vdim
        return [WeightSpec(t["q"], (H * D, w)), WeightSpec(t["k"], (G * D, w)), WeightSpec(t["v"], (G * Dv, w)),
                WeightSpec(t["q_norm"], (H * D,), kind="vector", init="one_plus_normal"),
                WeightSpec(t["k_norm"], (G * D,), kind="vector", init="one_plus_normal"),
                WeightSpec(t["out"], (w, H * Dv))] + self.position.weight_specs()

    def cache_spec(self):
        G = self.num_kv_heads
        return {"": PagedCacheSpec((CachePlane("k", G, self.dim), CachePlane("v", G, self.vdim)),
                                   window=max(self.window, self.pool)),
                "pooled": PagedCacheSpec((CachePlane("pk", G, self.dim), CachePlane("pv", G, self.vdim)),
                                         entry_tokens=self.pool)}

    # ------------------------------------------------------------------ the two products and what lies between
    def input_weight(self, weights: Dict[str, torch.Tensor]) -> torch.Tensor:
        t = self.tensors
        q, k, v = weights.pop(t["q"]), weights.pop(t["k"]), weights.pop(t["v"])
        dtype = torch.float32 if torch.float32 in (q.dtype, k.dtype, v.dtype) else q.dtype
        return torch.cat([q.to(dtype), k.to(dtype), v.to(dtype)], dim=0)  # columns of the product: q, k, v

    def output_weight(self, weights: Dict[str, torch.Tensor]) -> torch.Tensor:
        return weights.pop(self.tensors["out"])

    @property
    def input_rows(self) -> int:
        return (self.num_heads + self.num_kv_heads) * self.dim + self.num_kv_heads * self.vdim

    @property
    def output_columns(self) -> int:
        return self.num_heads * self.vdim

    def setup_core(self, rt: Runtime, weights: Dict[str, torch.Tensor]) -> None:
        self.rt = rt
        self.q_norm, self.k_norm = weights[self.tensors["q_norm"]], weights[self.tensors["k_norm"]]
        self.position.setup(rt, weights)
        self._q = rt.shared("pwattn.q", rt.max_tokens, self.num_heads, self.dim)
        self._partial = None
        if ops.pw_attention_fast(rt.dtype, self.dim, self.vdim):
            self._partial = ops.pw_attn_partial(rt.shared, rt.max_seqs, self.num_heads, self.vdim)

    def setup(self, rt: Runtime, weights: Dict[str, torch.Tensor]) -> None:
        super().setup(rt, weights)
        self.in_proj = Linear(self.input_weight(weights), rt, tag="pwattn.in")
        self.out_proj = Linear(self.output_weight(weights), rt, tag="pwattn.out")
        self.setup_core(rt, weights)
        self._o = rt.shared("pwattn.o", rt.max_tokens, self.output_columns)

    def core(self, proj: torch.Tensor, column: int, ctx: StepContext, cache_id: Optional[int], write_cache: bool,
             out: torch.Tensor, out_scale: float) -> None:
        T, H, G, D, Dv = proj.shape[0], self.num_heads, self.num_kv_heads, self.dim, self.vdim
        planes, table = ctx.pages(cache_id)
        pooled, ptable = ctx.pages(cache_id, "pooled")
        freq, mag, dims = self.position.frequencies()
        status = self.rt.status
        q = self._q[:T]
        ops.pw_qkv_post(proj, column, column + H * D, column + (H + G) * D, H, G, D, Dv, self.q_norm, self.k_norm,
                        self.norm_eps, dims, freq, mag, ctx.positions, ctx.tok_seq, table, q, planes["k"], planes["v"],
                        write_cache, status)
        if write_cache:
            ops.pool_blocks(planes["k"], planes["v"], pooled["pk"], pooled["pv"], ctx.q_start, ctx.kv_len, table, ptable,
                            ctx.num_seqs, ctx.max_q_len, self.pool, status)
        ops.pooled_window_attention(q, planes["k"], planes["v"], pooled["pk"], pooled["pv"], ctx, table, ptable, out,
                                    self.window, self.pool, self.scale, self.softcap, out_scale, status, self._partial)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache_id: Optional[int], write_cache: bool) -> torch.Tensor:
        o = self._o[: x.shape[0]]
        self.core(self.in_proj(x), 0, ctx, cache_id, write_cache, o, 1.0)
        return self.out_proj(o)


def distance_buckets(rows: int, most: float) -> List[int]:
    """The row of a distance bias's table for every distance 0, 1, ... up to the first one from which all further ones
    read the last row (see ``KeptWindowAttention``)."""
    half = rows // 2
    out = []
    while not out or out[-1] < rows - 1:
        n = len(out)
        if n < half:
            out.append(n)
        elif half == 0 or most <= half:
            out.append(rows - 1)
        else:
            out.append(min(rows - 1, half + math.floor(math.log(n / half) / math.log(most / half) * (rows - half))))
    return out


@register_part("mixer", "kept_window_attention")
class KeptWindowAttention(Mixer):
    """Grouped-query softmax attention over a sliding window that also keeps a request's first tokens, or (``window`` None)
    over every earlier token.  With h the input, H heads on G key/value heads (head n reads key/value head n // (H / G)),
    keys of ``dim`` and values of ``vdim`` values:

        q = W_q h;  k = W_k h;  v = W_v h;  q, k rotated by ``position`` (a part with ``frequencies()``: the first ``dims``
        values of every head, value i with value i + dims / 2; None: no rotation), the values not
        score = q . k * scale + rel[bucket(i - j), head];  position i reads j <= i with i - j < window or j < keep_first, the
        kept tokens at their true positions
        softmax over what is read, the denominator with one more term exp(sink_head)
        out = W_o (concat_heads(softmax(scores) values) * sigmoid(W_g h))          (``gate``; without it no W_g)

    ``bias`` = {"most": D, "rows": B}: the learned distance bias of T5 (Raffel et al., "Exploring the Limits of Transfer
    Learning with a Unified Text-to-Text Transformer"), a table ``<name>.rel`` [B, H] whose rows stand for distances:
    bucket(n) = n below B / 2, then min(B - 1, B / 2 + floor(ln(n / (B / 2)) / ln(D / (B / 2)) (B - B / 2))).  The table's
    stored size says what B is ("rows" only sizes random weights); at load it becomes one value per head and distance up
    to the distance from which the last row is read.  None: no bias.  It does not go with kept first tokens.
    ``sink``: the learned logits ``<name>.sink`` [H]; nothing is scored or weighted by them and ``scale`` is not applied.
    ``fixed_sink``: the same with one given logit for all heads and no tensor (0: a one in the denominator).

    ``proj_bias``: the four projections have biases (``<name>.q.b`` and so on), added in float32 before anything else; the
    output's is left open (``forward`` returns a ``PendingTerm``).  ``qk_norm_eps``: every head of q and of k goes through an
    RMS norm over ``dim`` before the rotation, with one weight for all heads (``<name>.q.norm``, ``<name>.k.norm`` [dim]).
    ``shares_kv``: the layer has no tensors for keys and values; its entry of the run order names the cache of a layer that
    has (of the same head counts, sizes and rotation) and does not write it.

    One paged cache (planes ``k`` and ``v``), of which the manager keeps the pages of the last ``window`` tokens and those
    of the first ``keep_first`` (all pages without a window).  The attention kernels are those of the window with pooled
    blocks, run with blocks of one token whose pages are the token pages themselves and with no more than ``keep_first`` of
    them; a window alone, with or without a sink, runs on the TMA-fed decode kernel and the tcgen05 portion kernel where those
    take the sizes.  ``scale`` is used
    as given.  Angles, scores, weights and the gate are float32 in every run.  ``names``: the tensors' names after the
    part's own."""

    graph_capturable = True
    NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "out": "o", "bias": "rel", "sink": "sink", "q_bias": "q.b",
             "k_bias": "k.b", "v_bias": "v.b", "out_bias": "o.b", "q_norm": "q.norm", "k_norm": "k.norm"}

    def __init__(self, name: str, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float,
                 window: Optional[int] = None, keep_first: int = 0, position: Optional[PartSpec] = None, gate: bool = True,
                 names: Optional[Dict[str, str]] = None, bias: Optional[dict] = None, sink: bool = False,
                 fixed_sink: Optional[float] = None, proj_bias: bool = False, qk_norm_eps: Optional[float] = None,
                 shares_kv: bool = False):
        super().__init__(name)
        self.fixed_sink = None if fixed_sink is None else float(fixed_sink)
        self.proj_bias, self.shares_kv = bool(proj_bias), bool(shares_kv)
        self.qk_norm_eps = None if qk_norm_eps is None else float(qk_norm_eps)
        if sink and self.fixed_sink is not None:
            raise ValueError(f"attention {name}: a learned sink or a fixed one")
        if self.proj_bias and gate:
            raise ValueError(f"attention {name}: output gates beside biases on the projections are not built")
        self.splittable = not self.proj_bias  # the output's bias stays open, which merged products have no place for
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        if self.num_heads % self.num_kv_heads:
            raise ValueError(f"{self.num_heads} query heads are not a multiple of {self.num_kv_heads} kv heads")
        self.dim, self.vdim, self.scale = int(dim), int(vdim), float(scale)
        self.window, self.keep_first, self.has_gate = None if window is None else int(window), int(keep_first), bool(gate)
        if (self.window is not None and self.window < 1) or self.keep_first < 0:
            raise ValueError(f"attention {name}: window {self.window} must be positive, keep_first {self.keep_first} not negative")
        self.bias, self.has_sink = dict(bias) if bias else None, bool(sink)
        if self.bias and self.keep_first and self.window is not None:
            raise ValueError(f"attention {name}: a distance bias and kept first tokens together are not built")
        self.position = None if position is None else create_part("position", position, name=f"{name}.position")
        n = dict(self.NAMES)
        n.update(names or {})
        self.tensors = {k: f"{name}.{v}" for k, v in n.items()}

    def weight_specs(self) -> List[WeightSpec]:
        t, w, H, G, D, Dv = self.tensors, self.hidden_size, self.num_heads, self.num_kv_heads, self.dim, self.vdim
        own = [("q", H * D)] + ([] if self.shares_kv else [("k", G * D), ("v", G * Dv)])
        vectors = [(f"{k}_bias", n, "normal") for k, n in own + [("out", w)]] if self.proj_bias else []
        if self.qk_norm_eps is not None:
            vectors += [(f"{k}_norm", D, "one_plus_normal") for k, _ in own if k != "v"]
        return [WeightSpec(t[k], (n, w)) for k, n in own] + [
            WeightSpec(t[k], (n,), kind="vector", init=init) for k, n, init in vectors] + (
            [WeightSpec(t["gate"], (H * Dv, w))] if self.has_gate else []) + (
            [WeightSpec(t["bias"], (int(self.bias["rows"]), H), kind="vector", init="normal", free_dims=(0,))] if self.bias else []) + (
            [WeightSpec(t["sink"], (H,), kind="vector", init="normal")] if self.has_sink else []) + [
            WeightSpec(t["out"], (w, H * Dv))] + (self.position.weight_specs() if self.position is not None else [])

    def cache_spec(self):
        G = self.num_kv_heads
        return PagedCacheSpec((CachePlane("k", G, self.dim), CachePlane("v", G, self.vdim)), window=self.window,
                              keep_first=self.keep_first if self.window is not None else 0)

    # ------------------------------------------------------------------ the two products and what lies between
    def input_weight(self, weights: Dict[str, torch.Tensor]) -> torch.Tensor:
        t = self.tensors
        keys = ["q"] + ([] if self.shares_kv else ["k", "v"]) + (["gate"] if self.has_gate else [])
        parts = [weights.pop(t[k]) for k in keys]
        dtype = torch.float32 if any(p.dtype == torch.float32 for p in parts) else parts[0].dtype
        return torch.cat([p.to(dtype) for p in parts], dim=0)  # columns of the product: q, k, v, gates

    def output_weight(self, weights: Dict[str, torch.Tensor]) -> torch.Tensor:
        return weights.pop(self.tensors["out"])

    @property
    def output_columns(self) -> int:
        return self.num_heads * self.vdim

    def setup_core(self, rt: Runtime, weights: Dict[str, torch.Tensor]) -> None:
        self.rt = rt
        self.freq, self.magnitude, self.dims = torch.empty(0, dtype=torch.float32, device=rt.device), 1.0, 0
        if self.position is not None:
            self.position.setup(rt, weights)
            self.freq, self.magnitude, self.dims = self.position.frequencies()
        t = self.tensors
        self.dist_bias, self.sink = None, weights[t["sink"]] if self.has_sink else None
        if self.fixed_sink is not None:
            self.sink = torch.full((self.num_heads,), self.fixed_sink, dtype=torch.float32, device=rt.device)
        self.in_bias = self.out_bias = None
        if self.proj_bias:
            self.in_bias = torch.cat([weights[t[f"{k}_bias"]] for k in (("q",) if self.shares_kv else ("q", "k", "v"))]).contiguous()
            self.out_bias = weights[t["out_bias"]]
        normed = self.qk_norm_eps is not None
        self.q_norm = weights[t["q_norm"]] if normed else None
        self.k_norm = weights[t["k_norm"]] if normed and not self.shares_kv else None
        if self.bias:
            table = weights[self.tensors["bias"]]  # [rows, heads]
            index = torch.tensor(distance_buckets(table.shape[0], float(self.bias["most"])), device=rt.device)
            self.dist_bias = table[index].t().contiguous()
        elif self.sink is not None:  # the kernels take a sink beside a bias: one of zeros
            self.dist_bias = torch.zeros(self.num_heads, 1, dtype=torch.float32, device=rt.device)
        self._q = rt.shared("kwattn.q", rt.max_tokens, self.num_heads, self.dim)
        self._window_partial = None  # scratch of the kernels for a window alone
        if (not self.bias and (self.keep_first == 0 or self.window is None)
                and ops.window_attention_sizes(rt.dtype, self.num_heads, self.num_kv_heads, self.dim, self.vdim, self.scale)):
            self._window_partial = rt.shared("attn.partial", ops.decode_partial_numel(rt.max_seqs, self.num_heads, self.dim),
                                             dtype=torch.float32)
        self._partial = None
        if ops.pw_attention_fast(rt.dtype, self.dim, self.vdim):
            self._partial = ops.pw_attn_partial(rt.shared, rt.max_seqs, self.num_heads, self.vdim)

    def setup(self, rt: Runtime, weights: Dict[str, torch.Tensor]) -> None:
        super().setup(rt, weights)
        self.in_proj = Linear(self.input_weight(weights), rt, tag="kwattn.in")
        self.out_proj = Linear(self.output_weight(weights), rt, tag="kwattn.out")
        self.setup_core(rt, weights)
        self._o = rt.shared("kwattn.o", rt.max_tokens, self.output_columns)

    def core(self, proj: torch.Tensor, column: int, ctx: StepContext, cache_id: Optional[int], write_cache: bool,
             out: torch.Tensor, out_scale: float) -> None:
        T, H, G, D, Dv = proj.shape[0], self.num_heads, self.num_kv_heads, self.dim, self.vdim
        planes, table = ctx.pages(cache_id)
        k_pages, v_pages = planes["k"], planes["v"]
        status = self.rt.status
        q = self._q[:T]
        k_col, v_col = column + H * D, column + (H + G) * D
        if self.shares_kv and write_cache:
            raise ValueError(f"attention {self.name}: it has no keys and values of its own to write")
        if self.proj_bias or self.qk_norm_eps is not None or self.shares_kv:
            own = write_cache and not self.shares_kv
            ops.head_qkv_post(proj, column, k_col if own else None, v_col if own else None, H, G, D, Dv, self.in_bias, self.q_norm,
                              self.k_norm, self.qk_norm_eps or 0.0, self.dims, self.freq, self.magnitude, ctx.positions,
                              ctx.tok_seq, table, q, k_pages, v_pages, status)
        else:
            ops.pw_qkv_post(proj, column, k_col, v_col, H, G, D, Dv, None, None, 0.0, self.dims, self.freq, self.magnitude,
                            ctx.positions, ctx.tok_seq, table, q, k_pages, v_pages, write_cache, status)
        window, first = (ops.NO_WINDOW, 0) if self.window is None else (self.window, self.keep_first)
        if (self._window_partial is not None and out_scale == 1.0
                and ops.window_attention_takes(q, k_pages, v_pages, out, ctx, self.scale)):
            ops.window_attention(q, k_pages, v_pages, out, ctx, table, window, self.scale, self.sink, status, self._window_partial)
            if self.has_gate:
                ops.sigmoid_gate(out, proj, v_col + G * Dv)
            return
        # the kept first tokens are "blocks" of one token read from the token pages, at most keep_first of them
        ops.pooled_window_attention(q, k_pages, v_pages, k_pages, v_pages, ctx, table, table, out, window, 1,
                                    self.scale, None, out_scale, status, self._partial, block_limit=first,
                                    dist_bias=self.dist_bias, sink=self.sink)
        if self.has_gate:
            ops.sigmoid_gate(out, proj, v_col + G * Dv)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache_id: Optional[int], write_cache: bool):
        o = self._o[: x.shape[0]]
        self.core(self.in_proj(x), 0, ctx, cache_id, write_cache, o, 1.0)
        y = self.out_proj(o)
        return y if self.out_bias is None else PendingTerm(y, bias=self.out_bias)
