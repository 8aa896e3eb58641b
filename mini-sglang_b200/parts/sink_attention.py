from __future__ import annotations

import math
from typing import Dict

import torch

from .. import ops
from ..cache.manager import PagedKVNeed
from ..config.spec import PartSpec
from ..weights.loader import TensorDecl
from .attention import paged_attend
from .base import Mixer, register_mixer
from .context import KVCacheView, StepContext


@register_mixer("sink_attention")
class SinkAttention(Mixer):
    """Causal grouped-query softmax attention over the paged cache, with one more term in every softmax's denominator or without.

    q = Wq x (+ bq) [heads, key_dim], k = Wk x (+ bk) [kv heads, key_dim], v = Wv x (+ bv) [kv heads, value_dim]; the layer's
    position encoding turns the first elements of every q and k head (a partial rotation in halves or in neighbouring pairs, as
    the encoding says; v is not turned);
    score(i, j) = q_i . k_j * scale, then cap * tanh(score / cap) where the part has a `softcap`; the query at i sees the keys
    j <= i with i - j < window, or those of its own chunk of the sequence (j // chunk == i // chunk), or all; weights = exp(score) / (sum_seen exp(score) + exp(sink_h))
    with a learned number per head that has no key and no value, is neither scaled nor capped and counts once (`sink` gives
    all heads one fixed number instead; "none" leaves the term out); optionally the heads side by side times sigmoid(Wg x), element by element (`gate`);
    output projection.

    Optionally (`qk_norm`) every q and k head is RMS-normed by itself before the rotation, with one weight of key_dim for all
    q heads and one for all k heads, and (`value_norm`) every value head is divided by its root mean square, without a weight,
    and cached so.  Optionally (`qk_unit`) every q and k head is divided by its root mean square after the rotation, without a
    weight.

    With `own_kv` false the part has no k and v projections: it reads the keys and values that an earlier run of the schedule
    wrote into the same cache (its `Run` has `writes_cache` false), with its own queries.

    Blended values (`value_mix`): the first layer of a model that has it ("first") hands its values of the step's tokens on
    under `value_mix_key`; a later layer ("blend") caches and reads v <- (1 - lambda) v + lambda v_first with a learned number
    lambda.  Both must have the same kv heads and value size.

    Scores, soft cap, softmax and its weights, the sink and the rotation's angles are float32 in both precisions; in
    bfloat16 the rotated q and k, the (blended) v as cached and the weights as operands of the value product are rounded.

    params: hidden_size, num_heads, num_kv_heads, key_dim, value_dim, scale, window (None: all keys), softcap (None: none),
            bias, value_mix (None, "first", "blend"), value_mix_key, sink (None: learned), qk_norm, value_norm, norm_eps,
            gate (None, "sigmoid"), chunk (None: no chunks), qk_unit, own_kv, names (q, k, v, q_bias, k_bias, v_bias, sink, mix, q_norm, k_norm, gate, out).
    """

    graph_safe = True
    difference = None     # (lambda, eps, scale) of heads that are the difference of two maps
    maps = 1              # vectors of key_dim elements that a q or kv head has side by side, each with a softmax of its own

    def __init__(self, spec, prefix, env, position=None):
        super().__init__(spec, prefix, env)
        s = spec
        self.E, self.n_q, self.n_kv = int(s["hidden_size"]), int(s["num_heads"]), int(s["num_kv_heads"])
        self.d, self.dv = int(s["key_dim"]), int(s["value_dim"])
        if self.n_q % self.n_kv:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        self.D = self.maps * self.d                  # a key row of the cache
        if max(self.D, self.dv) > ops.SINK_ATTENTION_MAX_HEAD_DIM:
            raise ValueError(f"head sizes {self.D}, {self.dv}: the attention kernel takes up to {ops.SINK_ATTENTION_MAX_HEAD_DIM}")
        self.scale = float(s["scale"])
        self.window = int(s["window"]) if s.get("window") else None
        self.chunk = int(s["chunk"]) if s.get("chunk") else None
        if self.window and self.chunk:
            raise ValueError("an attention has a window or chunks, not both")
        self.softcap = float(s["softcap"]) if s.get("softcap") else 0.0
        self.bias = bool(s.get("bias", False))
        self.value_mix, self.value_mix_key = s.get("value_mix"), s.get("value_mix_key", "first_values")
        if self.value_mix not in (None, "first", "blend"):
            raise ValueError(f"value_mix {self.value_mix!r}: None, 'first' or 'blend'")
        self.has_sink = s.get("sink") != "none"
        self.fixed_sink = float(s["sink"]) if self.has_sink and s.get("sink") is not None else None
        self.qk_unit, self.own_kv = bool(s.get("qk_unit", False)), bool(s.get("own_kv", True))
        self.qk_norm, self.value_norm, self.eps = bool(s.get("qk_norm", False)), bool(s.get("value_norm", False)), float(s.get("norm_eps", 0.0))
        self.gate = s.get("gate")
        if self.gate not in (None, "sigmoid"):
            raise ValueError(f"unknown output gate {self.gate!r}; known: sigmoid")
        self.position = position
        if position is not None and not hasattr(position, "step_angles"):
            raise ValueError("this mixer takes a position encoding that makes the angles of a step's positions (step_angles)")
        names = {"q": "q", "k": "k", "v": "v", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "sink": "sink", "mix": "vmix",
                 "q_norm": "q.norm", "k_norm": "k.norm", "gate": "g", "out": "o"}
        names.update(s.get("names") or {})
        self.names = {k: self.name(v) for k, v in names.items()}
        self.Cq, self.Ck, self.Cv = self.n_q * self.D, self.n_kv * self.D, self.n_kv * self.dv
        if not self.own_kv:
            if self.value_mix is not None:
                raise ValueError("an attention without values of its own blends none")
            self.Ck = self.Cv = 0
        # equal head sizes that the engine's paged attention kernels take in bfloat16, and no cap on the scores: those kernels
        # (tcgen05 for prompts at head size 128, kv splits in decode steps); else the ones that take any pair of head sizes
        self.paged = self.D == self.dv and not self.softcap and ops.mma_supported(self.D, env.dtype)
        self.w_in = self.b_in = self.w_out = self.sink = self.sink_log2 = self.q_norm = self.k_norm = None
        self.lam = 0.0

    def tensors(self) -> Dict[str, TensorDecl]:
        n = self.names
        t = {n["q"]: TensorDecl((self.Cq, self.E)), n["out"]: TensorDecl((self.E, self.n_q * self.dv))}
        if self.own_kv:
            t[n["k"]], t[n["v"]] = TensorDecl((self.Ck, self.E)), TensorDecl((self.Cv, self.E))
        if self.has_sink and self.fixed_sink is None:
            t[n["sink"]] = TensorDecl((self.n_q,), kind="vector", std=1.0)
        if self.qk_norm:
            t[n["q_norm"]] = TensorDecl((self.d,), kind="vector", init="norm")
            t[n["k_norm"]] = TensorDecl((self.d,), kind="vector", init="norm")
        if self.gate:
            t[n["gate"]] = TensorDecl((self.n_q * self.dv, self.E))
        if self.bias:
            t[n["q_bias"]] = TensorDecl((self.Cq,), kind="vector", std=0.1)
            if self.own_kv:
                t[n["k_bias"]] = TensorDecl((self.Ck,), kind="vector", std=0.1)
                t[n["v_bias"]] = TensorDecl((self.Cv,), kind="vector", std=0.1)
        if self.value_mix is not None:
            t[n["mix"]] = TensorDecl((), kind="vector", std=0.3, optional=self.value_mix == "first")
        return t

    def load(self, src) -> None:
        f, n = src.fetch, self.names
        which = ["q", "k", "v"] if self.own_kv else ["q"]
        rows = [f(n[k]) for k in which] + ([f(n["gate"])] if self.gate else [])        # one product: [q | k | v | gate]
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_out = f(n["out"]).contiguous()
        if self.bias:
            b = [f(n[k + "_bias"]) for k in which]
            if self.gate:
                b.append(torch.zeros_like(b[0][:1]).expand(self.n_q * self.dv))
            self.b_in = torch.cat(b, dim=0).to(self.env.dtype).contiguous()
        if not self.has_sink:
            pass
        elif self.fixed_sink is None:
            self.sink = f(n["sink"]).float().contiguous()
        else:
            self.sink = torch.full((self.n_q,), self.fixed_sink, dtype=torch.float32, device=self.w_in.device)
        if self.has_sink:
            self.sink_log2 = (self.sink * math.log2(math.e)).contiguous()
        if self.qk_norm:
            self.q_norm, self.k_norm = f(n["q_norm"]).float().contiguous(), f(n["k_norm"]).float().contiguous()
        if self.value_mix == "blend":
            self.lam = float(f(n["mix"]).float().item())

    def cache_need(self) -> PagedKVNeed:
        if self.paged:
            return PagedKVNeed(self.n_kv, self.D, self.window, q_heads=self.n_q * self.maps, chunk=self.chunk)
        return PagedKVNeed(self.n_kv, self.D, self.window, q_heads=self.n_q * self.maps, library="mixers_delta", even_cut=False,
                           v_head_dim=self.dv, chunk=self.chunk)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: KVCacheView, writes_cache: bool = True) -> torch.Tensor:
        Cq, Ck, Cv = self.Cq, self.Ck, self.Cv
        proj = ops.linear(x, self.w_in, self.b_in)
        v_own = proj[:, Cq + Ck:Cq + Ck + Cv]
        if not self.own_kv:
            assert not writes_cache, "an attention without keys of its own runs on a cache that another run wrote"
        v_first = None
        if self.value_mix == "first":
            ctx.shared[self.value_mix_key] = v_own
        elif self.value_mix == "blend":
            v_first = ctx.shared.get(self.value_mix_key)
            if v_first is None or v_first.shape != v_own.shape:
                raise ValueError("blended values: no earlier layer of the step handed on values of this layer's shape")
        angles = self.position.step_angles(ctx) if self.position is not None else None
        q = ops.sink_qkv_prep(proj, n_q=self.n_q, n_kv=self.n_kv, d=self.d, dv=self.dv, angles=angles, v_first=v_first, lam=self.lam,
                              out_loc=cache.group.out_loc if writes_cache else None, k_cache=cache.k if writes_cache else None,
                              v_cache=cache.v if writes_cache else None, page_size=cache.page_size, q_norm=self.q_norm,
                              k_norm=self.k_norm, v_unit=self.value_norm, eps=self.eps, qk_unit=self.qk_unit, maps=self.maps,
                              interleaved=bool(getattr(self.position, "interleaved", False)))
        gate = proj[:, Cq + Ck + Cv:Cq + Ck + Cv + self.n_q * self.dv] if self.gate else None
        return ops.linear(self.attend(q, ctx, cache, gate), self.w_out)

    def attend(self, q: torch.Tensor, ctx: StepContext, cache: KVCacheView, gate) -> torch.Tensor:
        """The attention launches of the step: q [T, heads, key row] -> what the output projection reads, [T, heads * value_dim]."""
        n_q = self.n_q * self.maps
        if self.paged:
            o = torch.empty((ctx.T, self.n_q, self.dv), dtype=q.dtype, device=q.device)
            paged_attend(q, o, ctx, cache, n_q=n_q, n_kv=self.n_kv, d=self.D, window=int(self.window or 0), scale=self.scale,
                         use_mma=True, null_log2=self.sink_log2, gate=gate, chunk=int(self.chunk or 0), diff=self.difference)
            return o.view(ctx.T, self.n_q * self.dv)
        out = torch.empty((ctx.T, n_q * self.dv), dtype=q.dtype, device=q.device)
        ops.sink_attention(q, out, cache.k, cache.v, q_start=ctx.q_start, kv_len=ctx.kv_len, block_table=cache.group.block_table,
                           n_kv=self.n_kv, page_size=cache.page_size, scale=self.scale, softcap=self.softcap, window=self.window or 0,
                           sink=self.sink, q_lens=None if ctx.uniform_decode else ctx.host_q_lens, workspace=ctx.workspace, gate=gate,
                           chunk=self.chunk or 0)
        return out if self.maps == 1 else self.join_maps(out)


@register_mixer("differential_attention")
class DifferentialAttention(SinkAttention):
    """Attention whose heads are the difference of two softmax maps over the same values.

    Every q and kv head has two vectors of key_dim elements side by side (q has heads * 2 * key_dim rows, k kv heads * 2 *
    key_dim, v kv heads * value_dim), each turned by the position encoding by itself.  Map m of a head is a causal softmax
    attention of the m-th vectors over the kv head's values, a_m; with lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff, one number
    of the layer,

        o = a_1 - lambda a_2;   o <- o / sqrt(mean(o^2) + eps) * (1 - diff)      per head over its value_dim elements

    then the output projection.  A kv head's cache row holds both key vectors; a query row holds one query vector in its place
    and zeros in the other, so that the attention kernels see 2 * heads query heads on rows of 2 * key_dim elements.

    lambda is made at load in double precision, the difference and its norm are float32.  The paged kernels take the difference
    where a row is normalised (`ops.attention(diff=...)`); behind the kernels for any pair of head sizes it is a kernel of its own.
    params: as `sink_attention` (without sink, gate and value_mix) and diff; names of the four vectors: lq1, lk1, lq2, lk2."""

    maps = 2

    def __init__(self, spec, prefix, env, position=None):
        super().__init__(PartSpec(spec.kind, {**spec.params, "sink": "none"}), prefix, env, position=position)
        if self.gate or self.value_mix is not None:
            raise ValueError("a differential attention takes no gate and no blended values")
        self.diff = float(spec["diff"])
        self.difference = (0.0, self.eps, 1.0 - self.diff)
        self.vec_names = [self.name((spec.get("names") or {}).get(k, k)) for k in ("lq1", "lk1", "lq2", "lk2")]

    def tensors(self) -> Dict[str, TensorDecl]:
        return {**super().tensors(), **{n: TensorDecl((self.d,), kind="vector", std=0.1) for n in self.vec_names}}

    def load(self, src) -> None:
        super().load(src)
        lq1, lk1, lq2, lk2 = (src.fetch(n).double() for n in self.vec_names)
        lam = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum())) + self.diff
        self.difference = (lam, self.eps, 1.0 - self.diff)

    def join_maps(self, heads: torch.Tensor) -> torch.Tensor:
        T = heads.shape[0]
        out = torch.empty((T, self.n_q * self.dv), dtype=self.env.dtype, device=heads.device)
        ops.map_difference(heads.view(T, 2 * self.n_q, self.dv), out, heads=self.n_q, lam=self.difference[0], eps=self.eps,
                           scale=self.difference[2])
        return out
