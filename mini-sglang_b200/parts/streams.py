from __future__ import annotations

import dataclasses
from typing import Dict

import torch

from .. import ops
from ..weights.loader import TensorDecl
from .base import FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, Block, BuildEnv, build_part, register_block


@dataclasses.dataclass
class StreamUpdate:
    """What a sublayer leaves to be done with the copies of the stream: copy t becomes sum_s mix[s][t] x_s + w_out[t] y.  It is
    done together with the norm that reads the copies next."""

    y: torch.Tensor            # [T, H], what the sublayer hands over
    mix: torch.Tensor          # float32 [S, S], from copy s to copy t
    w_out: torch.Tensor        # float32 [S]


@register_block("hyper_connections")
class HyperConnectionsBlock(Block):
    """S copies x_1 .. x_S of the residual stream, all equal to the embedding at the start.  For each of the two sublayers
    (mixer, feed-forward), with learned numbers in [S], mix [S, S], out [S] of its own:

        y = sublayer(norm(sum_s in[s] x_s));   x_t <- sum_s mix[s][t] x_s + out[t] y   (all copies at once, from the old ones)

    The copies are float32 [T, S, H]; one kernel (`ops.stream_mix_norm`) updates them with one sublayer's output, reads them for
    the next sublayer and norms what it read.  Before the first update they are one row per token [T, H]; the update makes them.
    The block returns its last sublayer's update undone (`StreamUpdate`), for the next block or the model's final norm
    (`stream_sum`) to fuse.  A layer may have no feed-forward.  Roles of the norms: "input", "post_mixer" (`rmsnorm` or
    `layernorm`).  block_params: streams, mixer_names, ffn_names (full tensor names of in, mix, out for each sublayer)."""

    def __init__(self, layer_spec, env: BuildEnv):
        super().__init__(None, layer_spec.prefix, env)
        at = layer_spec.part_prefix
        bp = layer_spec.block_params
        self.S = int(bp["streams"])
        if not 1 <= self.S <= ops.MAX_STREAMS:
            raise ValueError(f"{self.S} copies of the stream: the kernel takes 1 to {ops.MAX_STREAMS}")
        self.position = None
        if layer_spec.position is not None:
            self.position = env.shared(layer_spec.position, lambda: build_part(
                POSITION_ENCODINGS, "position encoding", layer_spec.position, layer_spec.prefix, env))
        self.norm_in = build_part(NORMS, "norm", layer_spec.norms["input"], at("input"), env)
        self.mixer = build_part(MIXERS, "mixer", layer_spec.mixer, at("mixer"), env, position=self.position)
        self.norm_post = self.ffn = None
        if layer_spec.feed_forward is not None:
            self.norm_post = build_part(NORMS, "norm", layer_spec.norms["post_mixer"], at("post_mixer"), env)
            self.ffn = build_part(FEED_FORWARDS, "feed-forward", layer_spec.feed_forward, at("feed_forward"), env)
        for n in (self.norm_in, self.norm_post):
            if n is not None and not hasattr(n, "center"):
                raise ValueError("this block fuses an RMS norm or a layer norm behind the copies' update; another kind is not taken here")
        self.names = [dict(bp["mixer_names"])] + ([dict(bp["ffn_names"])] if self.ffn is not None else [])
        self.coef = []          # per sublayer {"in", "mix", "out"}
        self.w_norm = []        # per sublayer: the norm's weight in float32 (exact: the checkpoint's values widened)

    def parts(self):
        return [p for p in (self.position, self.norm_in, self.mixer, self.norm_post, self.ffn) if p is not None]

    def tensors(self) -> Dict[str, TensorDecl]:
        out: Dict[str, TensorDecl] = {}
        for part in self.parts():
            out.update(part.tensors())
        S = self.S
        for n in self.names:
            out[n["in"]] = TensorDecl((S,), kind="vector", std=0.5)
            out[n["out"]] = TensorDecl((S,), kind="vector", init="norm")
            out[n["mix"]] = TensorDecl((S, S), kind="vector", std=0.5 / S ** 0.5)
        return out

    def load(self, src) -> None:
        for part in self.parts():
            part.load(src)
        self.coef = [{k: src.fetch(n[k]).float().contiguous() for k in ("in", "mix", "out")} for n in self.names]
        self.w_norm = [n.weight.float().contiguous() for n in (self.norm_in, self.norm_post) if n is not None]

    def _read(self, q: int, norm, residual, update):
        """The update that is still to be done, then what sublayer q reads of the copies, normed -> (normed [T, H], copies)."""
        x_out = None
        if update is not None:
            x_out = residual if residual.dim() == 3 else torch.empty((residual.shape[0], self.S, residual.shape[1]), dtype=torch.float32,
                                                                     device=residual.device)
        y = ops.stream_mix_norm(residual, streams=self.S, weight=self.w_norm[q], bias=norm.bias, eps=norm.eps, center=norm.center,
                                w_in=self.coef[q]["in"], y=update.y if update is not None else None,
                                mix=update.mix if update is not None else None, w_out=update.w_out if update is not None else None,
                                x_out=x_out, out_dtype=self.env.dtype)
        return y, (x_out if x_out is not None else residual)

    def _update(self, q: int, y) -> StreamUpdate:
        return StreamUpdate(y, self.coef[q]["mix"], self.coef[q]["out"])

    def forward(self, delta, residual, ctx, cache, writes_cache: bool = True):
        # residual: float32, the copies [T, S, H] (updated in place) or the embedding [T, H]; delta: the update still to be done
        y, residual = self._read(0, self.norm_in, residual, delta)
        up = self._update(0, self.mixer.forward(y, ctx, cache, writes_cache))
        if self.ffn is None:
            return up, residual
        y, residual = self._read(1, self.norm_post, residual, up)
        return self._update(1, self.ffn.forward(y, ctx)), residual
