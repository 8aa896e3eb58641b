"""Rubulix: typed configuration and model description.

A decoder whose layers are listed one by one in config.json (`layers`): every entry names the kind of its mixer (`type`), the
mixer's sizes and constants (`mixer`) and its feed-forward (`mlp`, or null for none).  The residual stream is kept in `streams`
copies that every sublayer reads as a weighted sum and rewrites by a learned mix (hyper-connections); the sublayers sit behind
layer norms with weight and bias.  Mixers:

  attention     grouped-query attention whose heads are the difference of two softmax maps over the same values, all earlier
                keys, rotation in neighbouring pairs (YaRN's frequency scaling where given); a layer with `kv_from` reads the keys
                and values of an earlier layer and has only queries of its own
  attention_2   grouped-query softmax attention within chunks of the sequence, rotation in neighbouring pairs, q and k of unit
                root mean square after it, the heads side by side times a sigmoid gate per element

Both have biases on q, k and v, and key and value sizes of their own.  The feed-forward (`dense`) is down(silu(gate x) * up x).
The head is a matrix of its own.  Everything that differs between models of the design is read here; nothing else in the engine
knows the design's name.
"""

from __future__ import annotations

import dataclasses
from typing import Any, Dict, List, Optional

from .registry import ConfigError, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, Run

NO_POSITION_LIMIT = 1 << 20      # the design has no table of places; the context is bounded by the cache alone


def _need(d: Dict[str, Any], key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: {where} has no {key!r}")
    return d[key]


@dataclasses.dataclass
class RubulixLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]
    kv_from: Optional[int] = None


@dataclasses.dataclass
class RubulixConfig:
    width: int
    vocab: int
    streams: int
    norm_eps: float
    layers: List[RubulixLayer]
    max_positions: int = NO_POSITION_LIMIT
    eos_token_ids: List[int] = dataclasses.field(default_factory=list)
    raw: Dict[str, Any] = dataclasses.field(default_factory=dict, repr=False)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "RubulixConfig":
        layers = []
        for i, entry in enumerate(_need(raw, "layers", "the model")):
            where = f"layer {i}"
            mixer = dict(_need(entry, "mixer", where))
            layers.append(RubulixLayer(type=str(_need(entry, "type", where)), mixer=mixer,
                                       mlp=dict(entry["mlp"]) if entry.get("mlp") is not None else None,
                                       kv_from=int(mixer["kv_from"]) if mixer.get("kv_from") is not None else None))
        eos = raw.get("eos_token_id", [])
        eos = [] if eos is None else ([int(e) for e in eos] if isinstance(eos, (list, tuple)) else [int(eos)])
        cfg = cls(width=int(_need(raw, "width", "the model")), vocab=int(_need(raw, "vocab", "the model")),
                  streams=int(_need(raw, "streams", "the model")),
                  norm_eps=float(_need(_need(raw, "norm", "the model"), "eps", "norm")), layers=layers,
                  max_positions=int(raw.get("max_positions") or NO_POSITION_LIMIT), eos_token_ids=eos, raw=dict(raw))
        cfg.check()
        return cfg

    def check(self) -> None:
        if self.width <= 0 or self.vocab <= 0 or self.streams <= 0 or not self.layers:
            raise ConfigError("width, vocab, streams and the number of layers must be positive")
        for i, l in enumerate(self.layers):
            if l.type not in _MIXERS:
                raise ConfigError(f"config.json: layer {i} has type {l.type!r}; known: " + ", ".join(sorted(_MIXERS)))
            if l.mlp is not None and l.mlp.get("kind") not in _FEED_FORWARDS:
                raise ConfigError(f"config.json: layer {i} has a feed-forward of kind {l.mlp.get('kind')!r}; known: "
                                  + ", ".join(sorted(_FEED_FORWARDS)))
            if l.kv_from is None:
                continue
            j = l.kv_from
            if not 0 <= j < i or self.layers[j].type != l.type or self.layers[j].kv_from is not None:
                raise ConfigError(f"config.json: layer {i} takes the keys and values of layer {j}, which is no earlier layer of the "
                                  "same kind with keys of its own")
            for key in ("heads", "kv_heads", "dim", "vdim"):
                if l.mixer.get(key) != self.layers[j].mixer.get(key):
                    raise ConfigError(f"config.json: layers {i} and {j} share keys and values but differ in {key!r}")

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)


def _rotation(m: Dict[str, Any], where: str) -> Optional[PartSpec]:
    rot = m.get("rot")
    dims = int(_need(rot, "dims", where + ".rot")) if rot is not None else 0
    if dims == 0:
        return None
    if dims < 0 or dims > int(m["dim"]) or dims % 2:
        raise ConfigError(f"config.json: {where}.rot: {dims} rotated dimensions must be even and at most dim = {m['dim']}")
    sc = rot.get("scaling")
    scaling = {k: float(_need(sc, k, where + ".rot.scaling")) for k in ("factor", "original", "fast", "slow")} if sc else None
    return PartSpec("rope_yarn", {"rotary_dim": dims, "theta": float(_need(rot, "base", where + ".rot")), "scaling": scaling,
                                  "interleaved": True})


def _attention_params(cfg: RubulixConfig, m: Dict[str, Any], where: str) -> Dict[str, Any]:
    heads, dim = int(_need(m, "heads", where)), int(_need(m, "dim", where))
    return {"hidden_size": cfg.width, "num_heads": heads, "num_kv_heads": int(m.get("kv_heads") or heads), "key_dim": dim,
            "value_dim": int(m.get("vdim") or dim), "scale": float(_need(m, "scale", where)), "bias": True, "sink": "none",
            "norm_eps": cfg.norm_eps}


def _differential(cfg: RubulixConfig, m: Dict[str, Any], where: str) -> PartSpec:
    return PartSpec("differential_attention", {**_attention_params(cfg, m, where), "diff": float(_need(m, "diff", where)),
                                               "own_kv": m.get("kv_from") is None})


def _chunked(cfg: RubulixConfig, m: Dict[str, Any], where: str) -> PartSpec:
    size = int(_need(_need(m, "mask", where), "size", where + ".mask"))
    if size < 1:
        raise ConfigError(f"config.json: {where}.mask: a chunk of {size} tokens")
    return PartSpec("sink_attention", {**_attention_params(cfg, m, where), "chunk": size, "qk_unit": True, "gate": "sigmoid",
                                       "own_kv": m.get("kv_from") is None})


def _dense(cfg: RubulixConfig, f: Dict[str, Any], where: str) -> PartSpec:
    return PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": int(_need(f, "ff", where)), "activation": "silu",
                                  "names": {"gate": "gate", "up": "up", "down": "down"}})


_MIXERS = {"attention": _differential, "attention_2": _chunked}
_FEED_FORWARDS = {"dense": _dense}
RUBULIX_LAYER_NAMES = {"mixer": "mix", "feed_forward": "mlp"}


def build_rubulix_spec(cfg: RubulixConfig) -> ModelSpec:
    """embedding -> layers of (read the copies, norm, mixer, rewrite them; read, norm, feed-forward, rewrite) -> the copies' sum,
    normed -> head.  One `LayerSpec` and one `Run` per listed layer; a layer that reads another's keys runs on that one's
    cache."""
    def norm(name: str) -> PartSpec:
        return PartSpec("layernorm", {"size": cfg.width, "eps": cfg.norm_eps, "name": name, "bias": True})

    def stream_names(i: int, q: int) -> Dict[str, str]:
        return {k: f"l{i}.hc{q}.{k}" for k in ("in", "mix", "out")}

    layers, schedule = [], []
    for i, l in enumerate(cfg.layers):
        where = f"layer {i}.mixer"
        norms = {"input": norm(f"l{i}.norm1")}
        ffn = None
        if l.mlp is not None:
            ffn = _FEED_FORWARDS[l.mlp["kind"]](cfg, l.mlp, f"layer {i}.mlp")
            norms["post_mixer"] = norm(f"l{i}.norm2")
        mixer = _MIXERS[l.type](cfg, l.mixer, where)
        layers.append(LayerSpec(prefix=f"l{i}", mixer=mixer, feed_forward=ffn, norms=norms, position=_rotation(l.mixer, where),
                                block="hyper_connections", names=RUBULIX_LAYER_NAMES,
                                block_params={"streams": cfg.streams, "mixer_names": stream_names(i, 1), "ffn_names": stream_names(i, 2)}))
        schedule.append(Run(layer=i, cache=i if l.kv_from is None else l.kv_from, writes_cache=l.kv_from is None))
    return ModelSpec(
        architecture="Rubulix", hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "embed"}),
        final_norm=PartSpec("stream_sum", {"norm": norm("final.norm"), "streams": cfg.streams}),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied": False, "name": "head"}),
        layers=layers, schedule=schedule, max_context_len=cfg.max_positions, eos_token_ids=list(cfg.eos_token_ids),
        checkpoint_dtype="bfloat16")


register_architecture("Rubulix", RubulixConfig, build_rubulix_spec)
