"""Pokatar: typed configuration and model description.

A decoder whose layers are listed one by one in config.json (`layers`): every entry names the kind of its mixer (`type`), the
mixer's sizes and constants (`mixer`) and its feed-forward (`mlp`, or null for none).  A layer is pre-norm with layer norms that
have a weight and no bias, on a float32 stream.  Mixers:

  attention          grouped-query softmax attention over all earlier keys without positions: q and k RMS-normed per head,
                     values of unit root mean square, one added to every softmax's denominator, the heads side by side times
                     a sigmoid gate per element
  latent_attention   keys and values of all heads from one RMS-normed latent per token, beside a rotated key part shared by all
                     heads (rotation in halves, YaRN's frequency scaling), one sigmoid gate per head

Feed-forwards: `dense` (down(relu(gate x) * up x), all three with biases) and `moe` (plain experts down(relu(up x)^2) chosen by
softmax score plus correction within the best groups and weighted by the score alone; some router outputs hand the input on;
a shared expert).  The head is the embedding table.  Everything that differs between models of the design is read here; nothing
else in the engine knows the design's name.
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
class PokatarLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


@dataclasses.dataclass
class PokatarConfig:
    width: int
    vocab: int
    norm_eps: float
    layers: List[PokatarLayer]
    max_positions: int = NO_POSITION_LIMIT
    eos_token_ids: List[int] = dataclasses.field(default_factory=list)
    raw: Dict[str, Any] = dataclasses.field(default_factory=dict, repr=False)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "PokatarConfig":
        layers = []
        for i, entry in enumerate(_need(raw, "layers", "the model")):
            where = f"layer {i}"
            layers.append(PokatarLayer(type=str(_need(entry, "type", where)), mixer=dict(_need(entry, "mixer", where)),
                                       mlp=dict(entry["mlp"]) if entry.get("mlp") is not None else None))
        eos = raw.get("eos_token_id", [])
        eos = [] if eos is None else ([int(e) for e in eos] if isinstance(eos, (list, tuple)) else [int(eos)])
        cfg = cls(width=int(_need(raw, "width", "the model")), vocab=int(_need(raw, "vocab", "the model")),
                  norm_eps=float(_need(_need(raw, "norm", "the model"), "eps", "norm")), layers=layers,
                  max_positions=int(raw.get("max_positions") or NO_POSITION_LIMIT), eos_token_ids=eos, raw=dict(raw))
        cfg.check()
        return cfg

    def check(self) -> None:
        if self.width <= 0 or self.vocab <= 0 or not self.layers:
            raise ConfigError("width, vocab and the number of layers must be positive")
        for i, l in enumerate(self.layers):
            if l.type not in _MIXERS:
                raise ConfigError(f"config.json: layer {i} has type {l.type!r}; known: " + ", ".join(sorted(_MIXERS)))
            if l.mlp is not None and l.mlp.get("kind") not in _FEED_FORWARDS:
                raise ConfigError(f"config.json: layer {i} has a feed-forward of kind {l.mlp.get('kind')!r}; known: "
                                  + ", ".join(sorted(_FEED_FORWARDS)))

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)


def _attention(cfg: PokatarConfig, m: Dict[str, Any], where: str):
    heads = int(_need(m, "heads", where))
    dim = int(_need(m, "dim", where))
    return PartSpec("sink_attention", {
        "hidden_size": cfg.width, "num_heads": heads, "num_kv_heads": int(m.get("kv_heads") or heads), "key_dim": dim,
        "value_dim": int(m.get("vdim") or dim), "scale": float(_need(m, "scale", where)), "window": None, "softcap": None,
        "bias": False, "value_mix": None, "sink": 0.0, "qk_norm": True, "value_norm": True, "norm_eps": cfg.norm_eps,
        "gate": "sigmoid", "names": {"q": "q", "k": "k", "v": "v", "q_norm": "q.norm", "k_norm": "k.norm", "gate": "g", "out": "o"}}), None


def _latent(cfg: PokatarConfig, m: Dict[str, Any], where: str):
    """-> (mixer, position encoding); without a rotated part (`rot_dim` 0 or absent) there is no encoding."""
    rot_dim = int(m.get("rot_dim") or 0)
    position = None
    if rot_dim:
        rot = _need(m, "rot", where)
        dims = int(rot.get("dims", rot_dim))
        if dims > rot_dim or dims % 2:
            raise ConfigError(f"config.json: {where}.rot: {dims} rotated dimensions must be even and at most rot_dim = {rot_dim}")
        sc = rot.get("scaling")
        scaling = {k: float(_need(sc, k, where + ".rot.scaling")) for k in ("factor", "original", "fast", "slow")} if sc else None
        position = PartSpec("rope_yarn", {"rotary_dim": dims, "theta": float(_need(rot, "base", where + ".rot")), "scaling": scaling})
    mixer = PartSpec("latent_attention", {
        "hidden_size": cfg.width, "num_heads": int(_need(m, "heads", where)), "key_dim": int(_need(m, "dim", where)),
        "rot_dim": rot_dim, "value_dim": int(_need(m, "vdim", where)), "kv_rank": int(_need(m, "kv_rank", where)), "q_rank": None,
        "scale": float(_need(m, "scale", where)), "window": None, "gate": "head_sigmoid", "norm_eps": cfg.norm_eps})
    return mixer, position


def _dense(cfg: PokatarConfig, f: Dict[str, Any], where: str) -> PartSpec:
    return PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": int(_need(f, "ff", where)), "activation": "relu",
                                  "bias": True, "names": {"gate": "gate", "up": "up", "down": "down", "gate_bias": "gate.b",
                                                          "up_bias": "up.b", "down_bias": "down.b"}})


def _moe(cfg: PokatarConfig, f: Dict[str, Any], where: str) -> PartSpec:
    r = _need(f, "router", where)
    g = r.get("groups") or {}
    count = int(g.get("count") or 1)
    sh = f.get("shared")
    return PartSpec("plain_experts", {
        "hidden_size": cfg.width, "intermediate_size": int(_need(_need(f, "expert", where), "ff", where + ".expert")),
        "activation": "relu2", "num_experts": int(_need(r, "experts", where + ".router")), "identity": int(r.get("identity") or 0),
        "top": int(_need(r, "top", where + ".router")), "groups": count, "keep_groups": int(g.get("keep") or count),
        "score": "softmax", "group_score": "max", "renormalize": False,
        "shared_size": int(_need(sh, "ff", where + ".shared")) if sh is not None else 0,
        "names": {"router": "router", "correction": "correction", "expert": "e{e}", "up": "up", "down": "down", "shared": "shared"}})


_MIXERS = {"attention": _attention, "latent_attention": _latent}
_FEED_FORWARDS = {"dense": _dense, "moe": _moe}
POKATAR_LAYER_NAMES = {"mixer": "mix", "feed_forward": "mlp"}


def build_pokatar_spec(cfg: PokatarConfig) -> ModelSpec:
    """embedding -> layers of (norm, mixer, sum; norm, feed-forward, sum) -> norm -> the embedding table as head.  One
    `LayerSpec` and one `Run` per listed layer."""
    def norm(name: str) -> PartSpec:
        return PartSpec("layernorm", {"size": cfg.width, "eps": cfg.norm_eps, "name": name})

    layers = []
    for i, l in enumerate(cfg.layers):
        norms = {"input": norm(f"l{i}.norm1")}
        ffn = None
        if l.mlp is not None:
            ffn = _FEED_FORWARDS[l.mlp["kind"]](cfg, l.mlp, f"layer {i}.mlp")
            norms["post_mixer"] = norm(f"l{i}.norm2")
        mixer, position = _MIXERS[l.type](cfg, l.mixer, f"layer {i}.mixer")
        layers.append(LayerSpec(prefix=f"l{i}", mixer=mixer, feed_forward=ffn, norms=norms, position=position,
                                block="prenorm_residual", names=POKATAR_LAYER_NAMES))
    return ModelSpec(
        architecture="Pokatar", hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "embed"}),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied": True, "name": "head", "tied_to": "embed"}),
        layers=layers, schedule=[Run(layer=i, cache=i) for i in range(len(cfg.layers))],
        max_context_len=cfg.max_positions, eos_token_ids=list(cfg.eos_token_ids), checkpoint_dtype="bfloat16")


register_architecture("Pokatar", PokatarConfig, build_pokatar_spec)
