"""Small Pokatar configurations with seeded random weights for the tests.

Sizes differ from configuration to configuration in everything the design lets differ: width, vocabulary, order and kinds of the
layers, heads and kv heads (also equal, also a single one, also more query heads a kv head than a kernel's block takes), key
and value sizes that are equal (the engine's paged attention kernels), differ from each other or are no multiple of 16 or of 8
(the kernels that take any pair), latent and rotated sizes whose sum is or is not one the tensor-core kernels take, frequency
scaling that puts pairs on the whole ramp, on one side of it, or none, experts with and without identity outputs, groups (also
one, also all kept, also of one output each), `top` of 1 and of all outputs, a shared expert or none, layers without
feed-forward.  The fixed configurations have few routers that really choose, so that few positions lie near a close call, where a
bfloat16 run may choose otherwise.  Weights are drawn in float32 from a generator seeded by (seed, tensor name), sized so that
every sublayer moves the stream visibly, and rounded to bfloat16 so that the engine and the plain implementation hold the same
numbers.  This file shares nothing with the engine package.
"""

from __future__ import annotations

import copy
import hashlib
import math
import random
from typing import Dict

import torch


def att(heads, kv_heads, dim, vdim, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                           "scale": scale if scale is not None else dim ** -0.5}}


def latent(heads, dim, rot_dim, vdim, kv_rank, *, base=10000.0, scaling=None, scale=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(scaling)
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": rot}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, *, identity=None, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if identity is not None:
        r["identity"] = identity
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(mixer, mlp):
    out = copy.deepcopy(mixer)
    out["mlp"] = copy.deepcopy(mlp)
    return out


def model(width, vocab, eps, layers):
    return {"architecture": "Pokatar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


RAMP = {"factor": 4.0, "original": 32, "fast": 8.0, "slow": 1.0}

# A: every kind of layer; key and value sizes that differ; a latent row of 56 (no tensor-core size) and equal head sizes of 32;
#    a router with groups and identity outputs, one that takes every output it has
TINY_KA = model(72, 107, 1e-5, [
    layer(att(6, 3, 40, 24, scale=0.2), dense(56)),
    layer(latent(3, 24, 16, 20, 40, base=500.0, scaling=RAMP, scale=0.3), moe(6, 3, 24, identity=2, groups=(4, 2), shared=40)),
    layer(att(4, 2, 32, 32), moe(3, 4, 40, identity=1)),
    layer(latent(2, 8, 4, 12, 12, base=100.0), None),
    layer(att(2, 1, 8, 8, scale=0.5), dense(33)),
])

# B: what a model may happen to make equal or 1: a single head, one kv head per head, one expert per token, one group, no identity
#    output, no shared expert, a head size that is no multiple of 8, pages of one token; no feed-forward behind the first layer
TINY_KB = model(50, 61, 1e-6, [
    layer(latent(1, 20, 8, 20, 20, base=50.0, scaling={"factor": 2.0, "original": 4096, "fast": 32.0, "slow": 1.0}), None),
    layer(att(1, 1, 36, 36, scale=0.25), moe(2, 1, 16, groups=(1, 1))),
    layer(att(3, 3, 16, 16), dense(8)),
    layer(att(2, 2, 10, 14), moe(1, 2, 24, identity=1, groups=(2, 2), shared=8)),
])

# C: sizes of the tensor-core kernels: head size 128 (prompts on tcgen05), 24 query heads on one kv head, latent rows of 64 and
#    of 128; many experts in many groups
TINY_KC = model(96, 131, 1e-5, [
    layer(att(4, 2, 128, 128), moe(14, 5, 32, identity=2, groups=(8, 3), shared=32)),
    layer(latent(4, 32, 16, 24, 48, base=50000.0, scaling={"factor": 8.0, "original": 128, "fast": 16.0, "slow": 2.0}), dense(80)),
    layer(att(24, 1, 16, 16, scale=0.4), moe(4, 6, 16, identity=2, groups=(2, 2))),
    layer(latent(2, 64, 32, 64, 96, base=10000.0, scaling=RAMP), dense(40)),
])

CONFIGS_K = {"KA": TINY_KA, "KB": TINY_KB, "KC": TINY_KC}


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    E, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, E), "final.norm": (E,)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        out[p + "norm1"] = (E,)
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if l["type"] == "attention":
            G = m["kv_heads"]
            out.update({p + "mix.q": (H * d, E), p + "mix.k": (G * d, E), p + "mix.v": (G * dv, E), p + "mix.q.norm": (d,),
                        p + "mix.k.norm": (d,), p + "mix.g": (H * dv, E), p + "mix.o": (E, H * dv)})
        else:
            r, rd = m["kv_rank"], m["rot_dim"]
            out.update({p + "mix.q": (H * (d + rd), E), p + "mix.dkv": (r + rd, E), p + "mix.dkv.norm": (r,), p + "mix.uk": (H * d, r),
                        p + "mix.uv": (H * dv, r), p + "mix.g": (H, E), p + "mix.o": (E, H * dv)})
        f = l["mlp"]
        if f is None:
            continue
        out[p + "norm2"] = (E,)
        if f["kind"] == "dense":
            ff = f["ff"]
            out.update({p + "mlp.gate": (ff, E), p + "mlp.gate.b": (ff,), p + "mlp.up": (ff, E), p + "mlp.up.b": (ff,),
                        p + "mlp.down": (E, ff), p + "mlp.down.b": (E,)})
        else:
            n, ff = f["router"]["experts"], f["expert"]["ff"]
            outs = n + f["router"].get("identity", 0)
            out.update({p + "mlp.router": (outs, E), p + "mlp.correction": (outs,)})
            for e in range(n):
                out.update({f"{p}mlp.e{e}.up": (ff, E), f"{p}mlp.e{e}.down": (E, ff)})
            if f.get("shared"):
                out.update({p + "mlp.shared.up": (f["shared"]["ff"], E), p + "mlp.shared.down": (E, f["shared"]["ff"])})
    return out


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors by checkpoint name."""
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        h = hashlib.sha256(f"{seed}:{name}".encode()).digest()
        g = torch.Generator(device="cpu").manual_seed(int.from_bytes(h[:7], "little"))
        r = torch.randn(shape, generator=g, dtype=torch.float32)
        last = name.rsplit(".", 1)[-1]
        if last == "b":
            t = 0.3 * r
        elif last == "correction":
            t = 0.25 * r                          # as large as the scores: choices with a negative score among them
        elif name.endswith("mix.q.norm") or name.endswith("mix.k.norm"):
            t = 1.4 + 0.2 * r                     # scores spread over a few units, so that keys are told apart
        elif len(shape) == 1:
            t = 1.0 + 0.1 * r                     # norm weights
        elif name == "embed":
            t = 0.5 * r
        elif last == "router":
            t = 2.0 * r / math.sqrt(shape[1])
        elif name.endswith("mix.q") or name.endswith("mix.dkv"):
            t = 1.5 * r / math.sqrt(shape[1])
        else:
            t = r / math.sqrt(shape[1])           # a projection: outputs about as large as its inputs
        out[name] = t.to(torch.bfloat16)
    return out


def random_config(seed: int) -> dict:
    """A seeded configuration: two to five layers of either kind in any order with a feed-forward of either kind or none."""
    rng = random.Random(4000 + seed)
    width = rng.choice([40, 56, 64, 90, 128])
    vocab = rng.choice([53, 89, 150, 257])
    layers = []
    for _ in range(rng.randint(2, 5)):
        if rng.random() < 0.5:
            G = rng.choice([1, 2, 3])
            d = rng.choice([8, 16, 32, 44, 64, 128])
            dv = d if rng.random() < 0.5 else rng.choice([8, 20, 48])
            mixer = att(G * rng.choice([1, 2, 5]), G, d, dv, scale=rng.choice([None, 0.15, 0.4]))
        else:
            rd = rng.choice([4, 8, 16])
            sc = rng.choice([None, {"factor": rng.choice([2.0, 16.0]), "original": rng.choice([16, 64, 512]), "fast": rng.choice([4.0, 32.0]),
                                    "slow": rng.choice([0.5, 1.0])}])
            mixer = latent(rng.choice([1, 2, 5]), rng.choice([8, 20, 32]), rd, rng.choice([8, 24, 30]), rng.choice([12, 24, 48]),
                           base=rng.choice([30.0, 10000.0, 500000.0]), scaling=sc, scale=rng.choice([None, 0.3]))
        kind = rng.choice(["none", "dense", "moe", "moe"])
        if kind == "none":
            mlp = None
        elif kind == "dense":
            mlp = dense(rng.choice([8, 24, 41]))
        else:
            count = rng.choice([1, 2, 4])
            size = rng.choice([1, 2, 3])
            keep = rng.randint(1, count)
            outs = count * size
            ident = rng.randint(0, min(outs - 1, 3))
            mlp = moe(outs - ident, rng.randint(1, keep * size), rng.choice([8, 20, 40]), identity=ident or None,
                      groups=(count, keep) if count > 1 or rng.random() < 0.5 else None, shared=rng.choice([None, 8, 24]))
        layers.append(layer(mixer, mlp))
    return model(width, vocab, rng.choice([1e-5, 1e-6]), layers)
