"""Small Rubulix configurations with seeded random weights for the tests.

Sizes differ from configuration to configuration in everything the design lets differ: width (also one no vector access divides),
vocabulary, number of copies of the stream (also one), order and kinds of the layers, heads and kv heads (also equal, also a
single one, also more query heads a kv head than a kernel's block takes), key and value sizes that put a layer on the engine's
paged attention kernels (a cache row of keys as long as one of values) or on the kernels that take any pair, rotated parts that
are the whole vector, a part of it or nothing, frequency scaling with pairs on the whole ramp, on one side of it, or none, chunks
of one token, of sizes that divide neither pages nor tiles, and wider than a prompt, layers that read the keys and values of an
earlier one (several of one, with other layers between), layers without feed-forward.  Weights are drawn in float32 from a
generator seeded by (seed, tensor name), sized so that every sublayer moves the stream visibly, and rounded to bfloat16 so that
the engine and the plain implementation hold the same numbers.  This file shares nothing with the engine package.
"""

from __future__ import annotations

import copy
import hashlib
import math
import random
from typing import Dict

import torch

RAMP = {"factor": 4.0, "original": 32, "fast": 8.0, "slow": 1.0}


def _rot(dims, base, scaling):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(scaling)
    return rot


def diff(heads, kv_heads, dim, vdim, *, dims, lam=0.3, base=10000.0, scaling=None, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": lam, "scale": scale if scale is not None else dim ** -0.5,
         "rot": _rot(dims, base, scaling)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def chunked(heads, kv_heads, dim, vdim, size, *, dims, base=10000.0, scale=None):
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
                                             "scale": scale if scale is not None else dim ** -0.5, "rot": _rot(dims, base, None)}}


def layer(mixer, ff):
    out = copy.deepcopy(mixer)
    out["mlp"] = {"kind": "dense", "ff": ff} if ff else None
    return out


def model(width, vocab, streams, eps, layers):
    return {"architecture": "Rubulix", "width": width, "vocab": vocab, "streams": streams, "norm": {"eps": eps}, "layers": layers}


# A: every kind of layer on both kinds of kernels; two layers on the keys and values of one, one of them not its neighbour
TINY_RA = model(72, 107, 3, 1e-5, [
    layer(chunked(6, 3, 40, 24, 20, dims=24, base=500.0), 56),
    layer(diff(4, 2, 16, 32, dims=8, base=100.0, scaling=RAMP), 40),
    layer(diff(4, 2, 16, 32, dims=8, base=100.0, scaling=RAMP, kv_from=1, lam=0.6, scale=0.4), 33),
    layer(chunked(4, 2, 32, 32, 33, dims=32), None),
    layer(diff(2, 1, 12, 20, dims=12, base=300.0, lam=0.1), 24),
    layer(diff(4, 2, 16, 32, dims=8, base=100.0, scaling=RAMP, kv_from=1, lam=0.2), None),
])

# B: what a model may happen to make equal or 1: one copy of the stream, a single head, a kv head per head, key and value sizes
#    alike, a width that is a multiple of 2 only, chunks of one token and chunks no prompt fills, pages of one token
TINY_RB = model(50, 61, 1, 1e-6, [
    layer(chunked(1, 1, 20, 20, 1, dims=20), 8),
    layer(diff(1, 1, 10, 20, dims=4, base=50.0, scaling={"factor": 2.0, "original": 4096, "fast": 32.0, "slow": 1.0}), None),
    layer(chunked(3, 3, 16, 16, 7, dims=2, base=20.0, scale=0.3), 24),
    layer(diff(2, 2, 7, 9, dims=6, lam=0.5), 17),
    layer(chunked(2, 2, 10, 14, 4096, dims=10), 16),
])

# C: sizes of the tensor-core kernels: rows of 128 (prompts on tcgen05), many query heads on one kv head, four copies
TINY_RC = model(96, 131, 4, 1e-5, [
    layer(diff(4, 2, 64, 128, dims=64, base=50000.0, scaling={"factor": 8.0, "original": 128, "fast": 16.0, "slow": 2.0}), 80),
    layer(chunked(4, 2, 128, 128, 48, dims=64, base=1000.0), 64),
    layer(diff(4, 2, 64, 128, dims=64, base=50000.0, scaling={"factor": 8.0, "original": 128, "fast": 16.0, "slow": 2.0}, kv_from=0), None),
    layer(chunked(24, 1, 16, 16, 100, dims=16, scale=0.4), 48),
    layer(diff(24, 1, 16, 32, dims=16, base=400.0, lam=0.4), 32),
])

CONFIGS_R = {"RA": TINY_RA, "RB": TINY_RB, "RC": TINY_RC}


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    E, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    out = {"embed": (V, E), "final.norm": (E,), "final.norm.b": (E,), "head": (V, E)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        two = 2 if l["type"] == "attention" else 1
        sub = 2 if l["mlp"] is not None else 1
        for q in range(1, sub + 1):
            out.update({f"{p}norm{q}": (E,), f"{p}norm{q}.b": (E,), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
        out.update({p + "mix.q": (H * two * d, E), p + "mix.q.b": (H * two * d,), p + "mix.o": (E, H * dv)})
        if m.get("kv_from") is None:
            out.update({p + "mix.k": (G * two * d, E), p + "mix.k.b": (G * two * d,), p + "mix.v": (G * dv, E), p + "mix.v.b": (G * dv,)})
        if l["type"] == "attention":
            out.update({p + "mix." + n: (d,) for n in ("lq1", "lk1", "lq2", "lk2")})
        else:
            out[p + "mix.g"] = (H * dv, E)
        if l["mlp"] is not None:
            ff = l["mlp"]["ff"]
            out.update({p + "mlp.gate": (ff, E), p + "mlp.up": (ff, E), p + "mlp.down": (E, ff)})
    return out


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors by checkpoint name."""
    out = {}
    S = cfg["streams"]
    for name, shape in tensor_shapes(cfg).items():
        h = hashlib.sha256(f"{seed}:{name}".encode()).digest()
        g = torch.Generator(device="cpu").manual_seed(int.from_bytes(h[:7], "little"))
        r = torch.randn(shape, generator=g, dtype=torch.float32)
        last = name.rsplit(".", 1)[-1]
        if ".hc" in name:
            t = {"in": 1.0 / math.sqrt(S) + 0.3 * r, "out": 0.8 + 0.4 * r, "mix": 0.35 * r + (0.8 * torch.eye(S) if last == "mix" else 0.0)}[last]
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.45 * r / shape[0] ** 0.25      # lambda near, but not at, its constant part
        elif last == "b":
            t = 0.3 * r
        elif len(shape) == 1:
            t = 1.0 + 0.1 * r                     # norm weights
        elif name == "embed":
            t = 0.5 * r
        elif name.endswith("mix.q") or name.endswith("mix.k"):
            t = 1.4 * r / math.sqrt(shape[1])     # scores spread over a few units, so that keys are told apart
        else:
            t = r / math.sqrt(shape[1])           # a projection: outputs about as large as its inputs
        out[name] = t.to(torch.bfloat16)
    return out


def random_config(seed: int) -> dict:
    """A seeded configuration: three to six layers of either kind in any order, some on an earlier layer's keys and values."""
    rng = random.Random(7000 + seed)
    width = rng.choice([40, 56, 64, 90, 128])
    layers = []
    for i in range(rng.randint(3, 6)):
        own = [j for j, l in enumerate(layers) if l["type"] == "attention" and "kv_from" not in l["mixer"]]
        ff = rng.choice([None, 8, 24, 41, 64])
        if own and rng.random() < 0.4:
            j = rng.choice(own)
            m = copy.deepcopy(layers[j])
            m["mixer"].update(kv_from=j, diff=rng.choice([0.2, 0.5]))
            m["mlp"] = {"kind": "dense", "ff": ff} if ff else None
            layers.append(m)
            continue
        G = rng.choice([1, 2, 3])
        H = G * rng.choice([1, 2, 5])
        if rng.random() < 0.5:
            d = rng.choice([4, 8, 16, 22, 32, 64])
            dv = 2 * d if rng.random() < 0.6 else rng.choice([8, 20, 48])
            sc = rng.choice([None, {"factor": rng.choice([2.0, 16.0]), "original": rng.choice([16, 64, 512]), "fast": rng.choice([4.0, 32.0]),
                                    "slow": rng.choice([0.5, 1.0])}])
            layers.append(layer(diff(H, G, d, dv, dims=rng.choice([d, d // 2 // 2 * 2 or 2]), lam=rng.choice([0.1, 0.4]),
                                     base=rng.choice([30.0, 10000.0, 500000.0]), scaling=sc, scale=rng.choice([None, 0.3])), ff))
        else:
            d = rng.choice([8, 16, 32, 44, 64, 128])
            dv = d if rng.random() < 0.6 else rng.choice([8, 20, 48])
            layers.append(layer(chunked(H, G, d, dv, rng.choice([1, 5, 16, 24, 37, 64, 500]), dims=rng.choice([d, 4]),
                                        base=rng.choice([30.0, 500000.0]), scale=rng.choice([None, 0.15])), ff))
    return model(width, rng.choice([53, 89, 150, 257]), rng.choice([1, 2, 3, 4, 6]), rng.choice([1e-5, 1e-6]), layers)
