"""A plain, slow implementation of the Pokatar decoder, one function per mechanism, written from the
architecture's equations and sharing no code with the engine.  It takes the content of a config.json and a
dict of tensors by checkpoint name and runs one whole sequence at a time on the CPU; there is no cache: every
function sees all tokens of the sequence.

Notation: T tokens, width E, x the residual stream [T, E], u the normed input of a sublayer.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# -- norms ----------------------------------------------------------------------------------------------------------

def layer_norm(x, weight, eps):
    """Mean taken off, over the root of the mean squared deviation plus eps, times a weight; no bias."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * weight


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


# -- rotation -------------------------------------------------------------------------------------------------------

def frequencies(dims: int, base: float, scaling: Optional[dict]):
    """-> (frequencies [dims / 2], factor on cos and sin): geometric; with `scaling`, blended into frequencies divided by
    `factor` along a ramp over the pair index between the pairs that turn `fast` and `slow` times in `original` tokens."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=torch.float64), 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def rotate(x, freq, magnitude):
    """x [T, ..., d], token t at position t: element i turns against element i + n for the n frequencies; what lies beyond
    2 n passes."""
    n = freq.numel()
    if n == 0:
        return x
    ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * freq[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (n,)
    cos, sin = (ang.cos() * magnitude).to(x.dtype).view(shape), (ang.sin() * magnitude).to(x.dtype).view(shape)
    a, b = x[..., :n], x[..., n:2 * n]
    return torch.cat((a * cos - b * sin, b * cos + a * sin, x[..., 2 * n:]), dim=-1)


# -- mixers ---------------------------------------------------------------------------------------------------------

def causal(s):
    T = s.shape[0]
    return s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))


def softmax_with_one(s):
    """exp(s_j) / (1 + sum_j exp(s_j)) along the last dimension, kept finite by taking off the larger of 0 and the maximum."""
    m = s.max(dim=-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(dim=-1, keepdim=True))


def attention(u, w, p: str, c: dict, eps: float):
    """Grouped-query attention without positions: per-head norms of q and k, values of unit root mean square, one added to
    every softmax's denominator, the heads side by side times sigmoid(Wg u)."""
    T = u.shape[0]
    H, G, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = rms_unit((u @ w[p + ".q"].T).view(T, H, d), eps) * w[p + ".q.norm"]
    k = rms_unit((u @ w[p + ".k"].T).view(T, G, d), eps) * w[p + ".k.norm"]
    v = rms_unit((u @ w[p + ".v"].T).view(T, G, dv), eps)
    out = torch.zeros(T, H, dv, dtype=u.dtype)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_with_one(causal(q[:, h] @ k[:, g].T * c["scale"])) @ v[:, g]
    gate = torch.sigmoid(u @ w[p + ".g"].T)
    return (out.reshape(T, H * dv) * gate) @ w[p + ".o"].T


def latent_attention(u, w, p: str, c: dict, eps: float):
    """Attention whose keys and values are made from one normed latent per token, with one rotated key part for all heads;
    every head's output times one sigmoid."""
    T = u.shape[0]
    H, d, rd, dv, r = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    rot = c["rot"]
    freq, mag = frequencies(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
    q = (u @ w[p + ".q"].T).view(T, H, d + rd)
    q_plain, q_rot = q[..., :d], rotate(q[..., d:], freq, mag)
    down = u @ w[p + ".dkv"].T
    lat = rms_unit(down[:, :r], eps) * w[p + ".dkv.norm"]
    k_rot = rotate(down[:, r:], freq, mag)
    k = (lat @ w[p + ".uk"].T).view(T, H, d)
    v = (lat @ w[p + ".uv"].T).view(T, H, dv)
    gate = torch.sigmoid(u @ w[p + ".g"].T)
    out = torch.zeros(T, H, dv, dtype=u.dtype)
    for h in range(H):
        s = (q_plain[:, h] @ k[:, h].T + q_rot[:, h] @ k_rot.T) * c["scale"]
        out[:, h] = (torch.softmax(causal(s), dim=-1) @ v[:, h]) * gate[:, h:h + 1]
    return out.reshape(T, H * dv) @ w[p + ".o"].T


# -- feed-forwards --------------------------------------------------------------------------------------------------

def dense(u, w, p: str):
    gate = u @ w[p + ".gate"].T + w[p + ".gate.b"]
    up = u @ w[p + ".up"].T + w[p + ".up.b"]
    return (torch.relu(gate) * up) @ w[p + ".down"].T + w[p + ".down.b"]


def expert(u, w, p: str):
    return torch.relu(u @ w[p + ".up"].T) ** 2 @ w[p + ".down"].T


def choose(s, correction, groups: int, keep: int, top: int):
    """One token's scores [n] -> (chosen indices, gap of the choice).  The gap is the smaller of the distances between the last
    kept and the first dropped group, and between the last chosen and the first eligible one that was not."""
    choice = (s + correction).tolist()
    n = len(choice)
    size = n // groups
    best = [max(choice[g * size:(g + 1) * size]) for g in range(groups)]
    order = sorted(range(groups), key=lambda g: (-best[g], g))
    gap = best[order[keep - 1]] - best[order[keep]] if keep < groups else math.inf
    kept = set(order[:keep])
    eligible = sorted((e for e in range(n) if e // size in kept), key=lambda e: (-choice[e], e))
    if top < len(eligible):
        gap = min(gap, choice[eligible[top - 1]] - choice[eligible[top]])
    return eligible[:top], gap


def mixture(u, w, p: str, c: dict, margins: Optional[list] = None):
    """Experts chosen within the best groups by softmax score plus correction, weighted by the score alone; the last
    `identity` router outputs hand the input on; a shared expert is added.  margins, if given, receives the choices' gaps [T]."""
    r = c["router"]
    n, ident = int(r["experts"]), int(r.get("identity") or 0)
    g = r.get("groups") or {}
    count = int(g.get("count") or 1)
    keep = int(g.get("keep") or count)
    scores = torch.softmax(u @ w[p + ".router"].T, dim=-1)
    correction = w.get(p + ".correction")
    if correction is None:
        correction = torch.zeros(n + ident, dtype=u.dtype)
    out = torch.zeros_like(u)
    gaps = []
    for t in range(u.shape[0]):
        chosen, gap = choose(scores[t], correction, count, keep, int(r["top"]))
        gaps.append(gap)
        for e in chosen:
            y = expert(u[t:t + 1], w, f"{p}.e{e}")[0] if e < n else u[t]
            out[t] += scores[t, e] * y
    if c.get("shared"):
        out = out + expert(u, w, p + ".shared")
    if margins is not None:
        margins.append(torch.tensor(gaps))
    return out


# -- the model ------------------------------------------------------------------------------------------------------

MIXERS = {"attention": attention, "latent_attention": latent_attention}


def forward_sequence(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float32, layers_out: Optional[list] = None,
                     margins: Optional[list] = None):
    """-> logits [T, vocab] for every place of the sequence.  layers_out, if given, receives the stream after every layer;
    margins the routers' gaps, one tensor [T] per routed layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        x = x + MIXERS[layer["type"]](layer_norm(x, w[p + ".norm1"], eps), w, p + ".mix", layer["mixer"], eps)
        f = layer.get("mlp")
        if f is not None:
            u = layer_norm(x, w[p + ".norm2"], eps)
            x = x + (dense(u, w, p + ".mlp") if f["kind"] == "dense" else mixture(u, w, p + ".mlp", f, margins))
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy_generate(cfg: dict, w: Dict[str, torch.Tensor], prompt: List[int], n: int) -> List[int]:
    toks = list(prompt)
    for _ in range(n):
        with torch.no_grad():
            toks.append(int(forward_sequence(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
