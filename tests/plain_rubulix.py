"""A plain, slow implementation of the Rubulix decoder, one function per mechanism, written from the
architecture's equations and sharing no code with the engine.  It takes the content of a config.json and a
dict of tensors by checkpoint name and runs one whole sequence at a time on the CPU; there is no cache: every
function sees all tokens of the sequence.

Notation: T tokens, width E, S copies of the stream X [T, S, E], u the normed input of a sublayer.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# -- norms ----------------------------------------------------------------------------------------------------------

def layer_norm(x, weight, bias, eps):
    """Mean taken off, over the root of the mean squared deviation plus eps, times a weight, plus a bias."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * weight + bias


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


# -- several copies of the stream -------------------------------------------------------------------------------------

def read_streams(X, w_in):
    """What a sublayer sees: the copies weighted and added."""
    out = torch.zeros_like(X[:, 0])
    for s in range(X.shape[1]):
        out = out + w_in[s] * X[:, s]
    return out


def write_streams(X, y, mix, w_out):
    """Every copy anew from all old ones (mix[from][to]) plus its share of the sublayer's output y."""
    new = []
    for t in range(X.shape[1]):
        acc = w_out[t] * y
        for s in range(X.shape[1]):
            acc = acc + mix[s, t] * X[:, s]
        new.append(acc)
    return torch.stack(new, dim=1)


# -- rotation -------------------------------------------------------------------------------------------------------

def frequencies(dims: int, base: float, scaling: Optional[dict]):
    """-> (frequencies [dims / 2], factor on cos and sin): geometric; with `scaling`, blended into frequencies divided by
    `factor` along a ramp over the pair index between the pairs that turn `fast` and `slow` times in `original` tokens."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_neighbours(x, freq, magnitude):
    """x [T, ..., d], token t at position t: elements 2 i and 2 i + 1 turn together by t * freq[i]; what lies beyond the pairs
    passes."""
    y = x.clone()
    t = torch.arange(x.shape[0], dtype=torch.float64)
    for i, f in enumerate(freq):
        shape = (x.shape[0],) + (1,) * (x.dim() - 2)
        c = (torch.cos(t * f) * magnitude).to(x.dtype).view(shape)
        s = (torch.sin(t * f) * magnitude).to(x.dtype).view(shape)
        a, b = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = a * c - b * s
        y[..., 2 * i + 1] = b * c + a * s
    return y


def rotation_of(c: dict):
    rot = c["rot"]
    return frequencies(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))


# -- mixers ---------------------------------------------------------------------------------------------------------

def causal(T: int):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return j <= i


def same_chunk(T: int, size: int):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def softmax_attention(q, k, v, scale, seen):
    """One head: q [T, d], k [T, d], v [T, dv], seen [T, T]."""
    s = (q @ k.T * scale).masked_fill(~seen, float("-inf"))
    return torch.softmax(s, dim=-1) @ v


def project(u, w, name):
    return u @ w[name].T + w[name + ".b"]


def difference_weight(w, p: str, diff: float):
    a = torch.exp((w[p + ".lq1"].double() * w[p + ".lk1"].double()).sum())
    b = torch.exp((w[p + ".lq2"].double() * w[p + ".lk2"].double()).sum())
    return float(a - b) + diff


def differential_keys_values(u, w, p: str, c: dict):
    """-> keys [T, G, 2, d] (turned) and values [T, G, dv] of a layer that makes its own."""
    T, G, d = u.shape[0], c["kv_heads"], c["dim"]
    k = rotate_neighbours(project(u, w, p + ".k").view(T, G, 2, d), *rotation_of(c))
    return k, project(u, w, p + ".v").view(T, G, c["vdim"])


def differential_attention(u, kv, w, p: str, c: dict, eps: float):
    """Two softmax maps over the same values, the second taken off the first lambda times; every head's result brought to
    unit root mean square and scaled by one minus the constant part of lambda."""
    T = u.shape[0]
    H, G, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = rotate_neighbours(project(u, w, p + ".q").view(T, H, 2, d), *rotation_of(c))
    k, v = kv
    lam = difference_weight(w, p, float(c["diff"]))
    seen = causal(T)
    out = torch.zeros(T, H, dv, dtype=u.dtype)
    for h in range(H):
        g = h // (H // G)
        a1 = softmax_attention(q[:, h, 0], k[:, g, 0], v[:, g], c["scale"], seen)
        a2 = softmax_attention(q[:, h, 1], k[:, g, 1], v[:, g], c["scale"], seen)
        out[:, h] = rms_unit(a1 - lam * a2, eps) * (1.0 - float(c["diff"]))
    return out.reshape(T, H * dv) @ w[p + ".o"].T


def chunked_attention(u, w, p: str, c: dict, eps: float):
    """Attention within chunks of the sequence; q and k of unit root mean square after the rotation; the heads side by side
    times sigmoid(Wg u)."""
    T = u.shape[0]
    H, G, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    rot = rotation_of(c)
    q = rms_unit(rotate_neighbours(project(u, w, p + ".q").view(T, H, d), *rot), eps)
    k = rms_unit(rotate_neighbours(project(u, w, p + ".k").view(T, G, d), *rot), eps)
    v = project(u, w, p + ".v").view(T, G, dv)
    seen = same_chunk(T, int(c["mask"]["size"]))
    out = torch.zeros(T, H, dv, dtype=u.dtype)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_attention(q[:, h], k[:, g], v[:, g], c["scale"], seen)
    return (out.reshape(T, H * dv) * torch.sigmoid(u @ w[p + ".g"].T)) @ w[p + ".o"].T


# -- feed-forward -----------------------------------------------------------------------------------------------------

def dense(u, w, p: str):
    z = u @ w[p + ".gate"].T
    return (z * torch.sigmoid(z) * (u @ w[p + ".up"].T)) @ w[p + ".down"].T


# -- the model ------------------------------------------------------------------------------------------------------

def forward_sequence(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float32, layers_out: Optional[list] = None):
    """-> logits [T, vocab] for every place of the sequence.  layers_out, if given, receives the sum of the copies after every
    layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    X = torch.stack([x] * int(cfg["streams"]), dim=1)
    kv_of = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        u = layer_norm(read_streams(X, w[p + ".hc1.in"]), w[p + ".norm1"], w[p + ".norm1.b"], eps)
        c = layer["mixer"]
        if layer["type"] == "attention":
            if c.get("kv_from") is None:
                kv_of[i] = differential_keys_values(u, w, p + ".mix", c)
            y = differential_attention(u, kv_of[i if c.get("kv_from") is None else int(c["kv_from"])], w, p + ".mix", c, eps)
        else:
            y = chunked_attention(u, w, p + ".mix", c, eps)
        X = write_streams(X, y, w[p + ".hc1.mix"], w[p + ".hc1.out"])
        if layer.get("mlp") is not None:
            u = layer_norm(read_streams(X, w[p + ".hc2.in"]), w[p + ".norm2"], w[p + ".norm2.b"], eps)
            X = write_streams(X, dense(u, w, p + ".mlp"), w[p + ".hc2.mix"], w[p + ".hc2.out"])
        if layers_out is not None:
            layers_out.append(X.sum(dim=1))
    return layer_norm(X.sum(dim=1), w["final.norm"], w["final.norm.b"], eps) @ w["head"].T


def greedy_generate(cfg: dict, w: Dict[str, torch.Tensor], prompt: List[int], n: int) -> List[int]:
    toks = list(prompt)
    for _ in range(n):
        with torch.no_grad():
            toks.append(int(forward_sequence(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
