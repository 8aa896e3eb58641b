"""The Pokatar parts and the whole model in the engine against the plain implementation (tests/plain_pokatar.py).

Kernels one by one; the attention with one added to the denominator and gates on the output through every kernel that may run
it, with inputs made so that a fault shows (one key whose score stands far above hundreds of others: the first token, far
away, page borders, the borders of the pieces a decoded token's keys are cut into, the token itself, the future; scores so low
that the added one takes nearly all the weight); then the model through the step function: whole prompts, token by token, in
portions down to two tokens, mixed batches on a pool so small that pages and request slots are used again, long decoding,
greedy generation through the engine's entry point with and without a shared prefix, and the trace replay program.
"""

import functools
import json
import math
import os
import subprocess
import sys
import tempfile

import numpy as np
import pytest
import torch

import plain_pokatar as pk
import tiny_pokatar as tk
from helpers import play
from tiny_models import random_tokens, write_model_dir
from tiny_pokatar import CONFIGS_K, make_weights, random_config

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
SEED = {"KA": 3, "KB": 4, "KC": 5}
PAGE = {"KA": 4, "KB": 1, "KC": 16}
_tmp = tempfile.TemporaryDirectory(prefix="msgl_pokatar_")
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64
BOTH = ["float32", "bfloat16"]


@functools.lru_cache(None)
def weights(name):
    return make_weights(CONFIGS_K[name], SEED[name])


@functools.lru_cache(None)
def model_dir(name):
    return write_model_dir(os.path.join(_tmp.name, name), CONFIGS_K[name], weights(name))


def plain_of(cfg, w, tokens):
    """The plain implementation in double precision: logits and, per position, the closest call any router made there."""
    margins = []
    with torch.no_grad():
        logits = pk.forward_sequence(cfg, w, list(tokens), dtype=F64, margins=margins).float()
    return logits, (torch.stack(margins).amin(dim=0) if margins else torch.full((len(tokens),), math.inf, dtype=F64))


@functools.lru_cache(None)
def _plain_run(name, tokens):
    return plain_of(CONFIGS_K[name], weights(name), tokens)


def runner(name, dtype, num_pages, max_reqs=4, page_size=None, graphs=True, ctx=1024):
    from mini_sglang_b200.engine.step import ModelRunner
    return ModelRunner.from_model_dir(model_dir(name), dtype=dtype, page_size=page_size or PAGE[name], num_pages=num_pages,
                                      max_reqs=max_reqs, max_context_len=ctx, use_cuda_graph=graphs)


# The reference is the plain implementation in double precision.  float32 rows are held to 2e-4 of a row's rms (6 times that for
# the largest element).  bfloat16: projections, cached keys, values and latents and the activations between kernels are rounded to
# 8 mantissa bits; scores, softmax, norms, routers and the stream are float32 in both precisions.  The bound is 4 % of a row's
# rms; the faults it is meant to catch move the rows by 4.5 % or more (tests/test_pokatar_cpu.py).  A router whose input is
# rounded to bfloat16 may choose otherwise where two choice scores lie within CLOSE_CALL of each other: such a position, and
# the one behind it (it reads the changed keys and values), must only stay finite and within LOOSE of the reference; the
# float32 run of the same schedule holds their logic.
F32_RMS_FRACTION = 2e-4
BF16_RMS_FRACTION_K = 0.04
CLOSE_CALL, FADE, LOOSE = 0.015, 1, 0.9
TAIL_SHARE, TAIL_FACTOR = 0.1, 6.0


def row_close(row, want, dtype, bound=None):
    if bound is None:
        bound = F32_RMS_FRACTION if dtype == "float32" else BF16_RMS_FRACTION_K
    row, want = row.float(), want.float()
    assert torch.isfinite(row).all(), "logits are not finite"
    err = row - want
    scale = want.pow(2).mean().sqrt().item()
    rms, worst = err.pow(2).mean().sqrt().item(), err.abs().max().item()
    assert rms <= bound * scale, f"rms error {rms:.4g} is {rms / scale:.4%} of the row's rms {scale:.4g}"
    assert worst <= 6.0 * bound * scale, f"largest error {worst:.4g} is {worst / scale:.4%} of the row's rms {scale:.4g}"


def compare(name, dtype, got, seqs, ref=None, bound=None, min_firm=0.25, close=CLOSE_CALL):
    """Every row against the plain implementation.  bfloat16: rows at and right behind a router's close call are held loosely (see
    above), and up to TAIL_SHARE of a request's other rows (at least one) may lie in the tail of the noise, none by more than
    TAIL_FACTOR times the bound.  A fault of the cache or of the batch moves every row behind it, in float32 as well."""
    assert got
    if bound is None:
        bound = F32_RMS_FRACTION if dtype == "float32" else BF16_RMS_FRACTION_K
    over, firm = {}, 0
    for (rid, pos), row in sorted(got.items()):
        want, margin = ref[rid] if ref is not None else _plain_run(name, tuple(seqs[rid]))
        shaky = dtype == "bfloat16" and bool((margin[max(0, pos - FADE):pos + 1] < close).any())
        firm += not shaky
        try:
            row_close(row, want[pos], dtype, LOOSE if shaky else bound)
        except AssertionError as e:
            if dtype == "bfloat16" and not shaky and torch.isfinite(row).all():
                try:
                    row_close(row, want[pos], dtype, TAIL_FACTOR * bound)
                    over.setdefault(rid, []).append(pos)
                    continue
                except AssertionError:
                    pass
            raise AssertionError(f"request {rid!r} position {pos} ({dtype}, {name}): {e}") from None
    assert firm >= min_firm * len(got) or len(got) < 10, f"only {firm} of {len(got)} rows are away from every router's close calls"
    for rid, places in over.items():
        rows = sum(1 for k in got if k[0] == rid)
        assert len(places) <= max(1, int(TAIL_SHARE * rows)), \
            f"request {rid!r}: {len(places)} of {rows} rows beyond the bound ({dtype}, {name}): {places}"


def poison(r):
    """Whatever a page held before must not be read: fill the caches with NaN.  Page 0 is never handed out."""
    for k, v in r.storage.kv.values():
        k[1:].fill_(float("nan"))
        v[1:].fill_(float("nan"))


def tol_of(dtype, f32=1e-5, bf16=2e-2):
    return dict(rtol=f32, atol=f32) if dtype == "float32" else dict(rtol=bf16, atol=bf16)


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


class Src:
    """Weights by name for one part."""

    def __init__(self, w, dtype):
        self.w, self.dtype = w, dtype

    def fetch(self, name):
        return self.w[name].to(DT[self.dtype]).cuda()


def plain_ctx(T, uniform=False):
    from mini_sglang_b200.parts.context import StepContext
    return StepContext(T=T, B=1, page_size=1, input_ids=None, positions=None, q_start=None, kv_len=None, token_req=None, slots=None, groups=[],
                       host_q_lens=[T], host_kv_lens=[T], host_slots=[1], uniform_decode=uniform)


# ---------------------------------------------------------------------------------------------------------------------
# kernels alone
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H", [1, 50, 72, 1000, 4100, 9001, 12288])
def test_layer_norm_with_the_sum_in_front(dtype, H):
    from mini_sglang_b200 import ops
    torch.manual_seed(H)
    T = 6
    x = torch.randn(T, H).to(DT[dtype])
    res = torch.randn(T, H) + torch.tensor([0.0, 3.0, -40.0, 100.0, 0.0, 1.0])[:, None]        # rows far from a mean of zero
    w = (1 + 0.1 * torch.randn(H)).to(DT[dtype])
    rows = torch.tensor([4, 0, 3], dtype=torch.int32)
    for x_in in (None, x, x.float()):
        v = res.double() + (x.double() if x_in is not None else 0.0)
        want = pk.layer_norm(v, w.double(), 1e-5)
        r = res.clone().cuda()
        y = ops.rmsnorm(w.cuda(), 1e-5, x=None if x_in is None else x_in.cuda(), residual=r, residual_out=r if x_in is not None else None,
                        out_dtype=DT[dtype], center=True)
        torch.testing.assert_close(r.cpu().double(), v, rtol=1e-6, atol=1e-5)
        torch.testing.assert_close(y.cpu().double(), want, **tol_of(dtype, 5e-5, 1e-2))
        y = ops.rmsnorm(w.cuda(), 1e-5, x=None if x_in is None else x_in.cuda(), residual=res.cuda(), rows=rows.cuda(), out_dtype=DT[dtype], center=True)
        torch.testing.assert_close(y.cpu().double(), want[rows.long()], **tol_of(dtype, 5e-5, 1e-2))
    # the norm without the mean taken off takes a float32 sum too
    y = ops.rmsnorm(w.cuda(), 1e-5, x=x.float().cuda(), residual=res.cuda(), out_dtype=DT[dtype])
    torch.testing.assert_close(y.cpu().double(), pk.rms_unit(res.double() + x.double(), 1e-5) * w.double(), **tol_of(dtype, 5e-5, 1e-2))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("geo", [dict(H=6, G=3, d=40, dv=24), dict(H=1, G=1, d=36, dv=36), dict(H=8, G=2, d=128, dv=128), dict(H=3, G=3, d=10, dv=14),
                                 dict(H=4, G=1, d=16, dv=200), dict(H=2, G=2, d=264, dv=8), dict(H=5, G=5, d=64, dv=256), dict(H=2, G=1, d=16, dv=12, rot=8)])
def test_head_norms_unit_values_and_cache_rows(dtype, geo):
    from mini_sglang_b200 import ops
    H, G, d, dv, rot = (geo.get(k, 0) for k in ("H", "G", "d", "dv", "rot"))
    torch.manual_seed(d)
    T, P, pages = 11, 4, 9
    width = (H + G) * d + G * dv
    proj = torch.randn(T, width + 8).to(DT[dtype])
    proj[3] *= 0.01                                               # eps matters
    qn, kn = 1 + 0.3 * torch.randn(d), 1 + 0.3 * torch.randn(d)
    loc = torch.tensor([4 * 7 + 1, 4 * 2, 4 * 2 + 1, 4 * 2 + 2, 4 * 2 + 3, 4 * 5, 1, 33, 34, 13, 22], dtype=torch.int32)
    kc = torch.zeros(pages, G, P, d, dtype=DT[dtype], device="cuda")
    vc = torch.zeros(pages, G, P, dv, dtype=DT[dtype], device="cuda")
    pos = torch.arange(T, dtype=torch.int32)
    f, mag = pk.frequencies(rot, 100.0, None) if rot else (None, 1.0)
    angles = ops.rotary_angles(pos.cuda(), f.cuda(), mag, T) if rot else None
    q = ops.sink_qkv_prep(proj.cuda(), n_q=H, n_kv=G, d=d, dv=dv, angles=angles, v_first=None, lam=0.0, out_loc=loc.cuda(), k_cache=kc, v_cache=vc,
                          page_size=P, q_norm=qn.cuda(), k_norm=kn.cuda(), v_unit=True, eps=1e-3)
    pd = proj.double()
    wq = pk.rms_unit(pd[:, :H * d].reshape(T, H, d), 1e-3) * qn.double()
    wk = pk.rms_unit(pd[:, H * d:(H + G) * d].reshape(T, G, d), 1e-3) * kn.double()
    wv = pk.rms_unit(pd[:, (H + G) * d:width].reshape(T, G, dv), 1e-3)
    if rot:
        wq, wk = pk.rotate(wq, f, mag), pk.rotate(wk, f, mag)
    torch.testing.assert_close(q.cpu().double(), wq, **tol_of(dtype))
    kt = kc.cpu().double().permute(0, 2, 1, 3).reshape(pages * P, G, d)
    vt = vc.cpu().double().permute(0, 2, 1, 3).reshape(pages * P, G, dv)
    torch.testing.assert_close(kt[loc.long()], wk, **tol_of(dtype))
    torch.testing.assert_close(vt[loc.long()], wv, **tol_of(dtype))
    untouched = torch.ones(pages * P, dtype=torch.bool)
    untouched[loc.long()] = False
    assert kt[untouched].abs().max() == 0 and vt[untouched].abs().max() == 0
    q2 = ops.sink_qkv_prep(proj.cuda(), n_q=H, n_kv=G, d=d, dv=dv, angles=angles, v_first=None, lam=0.0, out_loc=None, k_cache=None, v_cache=None,
                           page_size=P, q_norm=qn.cuda(), k_norm=kn.cuda(), v_unit=True, eps=1e-3)           # a run that writes no cache
    assert torch.equal(q2, q)


def _attention_case(dtype, how, *, H, G, d, dv, P, ctx, n_new, spike, seed, low=0.0, splits=1, wide_table=0, null=0.0, gated=True, window=0):
    """One request with `ctx` cached tokens of which the last `n_new` are the step's queries, through the launches that the mixer
    makes: how = "paged" (the engine's paged attention kernels; head sizes alike), "pair" (the kernels for any pair of head
    sizes, as they are chosen) or "f32" (the float32-arithmetic one of those).  Key `spike` (if not None) stands far above all
    others for every query that may see it, and its value row is a constant that no other row has; `low` moves all scores down.
    Pages lie in a shuffled order, unwritten slots hold NaN.  -> (output [n_new, H, dv], float64 expectation without the gate)."""
    from mini_sglang_b200 import ops
    from mini_sglang_b200.parts.attention import paged_attend
    from mini_sglang_b200.parts.context import GroupContext, KVCacheView, StepContext, Workspace
    g = torch.Generator().manual_seed(seed)
    q = 0.3 * torch.randn(n_new, H, d, generator=g)
    k = 0.3 * torch.randn(ctx, G, d, generator=g)
    v = torch.randn(ctx, G, dv, generator=g)
    q[:, :, 0], k[:, :, 0] = 4.0, -0.625 * low
    if spike is not None:
        q[:, :, 1] = 3.0
        k[spike, :, 1] = 8.0
        v[spike] = 7.0
    gates = torch.randn(n_new, H * dv + 16, generator=g).to(DT[dtype])
    q, k, v = (t.to(DT[dtype]) for t in (q, k, v))
    n_pages = -(-ctx // P)
    order = torch.randperm(n_pages, generator=g) + 1
    kc = torch.full((n_pages + 2, G, P, d), float("nan"), dtype=DT[dtype])
    vc = torch.full((n_pages + 2, G, P, dv), float("nan"), dtype=DT[dtype])
    kc[0], vc[0] = 0, 0
    table = torch.zeros(1, max(n_pages, wide_table), dtype=torch.int32)
    for pg in range(n_pages):
        table[0, pg] = order[pg]
        n = min(P, ctx - pg * P)
        kc[order[pg], :, :n] = k[pg * P: pg * P + n].permute(1, 0, 2)
        vc[order[pg], :, :n] = v[pg * P: pg * P + n].permute(1, 0, 2)
    scale = 0.4
    gate = gates.cuda()[:, 8:8 + H * dv] if gated else None
    uniform = n_new == 1
    kc, vc = kc.cuda(), vc.cuda()
    if how == "paged":
        assert d == dv
        grp = GroupContext(block_table=table.cuda(), out_loc=i32([0] * n_new), nsplit=i32([splits]) if splits > 1 else None, max_split=splits,
                           window=None, host_nsplit=[splits], order=i32([0]) if uniform else None)
        sc = StepContext(T=n_new, B=1, page_size=P, input_ids=None, positions=None, q_start=i32([0, n_new]), kv_len=i32([ctx]),
                         token_req=i32([0] * n_new), slots=i32([1]), groups=[grp], host_q_lens=[n_new], host_kv_lens=[ctx], host_slots=[1],
                         uniform_decode=uniform, workspace=Workspace(torch.device("cuda")))
        out = torch.full((n_new, H, d), float("nan"), dtype=DT[dtype], device="cuda")
        paged_attend(q.cuda(), out, sc, KVCacheView(kc, vc, grp, P), n_q=H, n_kv=G, d=d, window=window, scale=scale, use_mma=ops.mma_supported(d, DT[dtype]),
                     null_log2=torch.full((H,), null * math.log2(math.e), device="cuda"), gate=gate)
        ops.check_kernel_status()
    else:
        out = torch.empty(n_new, H * dv, dtype=DT[dtype], device="cuda")
        ops.sink_attention(q.cuda(), out, kc, vc, q_start=i32([0, n_new]), kv_len=i32([ctx]), block_table=table.cuda(), n_kv=G, page_size=P, scale=scale,
                           softcap=0.0, window=window, sink=torch.full((H,), null, device="cuda"), q_lens=None if (uniform and wide_table) else [n_new],
                           tensor_cores=False if how == "f32" else None, gate=gate)
    got = out.double().cpu().view(n_new, H, dv)
    assert torch.isfinite(got).all()
    qd, kd, vd = q.double(), k.double(), v.double()
    want = torch.zeros(n_new, H, dv, dtype=F64)
    for i in range(n_new):
        p = ctx - n_new + i
        lo = max(0, p - window + 1) if window else 0
        for h in range(H):
            s = (kd[lo:p + 1, h // (H // G)] @ qd[i, h]) * scale
            m = max(float(s.max()), null)
            e = torch.exp(s - m)
            want[i, h] = (e @ vd[lo:p + 1, h // (H // G)]) / (e.sum() + math.exp(null - m))
    gated_want = want * torch.sigmoid(gates.double()[:, 8:8 + H * dv]).view(n_new, H, dv) if gated else want
    tol = dict(rtol=2e-5, atol=2e-5) if dtype == "float32" else dict(rtol=3e-2, atol=3e-2)
    torch.testing.assert_close(got, gated_want, **tol)
    return want


# head sizes of every kernel the paged launches may take: 128 (prompts on tcgen05), multiples of 32 and of 16, float32
PAGED = [("bfloat16", 128, 2, 4), ("bfloat16", 64, 2, 6), ("bfloat16", 48, 1, 3), ("bfloat16", 16, 1, 24), ("bfloat16", 160, 2, 2), ("bfloat16", 256, 1, 8),
         ("float32", 32, 2, 4), ("float32", 40, 1, 2)]


@pytest.mark.parametrize("dtype,d,G,H", PAGED)
@pytest.mark.parametrize("n_new", [1, 2, 13, 150])
def test_paged_attention_with_one_in_the_denominator_and_gates(dtype, d, G, H, n_new):
    """ctx 300: the spike on the first token, far back, on page and tile borders, on the first and the last query itself."""
    ctx, P = 300, 16
    first, last = ctx - n_new, ctx - 1
    places = sorted({0, 57, 127, 128, 255, 256, first, last})
    for spike in places if n_new < 100 else (0, 128, first, last):
        want = _attention_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=P, ctx=ctx, n_new=n_new, spike=spike, seed=spike)
        for i in range(n_new):
            assert (float(want[i].mean()) > 3.5) == (spike <= first + i), (spike, i)
    # scores far below 0: the one takes nearly all the weight; far above: it takes none
    w = _attention_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=P, ctx=ctx, n_new=n_new, spike=None, seed=7, low=12.0)
    assert float(w.abs().max()) < 0.02
    _attention_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=P, ctx=ctx, n_new=n_new, spike=None, seed=8, low=-12.0)
    w0 = _attention_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=P, ctx=ctx, n_new=n_new, spike=None, seed=9, low=6.0, gated=False)
    w1 = _attention_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=P, ctx=ctx, n_new=n_new, spike=None, seed=9, low=6.0, null=2.0)
    assert float((w0 - w1).abs().max()) > 0.4 * float(w0.abs().max())
    _attention_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=P, ctx=n_new, n_new=n_new, spike=0, seed=3)          # the first tokens of a sequence
    _attention_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=P, ctx=ctx, n_new=n_new, spike=first - 40, seed=4, window=41)


@pytest.mark.parametrize("dtype,d,G,H", PAGED)
@pytest.mark.parametrize("splits", [2, 5])
def test_paged_attention_whose_keys_are_cut(dtype, d, G, H, splits):
    """A decoded token and a few tokens whose keys go to several blocks: the one is added once, the gate applied once."""
    for n_new in (1, 2):
        for spike in (0, 160, 161, 400, 799):
            want = _attention_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=8, ctx=800, n_new=n_new, spike=spike, seed=spike, splits=splits)
            assert (float(want[-1].mean()) > 3.5) == (spike <= 799)
        _attention_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=8, ctx=800, n_new=n_new, spike=None, seed=1, low=7.0, splits=splits)


PAIR = [("float32", "pair"), ("bfloat16", "f32"), ("bfloat16", "pair")]


@pytest.mark.parametrize("dtype,how", PAIR)
def test_attention_of_any_pair_of_head_sizes_with_gates(dtype, how):
    cases = [dict(H=6, G=3, d=40, dv=24, P=4, ctx=140, n_new=9, spike=3), dict(H=2, G=2, d=10, dv=14, P=1, ctx=45, n_new=45, spike=0),
             dict(H=16, G=1, d=96, dv=64, P=16, ctx=90, n_new=2, spike=88), dict(H=2, G=1, d=200, dv=131, P=8, ctx=70, n_new=5, spike=41),
             dict(H=4, G=2, d=24, dv=40, P=16, ctx=300, n_new=130, spike=170), dict(H=4, G=2, d=24, dv=40, P=16, ctx=300, n_new=70, spike=None, low=8.0),
             dict(H=80, G=1, d=32, dv=24, P=8, ctx=50, n_new=3, spike=11)]
    for n, c in enumerate(cases):
        _attention_case(dtype, how, seed=n, **c)
    for spike in (0, 255, 256, 767, 768, 999):          # a decoded token over 1,000 keys cut into pieces
        _attention_case(dtype, how, H=4, G=2, d=32, dv=16, P=16, ctx=1000, n_new=1, spike=spike, seed=spike, wide_table=128)
    _attention_case(dtype, how, H=4, G=2, d=32, dv=16, P=16, ctx=1000, n_new=1, spike=None, seed=5, wide_table=128, low=8.0)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("I,K", [(64, 96), (136, 160), (24, 50), (33, 72)])
def test_relu_gated_product_with_biases(dtype, I, K):
    """A few rows (weight streaming), rows between, many rows (tcgen05 in bfloat16); sizes that the fused kernels take and sizes
    that go through the library product and the activation kernel; with and without biases; silu beside relu."""
    from mini_sglang_b200 import ops
    torch.manual_seed(I)
    w, b = torch.randn(2 * I, K) / math.sqrt(K), 0.5 * torch.randn(2 * I)
    w, b = w.to(DT[dtype]), b.to(DT[dtype])
    for T in (1, 7, 8, 40, 256, 300):
        x = torch.randn(T, K).to(DT[dtype])
        for bias in (None, b):
            z = x.double() @ w.double().T + (b.double() if bias is not None else 0.0)
            for act, f in ((ops.ACT_RELU, torch.relu), (ops.ACT_SILU, torch.nn.functional.silu), (ops.ACT_RELU2, lambda t: torch.relu(t) ** 2)):
                got = ops.linear_glu(x.cuda(), w.cuda(), bias.cuda() if bias is not None else None, act)
                torch.testing.assert_close(got.cpu().double(), f(z[:, :I]) * z[:, I:], **tol_of(dtype, 2e-5, 4e-2))
    ops.check_kernel_status()


def _routed(E, ident, top, groups, keep, H, seed, spread=2.0, corr=0.3):
    g = torch.Generator().manual_seed(seed)
    n = E + ident
    return (spread * torch.randn(n, H, generator=g) / math.sqrt(H)).to(torch.bfloat16), corr * torch.randn(n, generator=g)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("geo", [(6, 2, 3, 4, 2), (8, 0, 2, 1, 1), (28, 4, 6, 8, 3), (3, 1, 4, 1, 1), (5, 1, 2, 3, 1), (1, 1, 1, 2, 1), (254, 2, 8, 16, 4)])
def test_softmax_router_over_groups(dtype, geo):
    """Scores are the softmax over all outputs, groups count by their largest choice score, dropped groups lose to any negative
    choice score, weights are the scores as they are."""
    from mini_sglang_b200 import ops
    E, ident, top, count, keep = geo
    H, T = 72, 60
    router, corr = _routed(E, ident, top, count, keep, H, E + top)
    corr[: (E + ident) // 2] -= 0.6                                         # choice scores below 0 among them
    x = torch.randn(T, H, generator=torch.Generator().manual_seed(1)).to(DT[dtype])
    idx, wts = ops.route(x.cuda(), router.to(DT[dtype]).cuda(), corr.cuda(), n_groups=count, keep=keep, top=top, score="softmax", group_score="max",
                         renormalize=False)
    s = torch.softmax(x.double() @ router.double().T, dim=-1)
    clear = 0
    for t in range(T):
        chosen, gap = pk.choose(s[t], corr.double(), count, keep, top)
        if gap < 1e-5:
            continue
        clear += 1
        assert sorted(idx[t].tolist()) == sorted(chosen), t
        torch.testing.assert_close(wts[t].cpu().double(), s[t][idx[t].cpu().long()], rtol=1e-5, atol=1e-7)
    assert clear > 50


def test_router_ties_go_to_the_lower_index():
    from mini_sglang_b200 import ops
    x = torch.ones(2, 16).cuda()
    idx, wts = ops.route(x, torch.zeros(8, 16).cuda(), torch.zeros(8).cuda(), n_groups=4, keep=2, top=3, score="softmax", group_score="max", renormalize=False)
    assert idx.tolist() == [[0, 1, 2]] * 2
    torch.testing.assert_close(wts.cpu(), torch.full((2, 3), 0.125))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("geo", [dict(E=6, ident=2, top=3, groups=(4, 2), F=24, Fs=40), dict(E=2, ident=0, top=1, groups=None, F=16, Fs=0),
                                 dict(E=1, ident=3, top=2, groups=None, F=8, Fs=8), dict(E=14, ident=2, top=5, groups=(8, 3), F=32, Fs=32),
                                 dict(E=3, ident=1, top=2, groups=(2, 2), F=21, Fs=0)])
@pytest.mark.parametrize("T", [1, 9, 150])
def test_plain_experts_both_ways(dtype, geo, T):
    """The few-pairs kernels and the path in expert order, with identity outputs (also tokens that choose nothing else)."""
    from mini_sglang_b200.config.spec import PartSpec
    from mini_sglang_b200.parts import BuildEnv
    from mini_sglang_b200.parts.experts import PlainExperts
    E, ident, top, F, Fs = (geo[k] for k in ("E", "ident", "top", "F", "Fs"))
    count, keep = geo["groups"] or (1, 1)
    H = 48
    g = torch.Generator().manual_seed(E * 7 + T)
    router, corr = _routed(E, ident, top, count, keep, H, E * 7 + T)
    w = {"f.router": router.float(), "f.correction": corr}
    for e in range(E):
        w[f"f.e{e}.up"], w[f"f.e{e}.down"] = torch.randn(F, H, generator=g) / 7, torch.randn(H, F, generator=g) / 5
    if Fs:
        w.update({"f.shared.up": torch.randn(Fs, H, generator=g) / 7, "f.shared.down": torch.randn(H, Fs, generator=g) / 5})
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    c = {"expert": {"ff": F}, "router": {"experts": E, "identity": ident, "top": top}}
    if geo["groups"]:
        c["router"]["groups"] = {"count": count, "keep": keep}
    if Fs:
        c["shared"] = {"ff": Fs}
    part = PlainExperts(PartSpec("plain_experts", {"hidden_size": H, "intermediate_size": F, "activation": "relu2", "num_experts": E, "identity": ident,
                                                   "top": top, "groups": count, "keep_groups": keep, "shared_size": Fs}),
                        "f", BuildEnv(dtype=DT[dtype], device=torch.device("cuda")))
    part.load(Src(w, dtype))
    x = torch.randn(T, H, generator=g).to(DT[dtype])
    margins = []
    want = pk.mixture(x.double(), {k: v.double() for k, v in w.items()}, "f", c, margins)
    clear = margins[0] > 1e-4
    got = part.forward(x.cuda(), plain_ctx(T)).double().cpu()
    assert clear.sum() >= 0.8 * T
    tol = dict(rtol=1e-4, atol=2e-5) if dtype == "float32" else dict(rtol=3e-2, atol=3e-2)
    torch.testing.assert_close(got[clear], want[clear], **tol)
    for t in range(0, T, 50):            # the same rows through the few-pairs kernels, one token at a time, as a decode step has it
        if clear[t]:
            torch.testing.assert_close(part.forward(x[t:t + 1].cuda(), plain_ctx(1, uniform=True)).double().cpu()[0], want[t], **tol)
    if ident >= top and count == 1:      # every token hands its input on and nothing else
        part.correction[:E] -= 10.0
        s = torch.softmax(x.double() @ w["f.router"].double().T, dim=-1)
        choice = s[:, E:] + w["f.correction"].double()[E:]
        order = choice.argsort(dim=1, descending=True)[:, :top]
        best = choice.gather(1, choice.argsort(dim=1, descending=True))
        sure = (best[:, top - 1] - best[:, top]) > 1e-4 if top < ident else torch.ones(T, dtype=torch.bool)
        base = pk.expert(x.double(), {k: v.double() for k, v in w.items()}, "f.shared") if Fs else 0.0
        want = s[:, E:].gather(1, order).sum(1, keepdim=True) * x.double() + base
        torch.testing.assert_close(part.forward(x.cuda(), plain_ctx(T)).double().cpu()[sure], want[sure], **tol)


def test_order_of_pairs_some_of_which_have_no_row():
    from mini_sglang_b200 import ops
    g = torch.Generator().manual_seed(3)
    E, top, T, H = 5, 3, 300, 24
    idx = torch.stack([torch.randperm(E + 2, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    counts, ends, place = (t.cpu() for t in ops.expert_order(idx.cuda(), E))
    flat = idx.reshape(-1)
    assert counts.tolist() == [int((flat == e).sum()) for e in range(E)] and ends.tolist() == counts.cumsum(0).tolist()
    order = sorted((i for i in range(T * top) if flat[i] < E), key=lambda i: (int(flat[i]), i))
    where = {i: n for n, i in enumerate(order)}
    assert place.tolist() == [where.get(i, -1) for i in range(T * top)]
    for dt in (torch.float32, torch.bfloat16):
        h = torch.randn(T, H, generator=g).to(dt)
        rows = ops.expert_gather(h.cuda(), place.cuda(), top).cpu()
        for i, at in enumerate(place.tolist()):
            assert at < 0 or torch.equal(rows[at], h[i // top])
        y, wts, extra = torch.randn(T * top, H, generator=g).to(dt), torch.rand(T, top, generator=g), torch.randn(T, H, generator=g)
        y[ends[-1]:] = float("nan")                        # rows that belong to no pair
        got = ops.expert_combine_self(y.cuda(), place.cuda(), wts.cuda(), h.cuda(), extra=extra.cuda()).cpu()
        want = torch.stack([extra[t].double() + sum(wts[t, k].double() * (y[at] if (at := int(place[t * top + k])) >= 0 else h[t]).double()
                                                    for k in range(top)) for t in range(T)])
        torch.testing.assert_close(got.double(), want, rtol=1e-5, atol=1e-5)


# ---------------------------------------------------------------------------------------------------------------------
# the model through the step function
# ---------------------------------------------------------------------------------------------------------------------
LENGTHS = {"KA": 75, "KB": 41, "KC": 60}


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["KA", "KB", "KC"])
def test_whole_prompt_token_by_token_and_in_portions(name, dtype):
    """The same sequence three ways: one step; five tokens and then one token a step (through the CUDA graph); portions of
    changing sizes down to two tokens.  Every position against the plain implementation."""
    V = CONFIGS_K[name]["vocab"]
    n = LENGTHS[name]
    toks = random_tokens(n, V, 100 + n)
    seqs = {"w": toks, "d": toks, "p": toks}
    r = runner(name, dtype, num_pages=3 * (-(-n // PAGE[name])) + 8)
    poison(r)
    compare(name, dtype, play(r, [{"entries": [("w", toks, list(range(n)))], "end": ["w"]}]), seqs)
    steps = [{"entries": [("d", toks[:5], list(range(5)))]}] + [{"entries": [("d", [t], [0])]} for t in toks[5:]]
    got = play(r, steps)
    assert r.last_step_used_graph
    compare(name, dtype, got, seqs)
    sizes, at, steps = [2, 3, 7, 2, 16, 1, 1, 2, 5, 2, 9], 0, []
    while at < n:
        c = min(sizes[len(steps) % len(sizes)], n - at)
        steps.append({"entries": [("p", toks[at:at + c], list(range(c)))]})
        at += c
    got = play(r, steps)
    compare(name, dtype, got, seqs)
    assert len(got) == n
    r.mgr.check_idle()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["KA", "KC"])
def test_long_prompt_whole_and_in_long_and_short_portions(name, dtype):
    """A prompt in one step (many rows: the products with the activation in their epilogue, the tcgen05 attention at head size
    128), and in long and short portions with a second request's single tokens beside them."""
    V = CONFIGS_K[name]["vocab"]
    n = 331
    toks, other = random_tokens(n, V, 900 + n), random_tokens(9, V, 77)
    seqs = {"w": toks, "p": toks, "o": other}
    r = runner(name, dtype, num_pages=2 * (-(-n // PAGE[name])) + 24)
    poison(r)
    compare(name, dtype, play(r, [{"entries": [("w", toks, list(range(n)))], "end": ["w"]}]), seqs)
    sizes, at, steps = [150, 1, 64, 2, 114], 0, []
    for i, c in enumerate(sizes):
        entries = [("p", toks[at:at + c], list(range(c)))]
        entries.insert(i % 2, ("o", other[i:i + 1], [0]))
        steps.append({"entries": entries})
        at += c
    assert at == n
    got = play(r, steps)
    compare(name, dtype, got, seqs)
    assert len(got) == n + len(sizes)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["KA", "KB", "KC"])
def test_mixed_batches_on_a_small_pool(name, dtype):
    """Five requests of unequal lengths through two request slots and a pool that holds little more than the two longest:
    portions of one beside single tokens of another; pages and block-table rows are used again, and what they held before
    (NaN at the start) must never be read."""
    V = CONFIGS_K[name]["vocab"]
    P = PAGE[name]
    lens = {"a": 50, "b": 23, "c": 1, "d": 66, "e": 34}
    seqs = {k: random_tokens(n, V, 7 + n) for k, n in lens.items()}
    r = runner(name, dtype, num_pages=-(-66 // P) + -(-50 // P) + 1, max_reqs=2)
    poison(r)
    a, b, c, d, e = (seqs[k] for k in "abcde")
    steps = [
        {"entries": [("a", a[:17], [0, 16]), ("b", b[:2], [1])]},
        {"entries": [("b", b[2:3], [0]), ("a", a[17:40], [5, 22])]},
        {"entries": [("a", a[40:41], [0]), ("b", b[3:23], list(range(20)))], "end": ["b"]},
        {"entries": [("c", c, [0]), ("a", a[41:42], [0])], "end": ["c"]},
        {"entries": [("a", a[42:43], [0]), ("d", d[:30], [29])]},
        {"entries": [("d", d[30:60], [0, 29]), ("a", a[43:50], list(range(7)))], "end": ["a"]},
        {"entries": [("d", d[60:61], [0]), ("e", e[:9], [8])]},
        {"entries": [("e", e[9:11], [0, 1]), ("d", d[61:62], [0])]},
    ] + [{"entries": [("d", d[62 + i:63 + i], [0]), ("e", e[11 + i:12 + i], [0])]} for i in range(4)] + [
        {"entries": [("e", e[15:34], [18])], "end": ["d", "e"]},
    ]
    got = play(r, steps)
    compare(name, dtype, got, seqs)
    r.mgr.check_idle()


@pytest.mark.parametrize("name", ["KA", "KC"])
def test_a_batch_equals_each_request_alone(name):
    """float32: the logits of requests fed together in unequal portions equal those of each alone, to rounding."""
    V = CONFIGS_K[name]["vocab"]
    lens = {"a": 70, "b": 3, "c": 41}
    seqs = {k: random_tokens(n, V, 60 + n) for k, n in lens.items()}
    r = runner(name, "float32", num_pages=3 * (-(-80 // PAGE[name])) + 4)
    together = play(r, [{"entries": [("a", seqs["a"][:33], list(range(33))), ("b", seqs["b"][:2], [0, 1]), ("c", seqs["c"][:40], list(range(40)))]},
                        {"entries": [("c", seqs["c"][40:], [0]), ("a", seqs["a"][33:], list(range(37))), ("b", seqs["b"][2:], [0])]}])
    for rid, toks in seqs.items():
        alone = play(r, [{"entries": [(rid, toks, list(range(len(toks))))]}])
        for k, row in alone.items():
            torch.testing.assert_close(together[k], row, rtol=1e-4, atol=2e-4)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["KA", "KC"])
def test_long_decoding(name, dtype):
    """Two requests decode together for 330 steps through the CUDA graph, past the point where a decoded token's keys are cut
    into pieces; a third joins late with a portion and leaves early."""
    V = CONFIGS_K[name]["vocab"]
    a, b, c = random_tokens(345, V, 1), random_tokens(352, V, 2), random_tokens(30, V, 3)
    seqs = {"a": a, "b": b, "c": c}
    r = runner(name, dtype, num_pages=-(-800 // PAGE[name]) + 4, max_reqs=3)
    poison(r)
    steps = [{"entries": [("a", a[:10], [9]), ("b", b[:20], [19])]}]
    for i in range(330):
        es = [("a", [a[10 + i]], [0]), ("b", [b[20 + i]], [0])]
        if i == 200:
            es.append(("c", c[:26], [25]))
        elif 200 < i <= 204:
            es.append(("c", [c[25 + i - 200]], [0]))
        steps.append({"entries": es, "end": ["c"] if i == 204 else []})
    got = play(r, steps)
    assert r.last_step_used_graph
    compare(name, dtype, got, seqs)
    r.mgr.check_idle()


@pytest.mark.parametrize("fields_on_device", [True, False])
def test_every_geometry_of_a_cache_group_has_kv_splits_of_its_own(fields_on_device):
    """Four caches of one group (one block table) differ in kv heads, query heads and row size: each has its keys cut for its
    own launches, by a decode step through the graph and by a step of short portions; the fields made on the device are the
    host's."""
    name = "KC"
    V = CONFIGS_K[name]["vocab"]
    n = 520
    a, b = random_tokens(n, V, 4), random_tokens(30, V, 9)
    r = runner(name, "bfloat16", num_pages=48, max_reqs=2, page_size=16)
    assert len(r.mgr.groups) == 1 and len(r._plan_group) == 4 and len(set(r._group_geom)) == 4
    r.device_meta = fields_on_device
    poison(r)
    checked = []
    inner = r._meta_on_device

    def checking(gr, entries, starts, nsplits, bucket, even_cuts=None):
        inner(gr, entries, starts, nsplits, bucket, even_cuts)
        lay = gr.layout
        want = np.zeros(lay.size, dtype=np.int32)
        r._fill(want, lay, entries, starts, list(range(bucket)), nsplits, even_cuts=even_cuts)
        have = gr.dev.cpu().numpy()
        B = len(entries)
        for p in range(4):
            for off, m in ((lay.nsplit[p], bucket), (lay.order[p], bucket), (lay.out_loc[p], B), (lay.kv_len, B)):
                assert (have[off:off + m] == want[off:off + m]).all()
            mp = lay.max_pages[p]
            for row, e in enumerate(entries):
                held = int(r.mgr.groups[0].n_pages[e.slot])
                o = lay.table[p] + row * mp
                assert (have[o:o + held] == want[o:o + held]).all()
        checked.append([list(ns) for ns in nsplits])

    r._meta_on_device = checking
    steps, at = [{"entries": [("a", a[:480], [0, 479])]}], 480
    for i, c in enumerate((3, 2, 1, 1, 8, 2, 1, 5, 1, 1, 1, 3, 6, 1, 4)):
        es = [("a", a[at:at + c], list(range(c)))]
        if i >= 3:
            es.append(("b", [b[i - 3]], [0]))
        steps.append({"entries": es})
        at += c
    assert at == n
    got = play(r, steps)
    compare(name, "bfloat16", got, {"a": a, "b": b})
    plans = [max(ns) for ns in r.last_plan["nsplits"]]
    assert max(plans) > 1 and len(r.last_plan["nsplits"]) == 4
    assert bool(checked) == fields_on_device
    # of many long requests the geometries' keys are cut differently: more blocks a request where there are fewer kv heads
    cuts = [r._plan_splits(p, [1] * 24, [4096] * 24, 16)[0] for p in range(4)]
    assert cuts[0] < max(cuts[1:]), cuts
    r.mgr.check_idle()


@pytest.mark.parametrize("dtype", BOTH)
def test_other_page_sizes(dtype):
    """Pages of one token and pages wider than a request, the same two ways."""
    for name, P in (("KA", 1), ("KB", 64), ("KC", 2), ("KC", 8), ("KA", 64)):
        V = CONFIGS_K[name]["vocab"]
        toks, other = random_tokens(45, V, 31), random_tokens(20, V, 32)
        seqs = {"w": toks, "p": toks, "o": other}
        r = runner(name, dtype, num_pages=3 * (-(-45 // P)) + 4, page_size=P)
        poison(r)
        got = play(r, [{"entries": [("w", toks, list(range(45)))], "end": ["w"]}])
        steps = [{"entries": [("p", toks[:2], [0, 1]), ("o", other[:11], [10])]}]
        steps += [{"entries": [("p", toks[2 + 5 * i:7 + 5 * i], list(range(5))), ("o", [other[11 + i]], [0])]} for i in range(8)]
        steps += [{"entries": [("p", toks[42:45], [0, 1, 2]), ("o", [other[19]], [0])]}]
        got.update(play(r, steps))
        compare(name, dtype, got, seqs)
        r.mgr.check_idle()


@pytest.mark.parametrize("seed", range(8))
def test_random_configurations(seed):
    """Whole, token by token and in portions beside another request's single tokens, float32 (the logic) and bfloat16."""
    from mini_sglang_b200.engine.step import ModelRunner
    cfg = random_config(seed)
    w = make_weights(cfg, 100 + seed)
    path = write_model_dir(os.path.join(_tmp.name, f"random{seed}"), cfg, w)
    V = cfg["vocab"]
    toks, other = random_tokens(100, V, seed), random_tokens(40, V, 50 + seed)
    ref = {"w": plain_of(cfg, w, toks), "o": plain_of(cfg, w, other)}
    ref["d"] = ref["p"] = ref["w"]
    P = [1, 4, 16, 8][seed % 4]
    for dtype in BOTH:
        r = ModelRunner.from_model_dir(path, dtype=dtype, page_size=P, num_pages=3 * (-(-100 // P)) + 6, max_reqs=2, max_context_len=128)
        poison(r)
        got = play(r, [{"entries": [("w", toks, list(range(100)))], "end": ["w"]}])
        steps = [{"entries": [("d", toks[:3], [0, 1, 2])]}] + [{"entries": [("d", [t], [0])]} for t in toks[3:]]
        got.update(play(r, steps))
        steps = [{"entries": [("o", other[:9], [8]), ("p", toks[:2], [0, 1])]}]
        steps += [{"entries": [("p", toks[2 + 4 * i:6 + 4 * i], [0, 1, 2, 3]), ("o", [other[9 + i]], [0])]} for i in range(24)]
        steps += [{"entries": [("p", toks[98:100], [0, 1])]}]
        got.update(play(r, steps))
        compare(f"random {seed}", dtype, got, None, ref=ref, bound=0.05 if dtype == "bfloat16" else None, min_firm=0.0, close=0.04)
        r.mgr.check_idle()


@functools.lru_cache(None)
def _wide():
    """Three layers whose sizes the serving kernels take: head size 128 on 4 kv heads, latent rows of 128 and 256, a feed-forward
    whose product has the activation in its epilogue, experts in multiples of 8."""
    cfg = tk.model(256, 200, 1e-5, [
        tk.layer(tk.att(16, 4, 128, 128), tk.dense(512)),
        tk.layer(tk.latent(8, 64, 32, 64, 96, scaling=tk.RAMP), tk.moe(6, 3, 64, identity=2, groups=(2, 1), shared=64)),
        tk.layer(tk.latent(4, 96, 64, 96, 192, base=50000.0), tk.dense(256)),
    ])
    w = make_weights(cfg, 21)
    path = write_model_dir(os.path.join(_tmp.name, "wide"), cfg, w)
    toks = random_tokens(620, 200, 8)
    return cfg, w, path, toks, plain_of(cfg, w, toks)


@pytest.mark.parametrize("dtype", BOTH)
def test_layers_at_serving_sizes(dtype):
    """A 300-token prompt, a 270-token portion behind it, short portions, then decoding through the graph."""
    from mini_sglang_b200.engine.step import ModelRunner
    cfg, w, path, toks, ref = _wide()
    r = ModelRunner.from_model_dir(path, dtype=dtype, page_size=16, num_pages=48, max_reqs=2, max_context_len=1024)
    poison(r)
    steps, at = [], 0
    for c in (300, 270, 2, 9, 3):
        steps.append({"entries": [("a", toks[at:at + c], list(range(0, c, 7)) + [c - 1])]})
        at += c
    steps += [{"entries": [("a", [t], [0])]} for t in toks[at:]]
    got = play(r, steps)
    assert r.last_step_used_graph and max(max(ns) for ns in r.last_plan["nsplits"]) > 1
    compare("wide", dtype, got, None, ref={"a": ref})


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("kinds", ["attention only", "latent only", "one layer without feed-forward"])
def test_models_of_one_kind_of_layer(kinds, dtype):
    """Through the step function (the attention-only model's decode steps may deal the keys of requests of unlike length out
    evenly) and through the entry point."""
    from mini_sglang_b200 import Engine, EngineArgs
    from mini_sglang_b200.engine.step import ModelRunner
    cfg = {"attention only": tk.model(64, 90, 1e-5, [tk.layer(tk.att(4, 2, 64, 64), tk.dense(24)), tk.layer(tk.att(8, 2, 64, 64), None)]),
           "latent only": tk.model(48, 70, 1e-5, [tk.layer(tk.latent(3, 16, 8, 16, 24, scaling=tk.RAMP), tk.moe(3, 2, 16, identity=1))]),
           "one layer without feed-forward": tk.model(40, 50, 1e-6, [tk.layer(tk.att(2, 2, 12, 20), None)])}[kinds]
    w = make_weights(cfg, 31)
    path = write_model_dir(os.path.join(_tmp.name, kinds.replace(" ", "_")), cfg, w)
    V = cfg["vocab"]
    lens = {"a": 2600, "b": 500, "c": 90} if kinds == "attention only" else {"a": 60, "b": 31, "c": 9}
    seqs = {k: random_tokens(n + 4, V, n) for k, n in lens.items()}
    ref = {k: plain_of(cfg, w, t) for k, t in seqs.items()}
    r = ModelRunner.from_model_dir(path, dtype=dtype, page_size=16, num_pages=208, max_reqs=3, max_context_len=4096)
    poison(r)
    steps = [{"entries": [(k, seqs[k][:n], [0, n - 1])]} for k, n in lens.items()]
    steps += [{"entries": [(k, [seqs[k][n + i]], [0]) for k, n in lens.items()]} for i in range(4)]
    got = play(r, steps)
    assert r.last_step_used_graph
    if kinds == "attention only" and dtype == "bfloat16":
        assert r.last_plan["graph_key"][2] == "even"
    compare(kinds, dtype, got, None, ref=ref, min_firm=0.0)
    eng = Engine(EngineArgs(model=path, dtype=dtype, page_size=4, num_pages=32, max_num_reqs=2, random_seed=0, max_context_len=64, log_level="WARNING"))
    prompts = [random_tokens(n, V, 3 + n) for n in (4, 17)]
    outs = eng.generate(input_ids=prompts, sampling_params={"temperature": 0.0, "max_new_tokens": 6, "ignore_eos": True})
    for p, o in zip(prompts, outs):
        if dtype == "float32":
            assert o["token_ids"] == pk.greedy_generate(cfg, w, p, 6)
    eng.scheduler.check_idle_invariants()


def _holds(cfg, w, prompt, got, dtype):
    if dtype == "float32":
        assert got == pk.greedy_generate(cfg, w, prompt, len(got))
        return
    toks = list(prompt)
    for t in got:           # bfloat16 may take another of two nearly equal logits, or another expert at a router's close call
        rows, margin = plain_of(cfg, w, toks)
        row = rows[-1]
        shaky = bool((margin[-FADE - 1:] < CLOSE_CALL).any())
        assert float(row.max() - row[t]) < (0.6 if shaky else 0.05) * float(row.std()) + 0.05
        toks.append(t)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["KA", "KC"])
def test_greedy_generation_through_the_entry_point(name, dtype):
    """Engine.generate with the scheduler: prompts of unequal lengths, portions of at most 16 tokens, a small pool; then prompts that
    share their first 24 tokens with one already served (the model keeps keys only, so the prefix tree serves them)."""
    from mini_sglang_b200 import Engine, EngineArgs
    cfg = CONFIGS_K[name]
    prompts = [random_tokens(n, cfg["vocab"], 50 + n) for n in (5, 47, 18)]
    eng = Engine(EngineArgs(model=model_dir(name), dtype=dtype, page_size=4, num_pages=64, max_num_reqs=3, random_seed=0, chunk_size=16,
                            max_context_len=256, log_level="WARNING"))
    params = {"temperature": 0.0, "max_new_tokens": 10, "ignore_eos": True}
    for p, o in zip(prompts, eng.generate(input_ids=prompts, sampling_params=params)):
        assert len(o["token_ids"]) == 10
        _holds(cfg, weights(name), p, o["token_ids"], dtype)
    again = [prompts[1][:24] + random_tokens(n, cfg["vocab"], 90 + n) for n in (3, 9)]
    for p, o in zip(again, eng.generate(input_ids=again, sampling_params=params)):
        _holds(cfg, weights(name), p, o["token_ids"], dtype)
    eng.scheduler.check_idle_invariants()


def test_trace_replay_program(tmp_path):
    name = "KB"
    V = CONFIGS_K[name]["vocab"]
    a, b = random_tokens(37, V, 1), random_tokens(21, V, 2)
    lines = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [0, 19]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[20:35], "want": []}, {"id": "b", "tokens": b[:21], "want": [20]}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": a[35:36], "want": [0]}], "end": []},
        {"step": 3, "entries": [{"id": "a", "tokens": a[36:37], "want": [0]}], "end": ["a"]},
    ]
    for dtype in BOTH:
        out = tmp_path / dtype
        proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", model_dir(name), "--dtype", dtype,
                               "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(l) for l in lines) + "\n",
                              capture_output=True, text=True, timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [l for l in proc.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(4)]
        rd = lambda i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, V))        # noqa: E731
        got = {("a", 0): rd(0)[0], ("a", 19): rd(0)[1], ("b", 20): rd(1)[0], ("a", 35): rd(2)[0], ("a", 36): rd(3)[0]}
        assert rd(0).shape == (2, V) and rd(1).shape == (1, V) and rd(2).shape == (1, V) and rd(3).shape == (1, V)
        compare(name, dtype, got, {"a": a, "b": b})
