"""The Rubulix parts and the whole model in the engine against the plain implementation (tests/plain_rubulix.py).

Kernels one by one; the attention within chunks and the attention whose heads are the difference of two maps through every kernel
that may run them, with inputs made so that a fault shows (one key whose score stands far above hundreds of others: on both sides
of a chunk's edge, far away, page and tile borders, the borders of the pieces a decoded token's keys are cut into, the token
itself; in one map of a head and not in the other); then the model through the step function: whole prompts, token by token, in
portions down to two tokens, mixed batches on a pool so small that pages and request slots are used again, long decoding, greedy
generation through the engine's entry point, and the trace replay program.
"""

import functools
import json
import os
import subprocess
import sys
import tempfile

import numpy as np
import pytest
import torch

import plain_rubulix as pr
import tiny_rubulix as tr
from helpers import play
from tiny_models import random_tokens, write_model_dir
from tiny_rubulix import CONFIGS_R, make_weights, random_config

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
SEED = {"RA": 3, "RB": 4, "RC": 3}
PAGE = {"RA": 4, "RB": 1, "RC": 16}
_tmp = tempfile.TemporaryDirectory(prefix="msgl_rubulix_")
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64
BOTH = ["float32", "bfloat16"]


@functools.lru_cache(None)
def weights(name):
    return make_weights(CONFIGS_R[name], SEED[name])


@functools.lru_cache(None)
def model_dir(name):
    return write_model_dir(os.path.join(_tmp.name, name), CONFIGS_R[name], weights(name))


def plain_of(cfg, w, tokens):
    with torch.no_grad():
        return pr.forward_sequence(cfg, w, list(tokens), dtype=F64).float()


@functools.lru_cache(None)
def _plain_run(name, tokens):
    return plain_of(CONFIGS_R[name], weights(name), tokens)


def runner(name, dtype, num_pages, max_reqs=4, page_size=None, graphs=True, ctx=1024):
    from mini_sglang_b200.engine.step import ModelRunner
    return ModelRunner.from_model_dir(model_dir(name), dtype=dtype, page_size=page_size or PAGE[name], num_pages=num_pages,
                                      max_reqs=max_reqs, max_context_len=ctx, use_cuda_graph=graphs)


# The reference is the plain implementation in double precision.  float32 rows are held to 2e-4 of a row's rms (6 times that for
# the largest element); bfloat16 rows (projections, cached keys and values and the activations between kernels rounded to 8
# mantissa bits; scores, softmax, norms and the copies of the stream float32) to 8 % (a difference of maps that nearly cancels is
# normed up, and with it the rounding of what it is made of), but for a tenth of a request's rows, which may lie in the noise's
# tail, none by more than TAIL_FACTOR times.  The faults of tests/test_rubulix_cpu.py move some row by 30 % or more.
F32_RMS_FRACTION = 2e-4
BF16_RMS_FRACTION_R = 0.08
TAIL_SHARE, TAIL_FACTOR = 0.1, 2.0


def row_close(row, want, bound):
    row, want = row.float(), want.float()
    assert torch.isfinite(row).all(), "logits are not finite"
    err = row - want
    scale = want.pow(2).mean().sqrt().item()
    rms, worst = err.pow(2).mean().sqrt().item(), err.abs().max().item()
    assert rms <= bound * scale, f"rms error {rms:.4g} is {rms / scale:.4%} of the row's rms {scale:.4g}"
    assert worst <= 6.0 * bound * scale, f"largest error {worst:.4g} is {worst / scale:.4%} of the row's rms {scale:.4g}"


def compare(name, dtype, got, seqs, ref=None, bound=None):
    """Every row against the plain implementation."""
    assert got
    if bound is None:
        bound = F32_RMS_FRACTION if dtype == "float32" else BF16_RMS_FRACTION_R
    over = {}
    for (rid, pos), row in sorted(got.items()):
        want = (ref[rid] if ref is not None else _plain_run(name, tuple(seqs[rid])))[pos]
        try:
            row_close(row, want, bound)
        except AssertionError as e:
            if dtype == "bfloat16":
                try:
                    row_close(row, want, TAIL_FACTOR * bound)
                    over.setdefault(rid, []).append(pos)
                    continue
                except AssertionError:
                    pass
            raise AssertionError(f"request {rid!r} position {pos} ({dtype}, {name}): {e}") from None
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


# ---------------------------------------------------------------------------------------------------------------------
# kernels alone
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,T", [(1, 5), (50, 5), (72, 5), (1000, 5), (1024, 32), (2056, 5), (4096, 5), (4096, 33), (8192, 3), (8200, 5), (12288, 5)])
def test_copies_of_the_stream(dtype, H, T):
    """Update, read and norm in one kernel: 1 to 6 copies (the forms with the row in registers, in one block or over a cluster where
    the rows are few, and the general one), a layer norm with a bias and an RMS norm without, the copies still one row or apart,
    updated in place, or only the wanted rows read."""
    from mini_sglang_b200 import ops
    torch.manual_seed(H)
    w, b = (1 + 0.1 * torch.randn(H)).cuda(), (0.3 * torch.randn(H)).cuda()
    rows = i32([T - 1, 0, 2])
    for S in (1, 2, 3, 4, 6):
        X = torch.randn(T, S, H)
        X[1:3] += torch.tensor([3.0, -40.0])[:, None, None]          # rows far from a mean of zero
        y = torch.randn(T, H).to(DT[dtype])
        c_in, mix, c_out = torch.randn(S), torch.randn(S, S), torch.randn(S)

        def norm(u, center, bias):
            bias = b.double().cpu() if bias is not None else 0.0
            return pr.layer_norm(u, w.double().cpu(), bias, 1e-5) if center else pr.rms_unit(u, 1e-5) * w.double().cpu() + bias

        for center, bias in ((True, b), (False, None)):
            for apart in (True, False):
                x0 = X if apart else X[:, 0].contiguous()
                Xd = (X if apart else X[:, :1].expand(T, S, H)).double()
                kw = dict(streams=S, weight=w, bias=bias, eps=1e-5, center=center, out_dtype=DT[dtype])
                got = ops.stream_mix_norm(x0.cuda(), w_in=c_in.cuda(), **kw)
                torch.testing.assert_close(got.cpu().double(), norm(pr.read_streams(Xd, c_in.double()), center, bias), **tol_of(dtype, 2e-4, 2e-2))
                for yy in (y, y.float()):
                    new = pr.write_streams(Xd, y.double(), mix.double(), c_out.double())
                    upd = dict(y=yy.cuda(), mix=mix.cuda(), w_out=c_out.cuda())
                    x = x0.cuda()
                    x_out = x if apart else torch.full((T, S, H), float("nan"), device="cuda")
                    got = ops.stream_mix_norm(x, w_in=c_in.cuda(), x_out=x_out, **upd, **kw)
                    torch.testing.assert_close(x_out.cpu().double(), new, rtol=1e-5, atol=1e-4)
                    torch.testing.assert_close(got.cpu().double(), norm(pr.read_streams(new, c_in.double()), center, bias), **tol_of(dtype, 2e-4, 2e-2))
                    got = ops.stream_mix_norm(x0.cuda(), w_in=None, rows=rows, **upd, **kw)               # the end of a model
                    torch.testing.assert_close(got.cpu().double(), norm(new.sum(1), center, bias)[rows.cpu().long()], **tol_of(dtype, 2e-4, 2e-2))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H", [1, 72, 1001, 4096])
def test_norms_with_a_bias(dtype, H):
    from mini_sglang_b200 import ops
    torch.manual_seed(H)
    x, res, w, b = torch.randn(6, H).to(DT[dtype]), torch.randn(6, H) + 5.0, (1 + 0.1 * torch.randn(H)).to(DT[dtype]), torch.randn(H)
    v = res.double() + x.double()
    for center, want in ((True, pr.layer_norm(v, w.double(), b.double(), 1e-5)), (False, pr.rms_unit(v, 1e-5) * w.double() + b.double())):
        r = res.clone().cuda()
        y = ops.rmsnorm(w.cuda(), 1e-5, x=x.cuda(), residual=r, residual_out=r, out_dtype=DT[dtype], center=center, bias=b.cuda())
        torch.testing.assert_close(y.cpu().double(), want, **tol_of(dtype, 5e-5, 2e-2))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("geo", [dict(H=6, G=3, d=40, dv=24, rot=24), dict(H=1, G=1, d=36, dv=36, rot=36), dict(H=4, G=2, d=64, dv=128, rot=64, maps=2),
                                 dict(H=8, G=2, d=128, dv=128, rot=2), dict(H=3, G=3, d=7, dv=9, rot=6, maps=2), dict(H=2, G=2, d=264, dv=8, rot=10),
                                 dict(H=5, G=5, d=16, dv=200, rot=16, maps=3), dict(H=2, G=1, d=16, dv=12, rot=0, maps=2), dict(H=24, G=1, d=16, dv=32, rot=12, maps=2)])
def test_pairs_turned_unit_heads_and_rows_of_several_maps(dtype, geo):
    """q, k and v of the packed projection: neighbouring pairs turned by the positions' angles (also where a lane's share holds turned
    and unturned pairs), unit root mean square after it, vectors of a head side by side in the cache rows and alone in their
    place of the query rows."""
    from mini_sglang_b200 import ops
    H, G, d, dv, rot, M = (geo.get(k, 1) for k in ("H", "G", "d", "dv", "rot", "maps"))
    torch.manual_seed(d)
    T, P, pages = 11, 4, 9
    width = (H + G) * M * d + G * dv
    proj = torch.randn(T, width + 8).to(DT[dtype])
    proj[3] *= 0.01                                               # eps matters
    loc = torch.tensor([4 * 7 + 1, 4 * 2, 4 * 2 + 1, 4 * 2 + 2, 4 * 2 + 3, 4 * 5, 1, 33, 34, 13, 22], dtype=torch.int32)
    f, mag = pr.frequencies(rot, 100.0, tr.RAMP) if rot else ([], 1.0)
    angles = ops.rotary_angles(torch.arange(T, dtype=torch.int32).cuda(), torch.tensor(f, dtype=F64).cuda(), mag, T) if rot else None
    pd = proj.double()
    for unit in (True, False):
        kc = torch.zeros(pages, G, P, M * d, dtype=DT[dtype], device="cuda")
        vc = torch.zeros(pages, G, P, dv, dtype=DT[dtype], device="cuda")
        kw = dict(n_q=H, n_kv=G, d=d, dv=dv, angles=angles, v_first=None, lam=0.0, page_size=P, eps=1e-3, interleaved=True, qk_unit=unit, maps=M)
        q = ops.sink_qkv_prep(proj.cuda(), out_loc=loc.cuda(), k_cache=kc, v_cache=vc, **kw)
        norm = (lambda x: pr.rms_unit(x, 1e-3)) if unit else (lambda x: x)
        wq = norm(pr.rotate_neighbours(pd[:, :H * M * d].reshape(T, H, M, d), f, mag))
        wk = norm(pr.rotate_neighbours(pd[:, H * M * d:(H + G) * M * d].reshape(T, G, M, d), f, mag))
        assert q.shape == (T, H * M, M * d)
        place = q.cpu().double().view(T, H, M, M, d)
        for m in range(M):
            torch.testing.assert_close(place[:, :, m, m], wq[:, :, m], **tol_of(dtype))
            assert all(place[:, :, m, o].abs().max() == 0 for o in range(M) if o != m)
        kt = kc.cpu().double().permute(0, 2, 1, 3).reshape(pages * P, G, M, d)
        vt = vc.cpu().double().permute(0, 2, 1, 3).reshape(pages * P, G, dv)
        torch.testing.assert_close(kt[loc.long()], wk, **tol_of(dtype))
        torch.testing.assert_close(vt[loc.long()], pd[:, (H + G) * M * d:width].reshape(T, G, dv), **tol_of(dtype))
        untouched = torch.ones(pages * P, dtype=torch.bool)
        untouched[loc.long()] = False
        assert kt[untouched].abs().max() == 0 and vt[untouched].abs().max() == 0
        q2 = ops.sink_qkv_prep(proj[:, :H * M * d].contiguous().cuda(), out_loc=None, k_cache=None, v_cache=None, **kw)      # only queries
        torch.testing.assert_close(q2, q, rtol=0, atol=0)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,dv", [(1, 9), (3, 32), (5, 96), (2, 130), (4, 512)])
def test_difference_of_maps_alone(dtype, H, dv):
    from mini_sglang_b200 import ops
    torch.manual_seed(dv)
    a = torch.randn(13, 2 * H, dv).to(DT[dtype])
    a[4] *= 0.001
    want = pr.rms_unit(a[:, 0::2].double() - 0.7 * a[:, 1::2].double(), 1e-3) * 0.6
    out = torch.full((13, H * dv), float("nan"), dtype=DT[dtype], device="cuda")
    ops.map_difference(a.cuda(), out, heads=H, lam=0.7, eps=1e-3, scale=0.6)
    torch.testing.assert_close(out.cpu().double().view(13, H, dv), want, **tol_of(dtype))


class Case:
    """One request with `ctx` cached tokens of which the last `n_new` are the step's queries.  Key rows of `maps` vectors of `d`
    elements, value rows of `dv`; pages in a shuffled order, unwritten slots and (with a chunk) the pages before the first chunk
    that is seen hold NaN, as after the cache manager has given them back (their table entries are 0)."""

    def __init__(self, dtype, *, H, G, d, dv, P, ctx, n_new, seed, maps=1, chunk=0, spike=None, spike_map=0):
        g = torch.Generator().manual_seed(seed)
        self.dtype, self.H, self.G, self.d, self.dv, self.P, self.ctx, self.n, self.maps, self.chunk = dtype, H, G, d, dv, P, ctx, n_new, maps, chunk
        q = 0.3 * torch.randn(n_new, H, maps, d, generator=g)
        k = 0.3 * torch.randn(ctx, G, maps, d, generator=g)
        v = torch.randn(ctx, G, dv, generator=g)
        if spike is not None:
            q[:, :, spike_map, 1] = 3.0
            k[spike, :, spike_map, 1] = 9.0
            v[spike] = 7.0 * torch.linspace(0.5, 1.5, dv)
        self.q, self.k, self.v = (t.to(DT[dtype]) for t in (q, k, v))
        n_pages = -(-ctx // P)
        order = torch.randperm(n_pages, generator=g) + 1
        kc = torch.full((n_pages + 2, G, P, maps * d), float("nan"), dtype=DT[dtype])
        vc = torch.full((n_pages + 2, G, P, dv), float("nan"), dtype=DT[dtype])
        kc[0], vc[0] = 0, 0
        table = torch.zeros(1, n_pages, dtype=torch.int32)
        first = ctx - n_new
        gone = (first - first % chunk) // P if chunk else 0
        for pg in range(gone, n_pages):
            table[0, pg] = order[pg]
            m = min(P, ctx - pg * P)
            kc[order[pg], :, :m] = self.k[pg * P: pg * P + m].reshape(m, G, maps * d).permute(1, 0, 2)
            vc[order[pg], :, :m] = self.v[pg * P: pg * P + m].permute(1, 0, 2)
        self.kc, self.vc, self.table = kc.cuda(), vc.cuda(), table.cuda()
        self.gates = torch.randn(n_new, H * dv + 16, generator=g).to(DT[dtype])
        self.scale = 0.4

    def query_rows(self):
        """[n, H * maps, maps * d]: a head's vectors in their places, zeros beside them."""
        rows = torch.zeros(self.n, self.H, self.maps, self.maps, self.d, dtype=DT[self.dtype])
        for m in range(self.maps):
            rows[:, :, m, m] = self.q[:, :, m]
        return rows.view(self.n, self.H * self.maps, self.maps * self.d).cuda()

    def expected(self):
        """-> the maps' outputs [maps, n, H, dv] in double precision."""
        out = torch.zeros(self.maps, self.n, self.H, self.dv, dtype=F64)
        for i in range(self.n):
            p = self.ctx - self.n + i
            lo = p - p % self.chunk if self.chunk else 0
            for h in range(self.H):
                gk = h // (self.H // self.G)
                for m in range(self.maps):
                    s = self.k[lo:p + 1, gk, m].double() @ self.q[i, h, m].double() * self.scale
                    out[m, i, h] = torch.softmax(s, 0) @ self.v[lo:p + 1, gk].double()
        return out

    def context(self, splits):
        from mini_sglang_b200.parts.context import GroupContext, KVCacheView, StepContext, Workspace
        uniform = self.n == 1
        grp = GroupContext(block_table=self.table, out_loc=i32([0] * self.n), nsplit=i32([splits]) if splits > 1 else None, max_split=splits,
                           window=None, chunk=self.chunk or None, host_nsplit=[splits], order=i32([0]) if uniform else None)
        sc = StepContext(T=self.n, B=1, page_size=self.P, input_ids=None, positions=None, q_start=i32([0, self.n]), kv_len=i32([self.ctx]),
                         token_req=i32([0] * self.n), slots=i32([1]), groups=[grp], host_q_lens=[self.n], host_kv_lens=[self.ctx], host_slots=[1],
                         uniform_decode=uniform, workspace=Workspace(torch.device("cuda")))
        return sc, KVCacheView(self.kc, self.vc, grp, self.P)

    def run(self, how, *, splits=1, gated=False, diff=None):
        """how: "paged" (the engine's paged attention kernels), "pair" (the kernels for any pair of head sizes, as they are chosen) or
        "f32" (the float32-arithmetic one of those) -> [n, H (* maps), dv]."""
        from mini_sglang_b200 import ops
        from mini_sglang_b200.parts.attention import paged_attend
        q, n_q, D = self.query_rows(), self.H * self.maps, self.maps * self.d
        gate = self.gates.cuda()[:, 8:8 + self.H * self.dv] if gated else None
        if how == "paged":
            sc, view = self.context(splits)
            out = torch.full((self.n, self.H if diff is not None else n_q, self.dv), float("nan"), dtype=DT[self.dtype], device="cuda")
            paged_attend(q, out, sc, view, n_q=n_q, n_kv=self.G, d=D, window=0, scale=self.scale, use_mma=ops.mma_supported(D, DT[self.dtype]),
                         gate=gate, chunk=self.chunk, diff=diff)
            ops.check_kernel_status()
        else:
            out = torch.empty(self.n, n_q * self.dv, dtype=DT[self.dtype], device="cuda")
            ops.sink_attention(q, out, self.kc, self.vc, q_start=i32([0, self.n]), kv_len=i32([self.ctx]), block_table=self.table, n_kv=self.G,
                               page_size=self.P, scale=self.scale, softcap=0.0, window=0, sink=None, q_lens=None if splits > 1 else [self.n],
                               tensor_cores=False if how == "f32" else None, gate=gate, chunk=self.chunk)
            if diff is not None:
                joined = torch.empty(self.n, self.H * self.dv, dtype=DT[self.dtype], device="cuda")
                ops.map_difference(out.view(self.n, n_q, self.dv), joined, heads=self.H, lam=diff[0], eps=diff[1], scale=diff[2])
                out = joined
        got = out.double().cpu().view(self.n, -1, self.dv)
        assert torch.isfinite(got).all()
        return got

    def tol(self):
        return dict(rtol=2e-5, atol=2e-5) if self.dtype == "float32" else dict(rtol=3e-2, atol=3e-2)


def _chunk_case(dtype, how, *, H, G, d, dv, P, ctx, n_new, chunk, spike, seed, splits=1):
    c = Case(dtype, H=H, G=G, d=d, dv=dv, P=P, ctx=ctx, n_new=n_new, chunk=chunk, spike=spike, seed=seed)
    want = c.expected()[0]
    gated = want * torch.sigmoid(c.gates.double()[:, 8:8 + H * dv]).view(n_new, H, dv)
    torch.testing.assert_close(c.run(how, splits=splits, gated=True), gated, **c.tol())
    if spike is not None:
        for i in range(n_new):
            p = ctx - n_new + i
            assert (float(want[i].mean()) > 3.5) == (spike <= p and spike // chunk == p // chunk), (spike, i)


# head sizes of every kernel the paged launches may take: 128 (prompts on tcgen05), multiples of 32 and of 16, float32
PAGED = [("bfloat16", 128, 2, 4), ("bfloat16", 64, 2, 6), ("bfloat16", 48, 1, 3), ("bfloat16", 16, 1, 24), ("bfloat16", 256, 1, 2), ("float32", 40, 1, 2)]


@pytest.mark.parametrize("dtype,d,G,H", PAGED)
@pytest.mark.parametrize("n_new", [1, 2, 13, 150])
def test_paged_attention_within_chunks(dtype, d, G, H, n_new):
    """The spike on the first and the last key of a chunk, just outside it, on page and tile borders inside it, on the first and
    last query itself; chunks of one token, shorter than a tile, off every border, and wider than everything."""
    for ctx, chunk, P in ((300, 100, 16), (300, 37, 4), (257, 64, 8), (400, 256, 16), (300, 1, 16), (290, 1000, 1)):
        first, last = ctx - n_new, ctx - 1
        a, b = first - first % chunk, last - last % chunk          # the chunks of the first and the last query
        places = {a, max(a - 1, 0), first, last, b, max(b - 1, 0), 0, min(last, (a // 128 + 1) * 128), min(last, a + chunk - 1)}
        if n_new >= 100 or chunk == 1000:
            places = {a, max(a - 1, 0), b, max(b - 1, 0)}
        for spike in sorted(places):
            _chunk_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=P, ctx=ctx, n_new=n_new, chunk=chunk, spike=spike, seed=spike)
    _chunk_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=16, ctx=n_new, n_new=n_new, chunk=48, spike=0, seed=3)          # the first tokens


@pytest.mark.parametrize("dtype,d,G,H", PAGED)
@pytest.mark.parametrize("splits", [2, 5])
def test_paged_attention_within_chunks_whose_keys_are_cut(dtype, d, G, H, splits):
    for n_new in (1, 2):
        for chunk, spikes in ((700, (699, 700, 701, 720, 959, 998)), (333, (665, 666, 800, 998)), (2000, (0, 160, 998))):
            for spike in spikes:
                _chunk_case(dtype, "paged", H=H, G=G, d=d, dv=d, P=8, ctx=999, n_new=n_new, chunk=chunk, spike=spike, seed=spike, splits=splits)


PAIR = [("float32", "pair"), ("bfloat16", "f32"), ("bfloat16", "pair")]


@pytest.mark.parametrize("dtype,how", PAIR)
@pytest.mark.parametrize("geo", [dict(H=6, G=3, d=40, dv=24, P=4), dict(H=3, G=1, d=64, dv=48, P=16), dict(H=24, G=1, d=16, dv=32, P=8), dict(H=80, G=1, d=8, dv=16, P=2),
                                 dict(H=1, G=1, d=36, dv=20, P=1)])
@pytest.mark.parametrize("n_new", [1, 2, 13, 90])
def test_attention_of_any_pair_of_sizes_within_chunks(dtype, how, geo, n_new):
    for ctx, chunk in ((300, 100), (300, 37), (256, 64), (300, 1)):
        first, last = ctx - n_new, ctx - 1
        a, b = first - first % chunk, last - last % chunk
        places = {a, max(a - 1, 0), first, last, b, max(b - 1, 0)} if n_new < 90 else {a, max(b - 1, 0)}
        for spike in sorted(places):
            _chunk_case(dtype, how, ctx=ctx, n_new=n_new, chunk=chunk, spike=spike, seed=spike, **geo)


@pytest.mark.parametrize("dtype,how", PAIR)
def test_attention_of_any_pair_of_sizes_within_chunks_in_pieces(dtype, how):
    """A decoded token whose chunk is cut into pieces of 256 keys for blocks of their own, chunks that begin inside a piece."""
    from mini_sglang_b200 import ops
    for chunk in (600, 500, 256, 1100, 90):
        assert ops.sink_attention_splits(70, 16, 0, chunk) == min(5, (chunk - 1) // 256 + 2)
        a = 1099 - 1099 % chunk
        for spike in sorted({a, max(a - 1, 0), 1024, 1098, 1099, min(1099, a + 255), min(1099, a + 256)}):
            _chunk_case(dtype, how, H=6, G=2, d=40, dv=24, P=16, ctx=1100, n_new=1, chunk=chunk, spike=spike, seed=spike, splits=2)


# (dtype, how, vector size, value size, kv heads, heads): cache rows of 128 (tcgen05), 256 ... 16, more maps a kv head than a
# decode block's columns and than a tile's rows; the kernels for any pair
DIFF = [("bfloat16", "paged", 64, 128, 2, 4), ("bfloat16", "paged", 64, 128, 1, 5), ("bfloat16", "paged", 48, 96, 2, 2), ("bfloat16", "paged", 32, 64, 1, 3),
        ("bfloat16", "paged", 16, 32, 1, 24), ("bfloat16", "paged", 24, 48, 2, 4), ("bfloat16", "paged", 8, 16, 1, 80), ("bfloat16", "paged", 64, 128, 1, 40),
        ("bfloat16", "paged", 128, 256, 1, 2), ("bfloat16", "paged", 40, 80, 2, 6), ("bfloat16", "pair", 32, 40, 2, 4), ("bfloat16", "f32", 20, 24, 1, 3), ("float32", "pair", 24, 48, 2, 4)]


@pytest.mark.parametrize("dtype,how,d,dv,G,H", DIFF)
@pytest.mark.parametrize("n_new", [1, 2, 13, 150])
def test_heads_that_are_the_difference_of_two_maps(dtype, how, d, dv, G, H, n_new):
    """A key that stands out in one map of every head and not in the other (its value then rules that map alone), with the
    second map taken off 0.4 and 1.7 times; far away, on borders, the query itself."""
    ctx = 300
    if H * n_new > 3000:
        ctx = 170
    first, last = ctx - n_new, ctx - 1
    for lam, eps in ((0.4, 1e-5), (1.7, 0.5)):
        diff = (lam, eps, 0.6)
        for spike, m in (((0, 0), (57, 1), (128, 0), (first, 1), (last, 0)) if n_new < 100 else ((0, 1), (128, 0), (last, 1))):
            c = Case(dtype, H=H, G=G, d=d, dv=dv, P=16, ctx=ctx, n_new=n_new, maps=2, spike=spike, spike_map=m, seed=spike + m)
            maps = c.expected()
            want = pr.rms_unit(maps[0] - lam * maps[1], eps) * 0.6
            torch.testing.assert_close(c.run(how, diff=diff), want, **c.tol())
            assert (float(maps[m, -1].mean()) > 3.5) and float(maps[1 - m, -1].mean()) < 2.0
    c = Case(dtype, H=H, G=G, d=d, dv=dv, P=16, ctx=n_new, n_new=n_new, maps=2, seed=1)           # the first tokens of a sequence
    maps = c.expected()
    torch.testing.assert_close(c.run(how, diff=(0.4, 1e-5, 0.6)), pr.rms_unit(maps[0] - 0.4 * maps[1], 1e-5) * 0.6, **c.tol())


@pytest.mark.parametrize("dtype,how,d,dv,G,H", [c for c in DIFF if c[5] < 80])
@pytest.mark.parametrize("splits", [2, 5])
def test_difference_of_two_maps_whose_keys_are_cut(dtype, how, d, dv, G, H, splits):
    for n_new in (1, 2):
        if how != "paged" and n_new == 2:
            continue
        for spike, m in ((0, 0), (160, 1), (400, 0), (799, 1)):
            c = Case(dtype, H=H, G=G, d=d, dv=dv, P=8, ctx=800, n_new=n_new, maps=2, spike=spike, spike_map=m, seed=spike)
            maps = c.expected()
            want = pr.rms_unit(maps[0] - 0.5 * maps[1], 1e-5) * 0.7
            torch.testing.assert_close(c.run(how, splits=splits, diff=(0.5, 1e-5, 0.7)), want, **c.tol())


# ---------------------------------------------------------------------------------------------------------------------
# the model through the step function
# ---------------------------------------------------------------------------------------------------------------------
LENGTHS = {"RA": 75, "RB": 41, "RC": 60}


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["RA", "RB", "RC"])
def test_whole_prompt_token_by_token_and_in_portions(name, dtype):
    """The same sequence three ways: one step; five tokens and then one token a step (through the CUDA graph); portions of
    changing sizes down to two tokens.  Every position against the plain implementation."""
    V = CONFIGS_R[name]["vocab"]
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
@pytest.mark.parametrize("name", ["RA", "RC"])
def test_long_prompt_whole_and_in_long_and_short_portions(name, dtype):
    """A prompt in one step over many chunks, and in long and short portions with a second request's single tokens beside them."""
    V = CONFIGS_R[name]["vocab"]
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
@pytest.mark.parametrize("name", ["RA", "RB", "RC"])
def test_mixed_batches_on_a_small_pool(name, dtype):
    """Five requests of unequal lengths through two request slots and a pool that holds little more than the two longest:
    portions of one beside single tokens of another; pages and block-table rows are used again, and what they held before
    (NaN at the start) must never be read."""
    V = CONFIGS_R[name]["vocab"]
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


@pytest.mark.parametrize("name", ["RA", "RC"])
def test_a_batch_equals_each_request_alone(name):
    """float32: the logits of requests fed together in unequal portions equal those of each alone, to rounding."""
    V = CONFIGS_R[name]["vocab"]
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
@pytest.mark.parametrize("name", ["RA", "RC"])
def test_long_decoding(name, dtype):
    """Two requests decode together for 330 steps through the CUDA graph over many chunks; a third joins late with a portion and
    leaves early.  The chunked groups' pools hold a few chunks, not the sequences."""
    V = CONFIGS_R[name]["vocab"]
    a, b, c = random_tokens(345, V, 1), random_tokens(352, V, 2), random_tokens(30, V, 3)
    seqs = {"a": a, "b": b, "c": c}
    from mini_sglang_b200.engine.step import ModelRunner
    r = ModelRunner.from_model_dir(model_dir(name), dtype=dtype, page_size=PAGE[name], num_pages=-(-800 // PAGE[name]) + 4, max_reqs=3,
                                   max_context_len=1024, max_step_tokens=30)
    for g in r.mgr.groups:
        if g.chunk:
            assert g.pool.num_pages == 3 * (-(-(g.chunk + 30) // PAGE[name]) + 2)
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
def test_fields_of_decode_steps_with_chunks(fields_on_device):
    """Requests in different places of their chunks: the order in which the launches walk them and everything else that the
    device makes of a decode step's fields is what the host makes."""
    name = "RC"
    V = CONFIGS_R[name]["vocab"]
    lens = {"a": 140, "b": 97, "c": 49, "d": 20}
    seqs = {k: random_tokens(n + 12, V, n) for k, n in lens.items()}
    r = runner(name, "bfloat16", num_pages=60, max_reqs=4)
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
        for p, g in r._plans():
            for off, m in ((lay.nsplit[p], bucket), (lay.order[p], bucket), (lay.out_loc[p], len(entries)), (lay.kv_len, len(entries))):
                assert (have[off:off + m] == want[off:off + m]).all(), (p, g.chunk)
        checked.append(1)

    r._meta_on_device = checking
    steps = [{"entries": [(k, seqs[k][:n], [n - 1]) for k, n in lens.items()]}]
    steps += [{"entries": [(k, [seqs[k][n + i]], [0]) for k, n in lens.items()]} for i in range(12)]
    compare(name, "bfloat16", play(r, steps), seqs)
    assert bool(checked) == fields_on_device


@pytest.mark.parametrize("dtype", BOTH)
def test_other_page_sizes(dtype):
    """Pages of one token and pages wider than a request, the same two ways."""
    for name, P in (("RA", 1), ("RB", 64), ("RC", 2), ("RC", 8), ("RA", 64), ("RC", 128)):
        V = CONFIGS_R[name]["vocab"]
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
        compare(f"random {seed}", dtype, got, None, ref=ref, bound=0.1 if dtype == "bfloat16" else None)
        r.mgr.check_idle()


@functools.lru_cache(None)
def _wide():
    """Layers whose sizes the serving kernels take: rows of 128 on 4 kv heads, chunks of 200 tokens, a feed-forward whose product
    has the activation in its epilogue."""
    rot = dict(dims=64, base=50000.0, scaling=tr.RAMP)
    cfg = tr.model(256, 200, 4, 1e-5, [
        tr.layer(tr.chunked(16, 4, 128, 128, 200, dims=128), 512),
        tr.layer(tr.diff(16, 4, 64, 128, **rot), 256),
        tr.layer(tr.diff(16, 4, 64, 128, kv_from=1, lam=0.5, **rot), 512),
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
    assert r.last_step_used_graph
    if dtype == "bfloat16":
        assert max(max(ns) for ns in r.last_plan["nsplits"]) > 1
    compare("wide", dtype, got, None, ref={"a": ref})


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("kinds", ["chunked only", "differential only", "one layer without feed-forward"])
def test_models_of_one_kind_of_layer(kinds, dtype):
    """Through the step function (decode steps of requests of unlike length may deal the keys out evenly, within chunks and in both
    maps) and through the entry point."""
    from mini_sglang_b200 import Engine, EngineArgs
    from mini_sglang_b200.engine.step import ModelRunner
    cfg = {"chunked only": tr.model(64, 90, 2, 1e-5, [tr.layer(tr.chunked(4, 2, 64, 64, 2500, dims=32), 24), tr.layer(tr.chunked(8, 2, 64, 64, 2500, dims=64), None)]),
           "differential only": tr.model(48, 70, 3, 1e-5, [tr.layer(tr.diff(4, 2, 32, 64, dims=32, scaling=tr.RAMP), 16),
                                                           tr.layer(tr.diff(4, 2, 32, 64, dims=32, scaling=tr.RAMP, kv_from=0), None)]),
           "one layer without feed-forward": tr.model(40, 50, 2, 1e-6, [tr.layer(tr.diff(2, 2, 6, 20, dims=4), None)])}[kinds]
    w = make_weights(cfg, 31)
    path = write_model_dir(os.path.join(_tmp.name, kinds.replace(" ", "_")), cfg, w)
    V = cfg["vocab"]
    lens = {"a": 60, "b": 31, "c": 9} if kinds.startswith("one") else {"a": 2400, "b": 500, "c": 2700}
    seqs = {k: random_tokens(n + 4, V, n) for k, n in lens.items()}
    ref = {k: plain_of(cfg, w, t) for k, t in seqs.items()}
    r = ModelRunner.from_model_dir(path, dtype=dtype, page_size=16, num_pages=370, max_reqs=3, max_context_len=4096)
    poison(r)
    steps = [{"entries": [(k, seqs[k][:n], [0, n - 1])]} for k, n in lens.items()]
    steps += [{"entries": [(k, [seqs[k][n + i]], [0]) for k, n in lens.items()]} for i in range(4)]
    got = play(r, steps)
    assert r.last_step_used_graph
    if not kinds.startswith("one") and dtype == "bfloat16":
        assert r.last_plan["graph_key"][2] == ("even" if kinds == "chunked only" else True if max(lens.values()) < 1.25 * sum(lens.values()) / 3 else "even")
    compare(kinds, dtype, got, None, ref=ref)
    eng = Engine(EngineArgs(model=path, dtype=dtype, page_size=4, num_pages=32, max_num_reqs=2, random_seed=0, max_context_len=64, log_level="WARNING"))
    prompts = [random_tokens(n, V, 3 + n) for n in (4, 17)]
    outs = eng.generate(input_ids=prompts, sampling_params={"temperature": 0.0, "max_new_tokens": 6, "ignore_eos": True})
    for p, o in zip(prompts, outs):
        if dtype == "float32":
            assert o["token_ids"] == pr.greedy_generate(cfg, w, p, 6)
    eng.scheduler.check_idle_invariants()


def _holds(cfg, w, prompt, got, dtype):
    if dtype == "float32":
        assert got == pr.greedy_generate(cfg, w, prompt, len(got))
        return
    toks = list(prompt)
    for t in got:           # bfloat16 may take another of two nearly equal logits
        row = plain_of(cfg, w, toks)[-1]
        assert float(row.max() - row[t]) < 0.25 * float(row.std())
        toks.append(t)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["RA", "RC"])
def test_greedy_generation_through_the_entry_point(name, dtype):
    """Engine.generate with the scheduler: prompts of unequal lengths, portions of at most 16 tokens, a small pool; then a second
    round of requests on the pages of the first."""
    from mini_sglang_b200 import Engine, EngineArgs
    cfg = CONFIGS_R[name]
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
    name = "RB"
    V = CONFIGS_R[name]["vocab"]
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
