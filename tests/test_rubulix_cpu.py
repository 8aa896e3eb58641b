"""Rubulix without a GPU: the configuration reader and the model description against the tiny configurations, the plain
implementation's mechanisms against closed forms and hand-made cases, what the model-level bound of the GPU tests can tell apart,
and what the cache manager and the planners of the attention launches make of chunks."""

import copy
import math

import numpy as np
import pytest
import torch

import plain_rubulix as pr
from tiny_models import random_tokens
from tiny_rubulix import CONFIGS_R, RAMP, make_weights, random_config, tensor_shapes

F64 = torch.float64
RANDOM = 8


def _raw(name):
    return CONFIGS_R[name] if name in CONFIGS_R else random_config(int(name[6:]))


@pytest.mark.parametrize("name", sorted(CONFIGS_R) + [f"random{s}" for s in range(RANDOM)])
def test_description_declares_the_checkpoints_tensors(name):
    from mini_sglang_b200.config import architecture_of
    from mini_sglang_b200.parts.model import expected_tensors
    raw = _raw(name)
    arch = architecture_of(raw)
    assert arch.name == "Rubulix"
    spec = arch.build_spec(arch.config_cls.from_dict(raw))
    spec.validate()
    want = tensor_shapes(raw)
    got = {k: d for k, d in expected_tensors(spec).items() if not d.optional}
    assert set(got) == set(want)
    for k, decl in got.items():
        assert tuple(decl.shape) == tuple(want[k]), (k, decl.shape, want[k])
    for i, (run, l, entry) in enumerate(zip(spec.schedule, spec.layers, raw["layers"])):
        m = entry["mixer"]
        src = m.get("kv_from")
        assert (run.layer, run.cache, run.writes_cache) == (i, i if src is None else src, src is None)
        assert l.mixer["scale"] == m["scale"] and l.mixer["norm_eps"] == raw["norm"]["eps"] and l.mixer["own_kv"] == (src is None)
        assert l.position["rotary_dim"] == m["rot"]["dims"] and l.position["theta"] == m["rot"]["base"] and l.position["interleaved"]
        assert (l.position["scaling"] is None) == ("scaling" not in m["rot"])
        if entry["type"] == "attention":
            assert l.mixer.kind == "differential_attention" and l.mixer["diff"] == m["diff"]
        else:
            assert l.mixer.kind == "sink_attention" and l.mixer["chunk"] == m["mask"]["size"] and l.mixer["qk_unit"]
        assert (l.feed_forward is None) == (entry["mlp"] is None)
        assert l.block_params["streams"] == raw["streams"]
    assert spec.final_norm["streams"] == raw["streams"] and not spec.head["tied"]


def test_needs_of_the_layers():
    """A cache row of differential keys is both vectors; chunked layers of one size share a group; a layer on another's keys needs
    no cache of its own."""
    from mini_sglang_b200.cache import CacheManager
    from mini_sglang_b200.config import architecture_of
    from mini_sglang_b200.parts import BuildEnv, DecoderModel
    raw = CONFIGS_R["RA"]
    arch = architecture_of(raw)
    model = DecoderModel(arch.build_spec(arch.config_cls.from_dict(raw)), BuildEnv(dtype=torch.bfloat16, device=torch.device("cpu")))
    needs = model.cache_needs()
    assert set(needs) == {0, 1, 3, 4}
    assert (needs[1].head_dim, needs[1].v_head_dim or 32, needs[1].q_heads, needs[1].chunk, needs[1].library) == (32, 32, 8, None, "attention")
    assert (needs[4].head_dim, needs[4].v_head_dim, needs[4].chunk, needs[4].library) == (24, 20, None, "mixers_delta")
    assert (needs[0].chunk, needs[3].chunk, needs[0].library, needs[3].library) == (20, 33, "mixers_delta", "attention")
    mgr = CacheManager(needs, page_size=4, num_pages=40, max_reqs=2, max_context_len=100, max_step_tokens=16)
    assert sorted((g.window, g.chunk, tuple(g.cache_ids)) for g in mgr.groups if g.chunk) == [(None, 20, (0,)), (None, 33, (3,))]
    assert [g.cache_ids for g in mgr.groups if g.span is None] == [[1, 4]]


def test_configuration_refusals():
    from mini_sglang_b200.config import ConfigError, architecture_of
    raw = CONFIGS_R["RA"]
    arch = architecture_of(raw)
    L = lambda c, i: c["layers"][i]        # noqa: E731
    for change in (lambda c: L(c, 0).__setitem__("type", "something"),
                   lambda c: L(c, 0)["mlp"].__setitem__("kind", "something"),
                   lambda c: L(c, 0)["mlp"].pop("ff"),
                   lambda c: L(c, 0)["mixer"].pop("heads"),
                   lambda c: L(c, 0)["mixer"].pop("scale"),
                   lambda c: L(c, 0)["mixer"].pop("mask"),
                   lambda c: L(c, 0)["mixer"]["mask"].__setitem__("size", 0),
                   lambda c: L(c, 1)["mixer"].pop("diff"),
                   lambda c: L(c, 1)["mixer"]["rot"].__setitem__("dims", 18),
                   lambda c: L(c, 1)["mixer"]["rot"].__setitem__("dims", 7),
                   lambda c: L(c, 1)["mixer"]["rot"]["scaling"].pop("fast"),
                   lambda c: L(c, 2)["mixer"].__setitem__("kv_from", 2),            # itself
                   lambda c: L(c, 2)["mixer"].__setitem__("kv_from", 4),            # a later one
                   lambda c: L(c, 2)["mixer"].__setitem__("kv_from", 0),            # another kind
                   lambda c: L(c, 5)["mixer"].__setitem__("kv_from", 2),            # one without keys of its own
                   lambda c: L(c, 5)["mixer"].__setitem__("kv_from", 4),            # other sizes
                   lambda c: c.pop("norm"),
                   lambda c: c.pop("streams"),
                   lambda c: c.__setitem__("streams", 0),
                   lambda c: c.pop("width")):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(ConfigError):
            arch.build_spec(arch.config_cls.from_dict(bad))


@pytest.mark.parametrize("dims,base,sc", [(16, 500.0, RAMP), (4, 100.0, None), (32, 250000.0, {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}),
                                          (8, 50.0, {"factor": 2.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                                          (8, 30.0, {"factor": 16.0, "original": 16, "fast": 4.0, "slow": 0.5})])
def test_frequencies_of_the_engine_equal_the_plain_ones(dims, base, sc):
    from mini_sglang_b200.parts.rope import yarn_frequencies
    got, mag = yarn_frequencies(dims, base, sc)
    want, wmag = pr.frequencies(dims, base, sc)
    torch.testing.assert_close(got, torch.tensor(want, dtype=F64), rtol=1e-14, atol=0)
    assert mag == wmag == (0.1 * math.log(sc["factor"]) + 1.0 if sc else 1.0)


# -- the plain mechanisms ----------------------------------------------------------------------------------------------

def test_layer_norm_with_a_bias():
    x = torch.tensor([[1.0, 2.0, 3.0, 6.0]], dtype=F64)
    w, b = torch.tensor([1.0, 1.0, 2.0, 1.0], dtype=F64), torch.tensor([0.0, 5.0, 0.0, -1.0], dtype=F64)
    var = (4 + 1 + 0 + 9) / 4
    torch.testing.assert_close(pr.layer_norm(x, w, b, 0.5), torch.tensor([[-2.0, -1.0, 0.0, 3.0]], dtype=F64) / math.sqrt(var + 0.5) + b)


def test_streams_are_read_and_rewritten_all_at_once():
    X = torch.tensor([[[1.0, 10.0], [2.0, 20.0]]], dtype=F64)            # one token, two copies
    torch.testing.assert_close(pr.read_streams(X, torch.tensor([3.0, -1.0], dtype=F64)), torch.tensor([[1.0, 10.0]], dtype=F64))
    mix = torch.tensor([[0.0, 1.0], [5.0, 0.0]], dtype=F64)              # from 1 to 2 as it is, from 2 to 1 five times
    y = torch.tensor([[100.0, 200.0]], dtype=F64)
    new = pr.write_streams(X, y, mix, torch.tensor([0.0, 1.0], dtype=F64))
    torch.testing.assert_close(new, torch.tensor([[[10.0, 100.0], [101.0, 210.0]]], dtype=F64))


def test_rotation_turns_neighbours_and_leaves_the_rest():
    x = torch.arange(1, 7, dtype=F64).view(1, 6).repeat(3, 1)
    y = pr.rotate_neighbours(x, [0.5, 0.25], 2.0)
    for t in range(3):
        for i, f in enumerate((0.5, 0.25)):
            c, s = 2 * math.cos(t * f), 2 * math.sin(t * f)
            u, v = 2 * i + 1.0, 2 * i + 2.0
            assert abs(y[t, 2 * i] - (u * c - v * s)) < 1e-12 and abs(y[t, 2 * i + 1] - (v * c + u * s)) < 1e-12
        assert y[t, 4:].tolist() == [5.0, 6.0]


def test_chunks_count_from_the_start_of_the_sequence():
    seen = pr.same_chunk(7, 3)
    assert [[j for j in range(7) if seen[i, j]] for i in range(7)] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]
    assert torch.equal(pr.same_chunk(5, 1), torch.eye(5, dtype=torch.bool)) and torch.equal(pr.same_chunk(5, 9), pr.causal(5))


def test_difference_of_two_maps():
    """One head, one visible key: both maps give its value, the difference is (1 - lambda) v, brought to unit rms."""
    c = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0, "diff": 0.25, "rot": {"base": 10.0, "dims": 2}}
    eye = torch.eye(2, dtype=F64)
    w = {"m.q": torch.zeros(4, 2, dtype=F64), "m.q.b": torch.zeros(4, dtype=F64), "m.k": torch.zeros(4, 2, dtype=F64), "m.k.b": torch.zeros(4, dtype=F64),
         "m.v": eye, "m.v.b": torch.tensor([0.0, 1.0], dtype=F64), "m.o": eye, "m.lq1": torch.tensor([0.5, 0.0], dtype=F64),
         "m.lk1": torch.tensor([1.0, 9.0], dtype=F64), "m.lq2": torch.tensor([0.0, 2.0], dtype=F64), "m.lk2": torch.tensor([7.0, 0.1], dtype=F64)}
    lam = math.exp(0.5) - math.exp(0.2) + 0.25
    assert abs(pr.difference_weight(w, "m", 0.25) - lam) < 1e-12
    u = torch.tensor([[3.0, 3.0]], dtype=F64)
    out = pr.differential_attention(u, pr.differential_keys_values(u, w, "m", c), w, "m", c, 0.0)
    v = torch.tensor([[3.0, 4.0]], dtype=F64)
    torch.testing.assert_close(out, v / math.sqrt(12.5) * 0.75 * math.copysign(1.0, 1 - lam))


def test_unit_keys_after_the_rotation():
    """Queries and keys of any length give the scores of unit ones: scaling Wk and its bias changes nothing."""
    cfg = CONFIGS_R["RA"]
    w = {k: v.double() for k, v in make_weights(cfg, 1).items()}
    u = torch.randn(9, cfg["width"], dtype=F64, generator=torch.Generator().manual_seed(0))
    c = cfg["layers"][0]["mixer"]
    base = pr.chunked_attention(u, w, "l0.mix", c, 0.0)
    w["l0.mix.k"], w["l0.mix.k.b"] = 3.0 * w["l0.mix.k"], 3.0 * w["l0.mix.k.b"]
    torch.testing.assert_close(pr.chunked_attention(u, w, "l0.mix", c, 0.0), base)


def _rel(a, b):
    return ((a - b).pow(2).mean(-1) / b.pow(2).mean(-1)).sqrt()


def test_model_level_bound_tells_faults_apart(monkeypatch):
    """Mistakes planted in the plain implementation move some row by more than the bound that the GPU tests hold bfloat16 rows
    to."""
    cfg, w = CONFIGS_R["RA"], make_weights(CONFIGS_R["RA"], 3)
    toks = random_tokens(60, cfg["vocab"], 5)

    def run(c, ww):
        with torch.no_grad():
            return pr.forward_sequence(c, ww, toks, dtype=F64)

    ref = run(cfg, w)

    def moved(change_cfg=None, change_w=None, **patches):
        c2, w2 = copy.deepcopy(cfg), dict(w)
        if change_cfg:
            change_cfg(c2)
        if change_w:
            change_w(w2)
        with monkeypatch.context() as m:
            for k, v in patches.items():
                m.setattr(pr, k, v)
            return float(_rel(run(c2, w2), ref).max())

    rms, write, neigh = pr.rms_unit, pr.write_streams, pr.rotate_neighbours

    def halves(x, freq, mag):
        n = len(freq)
        idx = torch.tensor([j for i in range(n) for j in (i, i + n)] + list(range(2 * n, x.shape[-1])))
        inv = torch.empty_like(idx)
        inv[idx] = torch.arange(len(idx))
        return neigh(x[..., idx], freq, mag)[..., inv]

    zero = lambda *names: (lambda d: d.update({n: 0.0 * d[n] for n in names}))        # noqa: E731
    L = lambda c, i: c["layers"][i]["mixer"]                                           # noqa: E731
    faults = {
        "a chunk one token longer": moved(lambda c: L(c, 0)["mask"].__setitem__("size", 21)),
        "chunks left out": moved(lambda c: L(c, 3)["mask"].__setitem__("size", 4096)),
        "rotation in halves": moved(rotate_neighbours=halves),
        "no scaling": moved(lambda c: [L(c, i)["rot"].pop("scaling") for i in (1, 2, 5)]),
        "no unit keys": moved(rms_unit=lambda x, eps: x if x.shape[-1] in (40, 32) and x.dim() == 3 else rms(x, eps)),
        "heads not normed": moved(rms_unit=lambda x, eps: x if x.dim() == 2 else rms(x, eps)),
        "second map left out": moved(difference_weight=lambda w_, p, d: 0.0),
        "lambda without its vectors": moved(difference_weight=lambda w_, p, d: d),
        "factor 1 - diff left out": moved(lambda c: None, None, rms_unit=lambda x, eps: rms(x, eps) * (1.0 if x.dim() == 3 else 1.0 / 0.7)),
        "scale of the layer that made the keys": moved(lambda c: L(c, 2).__setitem__("scale", 0.25)),
        "gate left out": moved(None, zero("l0.mix.g")),
        "q bias left out": moved(None, zero("l1.mix.q.b")),
        "v bias left out": moved(None, zero("l1.mix.v.b")),
        "norm bias left out": moved(None, zero("l1.norm1.b")),
        "mix transposed": moved(write_streams=lambda X, y, mix, out: write(X, y, mix.T, out)),
        "copies rewritten one after the other": moved(write_streams=_one_after_the_other),
        "a feed-forward's share": moved(None, zero("l2.hc2.out")),
    }
    for what, by in faults.items():
        assert by > 0.3, f"{what} moves the rows by {by:.2%} only"


def _one_after_the_other(X, y, mix, w_out):
    X = X.clone()
    for t in range(X.shape[1]):
        X[:, t] = w_out[t] * y + sum(mix[s, t] * X[:, s] for s in range(X.shape[1]))
    return X


# -- chunks in the cache manager and in the planners of the launches -----------------------------------------------------

def test_keys_seen():
    from mini_sglang_b200.cache import keys_seen
    assert [keys_seen(n, None, 4) for n in range(1, 10)] == [1, 2, 3, 4, 1, 2, 3, 4, 1]
    assert [keys_seen(n, 3, None) for n in (1, 3, 9)] == [1, 3, 3] and keys_seen(9, None, None) == 9 and keys_seen(9, None, 1) == 1


def test_pages_come_back_when_a_chunk_has_passed_them():
    """A pool that holds one chunk and a step serves a request of any length; pages that hold a token of the chunk under way stay,
    also when the chunk begins in the middle of one."""
    from mini_sglang_b200.cache import CacheManager, OutOfPages, PagedKVNeed
    for P, C in ((4, 10), (4, 8), (16, 5), (1, 3), (8, 64)):
        mgr = CacheManager({0: PagedKVNeed(1, 8, chunk=C)}, page_size=P, num_pages=1000, max_reqs=2, max_context_len=4000, max_step_tokens=7)
        g = mgr.groups[0]
        assert g.pool.num_pages == 2 * (-(-(C + 7) // P) + 2) and (g.window, g.chunk, g.span) == (None, C, C)
        slot, n = mgr.open(), 0
        rng = np.random.default_rng(P * 100 + C)
        while n < 500:
            k = int(rng.integers(1, 8))
            mgr.reserve(slot, k)
            live = g.table[slot, :int(g.n_pages[slot])]
            for pos in range(n - n % C, n + k):            # what the step's first token sees, and everything behind it
                assert live[pos // P] != 0
            assert len(set(live[live > 0].tolist())) == int((live > 0).sum())
            mgr.commit(slot, k)
            n += k
            first = n - n % C
            assert (g.table[slot, :first // P] == 0).all() and int(g.first_live[slot]) == min(first // P, int(g.n_pages[slot]))
            assert sorted(mgr.owned_pages(slot)) == sorted(int(p) for p in g.table[slot, :int(g.n_pages[slot])] if p)
        mgr.close(slot)
        mgr.check_idle()
    small = CacheManager({0: PagedKVNeed(1, 8, chunk=10)}, page_size=4, num_pages=2, max_reqs=1, max_context_len=100, max_step_tokens=4)
    slot = small.open()
    with pytest.raises(OutOfPages):
        small.reserve(slot, 9)
    for bad in (dict(chunk=0), dict(chunk=4, window=4)):
        with pytest.raises(ValueError):
            CacheManager({0: PagedKVNeed(1, 8, **bad)}, page_size=4, num_pages=4, max_reqs=1, max_context_len=16)
    with pytest.raises(ValueError):          # a chunk shares no prefixes
        small.adopt_prefix(slot, [1])


def test_chunks_in_the_planners():
    from mini_sglang_b200.engine.step import decode_order, plan_even_cut, plan_kv_splits
    common = dict(n_kv=8, group=4, blocks_per_sm=4, tile_tokens=2, cap=16, sm_count=148, window=None)
    # the keys of the chunk under way are cut, not those before it
    assert plan_kv_splits([1], [4096 + 100], chunk=4096, **common) == [1] == plan_kv_splits([1], [100], **common)
    assert plan_kv_splits([1], [4096 + 3000], chunk=4096, **common) == plan_kv_splits([1], [3000], **common) != [1]
    # two tokens across a chunk's edge read the old chunk too
    assert plan_kv_splits([2], [4097], chunk=4096, **common) == plan_kv_splits([2], [4097], **common)
    # order: by the keys of the chunk under way
    assert decode_order([130, 64, 100, 65], [1, 1, 1, 1], None, 5, chunk=64).tolist() == [1, 2, 0, 3, 4]
    rng = np.random.default_rng(0)
    for _ in range(40):
        kv = rng.integers(1, 9000, int(rng.integers(1, 20)))
        C = int(rng.choice([1, 16, 100, 1024, 5000]))
        n, start, blk_req, cum, first_blk, pieces = plan_even_cut(kv, None, int(rng.integers(1, 80)), 8, chunk=C)
        pos = kv - 1
        units = pos // 16 - (pos - pos % C) // 16 + 1
        assert (np.diff(cum) == units).all() and start[0] == 0 and start[n] == cum[-1] and (np.diff(start[:n + 1]) >= 0).all()
        assert pieces.max() <= 8 and (pieces >= 1).all()


def test_admission_counts_a_chunked_group_by_its_chunk():
    from types import SimpleNamespace
    from mini_sglang_b200.engine.scheduler import Scheduler
    from mini_sglang_b200.cache import CacheManager, PagedKVNeed
    mgr = CacheManager({0: PagedKVNeed(1, 8), 1: PagedKVNeed(1, 8, chunk=32)}, page_size=4, num_pages=64, max_reqs=2, max_context_len=200,
                       max_step_tokens=8)
    stub = SimpleNamespace(mgr=mgr, P=4)
    assert Scheduler._hold(stub, 0, 150.0, 8) == 150.0
    assert Scheduler._hold(stub, 1, 150.0, 8) == 32 + 8 + 4 and Scheduler._hold(stub, 1, 10.0, 8) == 10.0
