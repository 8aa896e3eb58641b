"""Pokatar without a GPU: the configuration reader and the model description against the tiny configurations, the engine's
frequencies against the plain ones, the plain implementation's mechanisms against closed forms and hand-made cases, what the
model-level bound of the GPU tests can tell apart, and the kv-split plans of a cache group with two geometries."""

import copy
import math

import pytest
import torch

import plain_pokatar as pk
from tiny_models import random_tokens
from tiny_pokatar import CONFIGS_K, RAMP, make_weights, random_config, tensor_shapes

F64 = torch.float64
RANDOM = 8


def _raw(name):
    return CONFIGS_K[name] if name in CONFIGS_K else random_config(int(name[6:]))


@pytest.mark.parametrize("name", sorted(CONFIGS_K) + [f"random{s}" for s in range(RANDOM)])
def test_description_declares_the_checkpoints_tensors(name):
    from mini_sglang_b200.config import architecture_of
    from mini_sglang_b200.parts.model import expected_tensors
    raw = _raw(name)
    arch = architecture_of(raw)
    assert arch.name == "Pokatar"
    spec = arch.build_spec(arch.config_cls.from_dict(raw))
    spec.validate()
    want = tensor_shapes(raw)
    got = {k: d for k, d in expected_tensors(spec).items() if not d.optional}
    assert set(got) == set(want)
    for k, decl in got.items():
        assert tuple(decl.shape) == tuple(want[k]), (k, decl.shape, want[k])
    assert [r.cache for r in spec.schedule] == list(range(len(raw["layers"])))
    for l, entry in zip(spec.layers, raw["layers"]):
        assert l.mixer.kind == {"attention": "sink_attention", "latent_attention": "latent_attention"}[entry["type"]]
        assert l.mixer["scale"] == entry["mixer"]["scale"] and l.mixer["norm_eps"] == raw["norm"]["eps"]
        assert (l.feed_forward is None) == (entry["mlp"] is None)
        assert l.norms["input"].kind == "layernorm" and l.norms["input"]["eps"] == raw["norm"]["eps"]
        if entry["type"] == "latent_attention":
            assert l.position["rotary_dim"] == entry["mixer"]["rot_dim"] and l.position["theta"] == entry["mixer"]["rot"]["base"]
            assert (l.position["scaling"] is None) == ("scaling" not in entry["mixer"]["rot"])
        else:
            assert l.position is None and l.mixer["sink"] == 0.0
    assert spec.head["tied"] and spec.head["tied_to"] == "embed"


def test_configuration_refusals():
    from mini_sglang_b200.config import ConfigError, architecture_of
    raw = CONFIGS_K["KA"]
    arch = architecture_of(raw)
    for change in (lambda c: c["layers"][0].__setitem__("type", "something"),
                   lambda c: c["layers"][0]["mlp"].__setitem__("kind", "something"),
                   lambda c: c["layers"][0]["mixer"].pop("heads"),
                   lambda c: c["layers"][0]["mixer"].pop("scale"),
                   lambda c: c["layers"][1]["mixer"].pop("kv_rank"),
                   lambda c: c["layers"][1]["mixer"].pop("rot"),
                   lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 18),
                   lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"),
                   lambda c: c["layers"][0]["mlp"].pop("ff"),
                   lambda c: c["layers"][1]["mlp"]["router"].pop("top"),
                   lambda c: c["layers"][1]["mlp"].pop("expert"),
                   lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"),
                   lambda c: c.pop("norm"),
                   lambda c: c.pop("width")):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(ConfigError):
            arch.build_spec(arch.config_cls.from_dict(bad))


def test_router_sizes_that_do_not_fit_are_refused():
    from mini_sglang_b200.config import architecture_of
    from mini_sglang_b200.parts.model import expected_tensors
    for router in ({"experts": 6, "top": 2, "identity": 1, "groups": {"count": 2, "keep": 1}},      # 7 outputs in 2 groups
                   {"experts": 6, "top": 4, "identity": 2, "groups": {"count": 4, "keep": 1}},      # a kept group holds 2
                   {"experts": 6, "top": 2, "identity": 2, "groups": {"count": 4, "keep": 5}}):
        raw = copy.deepcopy(CONFIGS_K["KA"])
        raw["layers"][1]["mlp"]["router"] = router
        arch = architecture_of(raw)
        with pytest.raises(ValueError):
            expected_tensors(arch.build_spec(arch.config_cls.from_dict(raw)))


@pytest.mark.parametrize("dims,base,sc", [(16, 500.0, RAMP), (4, 100.0, None), (32, 250000.0, {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}),
                                          (8, 50.0, {"factor": 2.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                                          (8, 30.0, {"factor": 16.0, "original": 16, "fast": 4.0, "slow": 0.5})])
def test_frequencies_of_the_engine_equal_the_plain_ones(dims, base, sc):
    from mini_sglang_b200.parts.rope import yarn_frequencies
    got, mag = yarn_frequencies(dims, base, sc)
    want, wmag = pk.frequencies(dims, base, sc)
    torch.testing.assert_close(got, want, rtol=1e-14, atol=0)
    assert mag == wmag == (0.1 * math.log(sc["factor"]) + 1.0 if sc else 1.0)
    if sc is RAMP:          # the ramp's both ends and its middle are there
        ratio = (got / pk.frequencies(dims, base, None)[0]).tolist()
        assert ratio[0] == 1.0 and abs(ratio[-1] - 0.25) < 1e-15 and any(0.26 < r < 0.99 for r in ratio)


# -- the plain mechanisms ----------------------------------------------------------------------------------------------

def test_layer_norm_takes_the_mean_off_and_keeps_eps_inside_the_root():
    x = torch.tensor([[1.0, 2.0, 3.0, 6.0]], dtype=F64)
    y = pk.layer_norm(x, torch.tensor([1.0, 1.0, 2.0, 1.0], dtype=F64), 0.5)
    var = (4 + 1 + 0 + 9) / 4
    torch.testing.assert_close(y, torch.tensor([[-2.0, -1.0, 0.0, 3.0]], dtype=F64) / math.sqrt(var + 0.5))
    torch.testing.assert_close(pk.layer_norm(x + 7.0, torch.ones(4, dtype=F64), 0.5), pk.layer_norm(x, torch.ones(4, dtype=F64), 0.5))


def test_softmax_with_one():
    s = torch.tensor([[0.0, float("-inf")], [math.log(3.0), math.log(2.0)], [-800.0, -900.0], [900.0, 0.0]], dtype=F64)
    p = pk.softmax_with_one(s)
    torch.testing.assert_close(p, torch.tensor([[0.5, 0.0], [0.5, 1 / 3], [0.0, 0.0], [1.0, 0.0]], dtype=F64))


def test_rotation_turns_pairs_in_halves_and_leaves_the_rest():
    x = torch.arange(1, 9, dtype=F64).view(1, 8).repeat(4, 1)
    f = torch.tensor([0.5, 0.25], dtype=F64)
    y = pk.rotate(x, f, 1.0)
    assert torch.equal(y[0], x[0]) and torch.equal(y[:, 4:], x[:, 4:])
    a = 3 * 0.25
    assert abs(float(y[3, 1]) - (2 * math.cos(a) - 4 * math.sin(a))) < 1e-12          # element 1 pairs with element 3
    assert abs(float(y[3, 3]) - (4 * math.cos(a) + 2 * math.sin(a))) < 1e-12
    torch.testing.assert_close(pk.rotate(x[:, None], f, 1.5)[2, 0, :4], 1.5 * y[2, :4])


def test_attention_closed_forms():
    torch.manual_seed(0)
    E, d, dv = 5, 4, 3
    c = {"heads": 2, "kv_heads": 1, "dim": d, "vdim": dv, "scale": 0.5}
    w = {"m.q": torch.randn(8, E, dtype=F64), "m.k": torch.randn(4, E, dtype=F64), "m.v": torch.randn(3, E, dtype=F64),
         "m.q.norm": torch.full((4,), 2.0, dtype=F64), "m.k.norm": torch.ones(4, dtype=F64), "m.g": torch.zeros(6, E, dtype=F64),
         "m.o": torch.eye(6, dtype=F64)}
    u = torch.randn(1, E, dtype=F64)
    q, k, v = (u @ w["m.q"].T).view(2, 4), u @ w["m.k"].T, u @ w["m.v"].T
    eps = 1e-3
    unit = lambda t: t / torch.sqrt((t * t).mean(-1, keepdim=True) + eps)            # noqa: E731
    out = pk.attention(u, w, "m", c, eps)
    for h in range(2):        # one token: its weight is e^s / (1 + e^s), half of it passes the gate
        s = float((2.0 * unit(q[h:h + 1]) * unit(k)).sum() * 0.5)
        torch.testing.assert_close(out[0, 3 * h:3 * h + 3], 0.5 * unit(v)[0] / (1 + math.exp(-s)))
    # the same token ten times: the weights grow towards 1, the values stay; nothing depends on the place
    many = pk.attention(u.repeat(10, 1), w, "m", c, eps)
    s = float((2.0 * unit(q[:1]) * unit(k)).sum() * 0.5)
    n = torch.arange(1, 11, dtype=F64)[:, None]
    torch.testing.assert_close(many[:, :3], 0.5 * unit(v) * n * math.exp(s) / (1 + n * math.exp(s)))


def test_latent_attention_against_keys_and_values_written_out():
    torch.manual_seed(3)
    E, H, d, rd, dv, r, T = 6, 2, 4, 4, 3, 5, 7
    c = {"heads": H, "dim": d, "rot_dim": rd, "vdim": dv, "kv_rank": r, "scale": 0.7, "rot": {"base": 10.0, "dims": rd, "scaling": RAMP}}
    w = {"m.q": torch.randn(H * (d + rd), E, dtype=F64), "m.dkv": torch.randn(r + rd, E, dtype=F64), "m.dkv.norm": torch.rand(r, dtype=F64) + 0.5,
         "m.uk": torch.randn(H * d, r, dtype=F64), "m.uv": torch.randn(H * dv, r, dtype=F64), "m.g": torch.randn(H, E, dtype=F64),
         "m.o": torch.eye(H * dv, dtype=F64)}
    u = torch.randn(T, E, dtype=F64)
    out = pk.latent_attention(u, w, "m", c, 1e-4).view(T, H, dv)
    freq, mag = pk.frequencies(rd, 10.0, RAMP)

    def turn(x, p):
        y = x.clone()
        for i in range(rd // 2):
            a = p * float(freq[i])
            y[i] = mag * (x[i] * math.cos(a) - x[i + rd // 2] * math.sin(a))
            y[i + rd // 2] = mag * (x[i + rd // 2] * math.cos(a) + x[i] * math.sin(a))
        return y

    down = u @ w["m.dkv"].T
    lat = down[:, :r] / torch.sqrt((down[:, :r] ** 2).mean(-1, keepdim=True) + 1e-4) * w["m.dkv.norm"]
    for i in (0, 3, 6):
        for h in range(H):
            q = (u[i] @ w["m.q"].T).view(H, d + rd)[h]
            e = []
            for j in range(i + 1):
                kj = torch.cat((w["m.uk"][h * d:(h + 1) * d] @ lat[j], turn(down[j, r:], j)))
                e.append(math.exp(float(torch.cat((q[:d], turn(q[d:], i))) @ kj) * 0.7))
            want = sum(x * (w["m.uv"][h * dv:(h + 1) * dv] @ lat[j]) for j, x in enumerate(e)) / sum(e)
            torch.testing.assert_close(out[i, h], want / (1 + math.exp(-float(w["m.g"][h] @ u[i]))))


def test_choice_within_the_best_groups():
    corr = torch.zeros(6, dtype=F64)
    s = torch.tensor([0.30, 0.02, 0.05, 0.28, 0.20, 0.15], dtype=F64)
    # three groups of two: their scores are 0.30, 0.28, 0.20 (the largest, not the sum)
    assert pk.choose(s, corr, 3, 1, 2)[0] == [0, 1]
    assert pk.choose(s, corr, 3, 2, 2)[0] == [0, 3]
    chosen, gap = pk.choose(s, corr, 3, 2, 3)
    assert chosen == [0, 3, 2] and abs(gap - 0.03) < 1e-12                          # index 2 (0.05) before index 1 (0.02)
    # negative choice scores: an output of a kept group goes before any output of a dropped one
    corr2 = torch.tensor([0.0, -0.9, 0.0, 0.0, -0.5, -0.5], dtype=F64)
    assert pk.choose(s, corr2, 3, 1, 2)[0] == [0, 1]
    corr3 = torch.full((6,), -1.0, dtype=F64)
    assert pk.choose(s, corr3, 3, 2, 4)[0] == [0, 3, 2, 1]
    # the correction steers the choice between groups too
    assert pk.choose(s, torch.tensor([0, 0, 0, 0, 0, 0.3], dtype=F64), 3, 1, 1)[0] == [5]


def test_mixture_closed_forms():
    torch.manual_seed(2)
    E = 4
    w = {"f.router": torch.zeros(4, E, dtype=F64), "f.correction": torch.tensor([0.0, 0.3, 0.2, 0.1], dtype=F64)}
    w["f.router"][0, 0] = 2.0
    for e in range(3):
        w[f"f.e{e}.up"], w[f"f.e{e}.down"] = torch.randn(5, E, dtype=F64), torch.randn(E, 5, dtype=F64)
    w["f.shared.up"], w["f.shared.down"] = torch.randn(2, E, dtype=F64), torch.randn(E, 2, dtype=F64)
    u = torch.tensor([[1.0, -0.5, 0.25, 2.0]], dtype=F64)
    z = math.exp(2.0)
    s = torch.tensor([z, 1.0, 1.0, 1.0], dtype=F64) / (z + 3.0)                    # 0.711, 0.096, 0.096, 0.096
    c = {"expert": {"ff": 5}, "router": {"experts": 3, "identity": 1, "top": 3}, "shared": {"ff": 2}}
    out = pk.mixture(u, w, "f", c)
    # choice scores 0.711, 0.396, 0.296, 0.196: the experts; weights are the scores, neither corrected nor brought to sum 1
    want = s[0] * pk.expert(u, w, "f.e0") + s[1] * pk.expert(u, w, "f.e1") + s[2] * pk.expert(u, w, "f.e2") + pk.expert(u, w, "f.shared")
    torch.testing.assert_close(out, want)
    w["f.correction"] = torch.tensor([0.0, 0.0, 0.0, 0.1], dtype=F64)              # now the identity output beats experts 1 and 2
    c2 = {"expert": {"ff": 5}, "router": {"experts": 3, "identity": 1, "top": 2}}
    torch.testing.assert_close(pk.mixture(u, w, "f", c2), s[0] * pk.expert(u, w, "f.e0") + s[3] * u)
    y = pk.expert(torch.tensor([[1.0, 2.0]], dtype=F64), {"x.up": torch.tensor([[1.0, 1.0], [-1.0, 0.0]], dtype=F64),
                                                            "x.down": torch.eye(2, dtype=F64)}, "x")
    torch.testing.assert_close(y, torch.tensor([[9.0, 0.0]], dtype=F64))


def test_dense_closed_form():
    w = {"f.gate": torch.eye(2, dtype=F64), "f.gate.b": torch.tensor([1.0, -3.0], dtype=F64), "f.up": 2 * torch.eye(2, dtype=F64),
         "f.up.b": torch.tensor([0.5, 0.5], dtype=F64), "f.down": torch.tensor([[1.0, 1.0], [0.0, 1.0]], dtype=F64),
         "f.down.b": torch.tensor([10.0, 20.0], dtype=F64)}
    torch.testing.assert_close(pk.dense(torch.tensor([[1.0, 2.0]], dtype=F64), w, "f"), torch.tensor([[2 * 2.5 + 10.0, 20.0]], dtype=F64))


# -- what the bounds can tell ------------------------------------------------------------------------------------------

def _rel(a, b):
    return ((a - b).pow(2).mean(dim=1).sqrt() / b.pow(2).mean(dim=1).sqrt())


def test_the_model_level_bound_tells_faults_apart(monkeypatch):
    """The GPU tests hold bfloat16 rows to 4 % of a row's rms (float32 rows to 0.02 %).  Faults of the mechanisms move rows by
    more: the one in the denominator left out, a norm left out, a gate, a bias, the frequencies' scaling or their magnitude, the
    groups, the correction in the weights, weights brought to sum 1, the identity outputs, the shared expert."""
    cfg = CONFIGS_K["KA"]
    w = {k: v.double() for k, v in make_weights(cfg, 3).items()}
    toks = random_tokens(60, cfg["vocab"], 5)

    def run(c=cfg, weights=w):
        with torch.no_grad():
            return pk.forward_sequence(c, weights, toks, dtype=F64)

    ref = run()

    def moved(change_cfg=None, change_w=None, **patches):
        c2, w2 = copy.deepcopy(cfg), dict(w)
        if change_cfg:
            change_cfg(c2)
        if change_w:
            change_w(w2)
        with monkeypatch.context() as m:
            for k, v in patches.items():
                m.setattr(pk, k, v)
            return float(_rel(run(c2, w2), ref).max())

    rms, choose = pk.rms_unit, pk.choose
    faults = {
        "no one in the denominator": moved(softmax_with_one=lambda s: torch.softmax(s, dim=-1)),
        "rms norm for layer norm": moved(layer_norm=lambda x, weight, eps: rms(x, eps) * weight),
        "values not normed": moved(rms_unit=lambda x, eps: x if x.shape[-1] == 24 else rms(x, eps)),
        "gate left out": moved(None, lambda d: d.__setitem__("l0.mix.g", 0.0 * d["l0.mix.g"])),
        "head gate left out": moved(None, lambda d: d.__setitem__("l1.mix.g", 0.0 * d["l1.mix.g"])),
        "no scaling": moved(lambda c: c["layers"][1]["mixer"]["rot"].pop("scaling")),
        "down bias left out": moved(None, lambda d: d.__setitem__("l0.mlp.down.b", 0.0 * d["l0.mlp.down.b"])),
        "gate bias left out": moved(None, lambda d: d.__setitem__("l0.mlp.gate.b", 0.0 * d["l0.mlp.gate.b"])),
        "no groups": moved(lambda c: c["layers"][1]["mlp"]["router"].pop("groups")),
        "no correction": moved(None, lambda d: d.__setitem__("l1.mlp.correction", 0.0 * d["l1.mlp.correction"])),
        "identity outputs add nothing": moved(choose=lambda s, corr, g, k, t: ([e for e in choose(s, corr, g, k, t)[0] if e < s.numel() - 2
                                                                                 or s.numel() != 8], 1.0)),
        "no shared expert": moved(lambda c: c["layers"][1]["mlp"].pop("shared")),
    }
    for what, by in faults.items():
        assert by > 0.045, f"{what} moves the rows by {by:.2%} only"


# -- kv splits of a group whose caches differ in geometry ---------------------------------------------------------------

def test_fields_of_a_step_with_two_plans_in_one_group():
    """Two plans of one cache group share token slots and block tables and have kv splits and an order of their own; a group
    without a second geometry has one plan."""
    from mini_sglang_b200.engine.step import _Layout
    lay = _Layout(5, 3, 2, [4, 4, 7], owner=[0, 0, 2])
    assert lay.out_loc[0] == lay.out_loc[1] != lay.out_loc[2] and lay.table[0] == lay.table[1] != lay.table[2]
    assert len({*lay.nsplit, *lay.order}) == 6
    fields = sorted([(lay.input_ids, 5), (lay.positions, 5), (lay.token_req, 5), (lay.q_start, 4), (lay.kv_len, 3), (lay.slots, 3), (lay.want, 2)]
                    + [(o, 5) for o in {*lay.out_loc}] + [(o, 3) for o in lay.nsplit + lay.order] + [(lay.table[0], 12), (lay.table[2], 21)])
    for (a, n), (b, _) in zip(fields, fields[1:]):
        assert a + n <= b
    assert fields[-1][0] + fields[-1][1] <= lay.size
