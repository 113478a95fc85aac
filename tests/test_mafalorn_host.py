"""Mafalorn without a GPU: the configuration reader and its refusals, the registry, and closed forms of the plain oracle (rotations,
interpolated frequencies, retention, values that are unrotated keys, delta rule, convolution, window, group-limited routing,
identity experts, norms on both sides)."""
import copy
import json
import math

import pytest
import torch

from jacobiforcing_b200 import hybrid_config as hcfg
from jacobiforcing_b200.hybrid_config import HybridConfig
from jacobiforcing_b200.registry import FAMILIES, family_of_config, resolve
from oracle import mafalorn_plain as plain
from tests.mafalorn_helpers import SCALING, SMALL, lat, model_config, moe, par, ret

D = torch.float64


def t(*rows):
    return torch.tensor(rows, dtype=D)


def test_config_reader_reads_every_size_and_constant():
    hc = HybridConfig.from_dict(SMALL)
    assert (hc.architecture, hc.width, hc.vocab, len(hc.layers), hc.norm_eps, hc.logit_scale, hc.emb_scale) == ("Mafalorn", 40, 70, 6, 2e-5, 0.7, 1.0)
    assert (hc.block_kind, hc.norm_kind, hc.pos_kind, hc.tied_head) == (hcfg.BLOCK_SANDWICH, hcfg.NORM_RMS, hcfg.POS_NONE, False)
    r = hc.layers[3]
    assert (r.mixer, r.g_heads, r.g_dim, r.g_vdim, r.r_dims, r.r_base, r.r_half, r.r_factor) == (hcfg.MIX_RETENTION, 2, 20, 8, 16, 90.0, 1, 0.0)
    assert r.decay == tuple(SMALL["layers"][3]["mixer"]["decay"]) and r.ff_kind == hcfg.FF_NONE
    p = hc.layers[1]
    assert (p.mixer, p.b_heads, p.b_kv_heads, p.b_dim, p.b_vdim, p.b_scale, p.b_bias) == (hcfg.MIX_ATTN_DELTA, 4, 2, 16, 16, 0.4, hcfg.BIAS_NONE)
    assert (p.d_heads, p.d_kv_heads, p.d_dim, p.d_vdim, p.d_conv, p.left_scale, p.right_scale) == (4, 2, 12, 20, 3, 0.7, 1.3)
    assert (p.r_dims, p.r_base, p.r_half, p.r_factor, p.r_original, p.r_fast, p.r_slow) == (12, 200.0, 1, 5.0, 40.0, 8.0, 0.5)
    assert (p.ff_kind, p.x_experts, p.x_top, p.ff, p.x_identity, p.x_groups, p.x_keep) == (hcfg.FF_ROUTED, 7, 3, 24, 2, 3, 2)
    assert (p.x_route, p.x_plain, p.x_act) == (hcfg.ROUTE_CORRECTED_SOFTMAX, 0, hcfg.ACT_SILU)
    la = hc.layers[5]
    assert (la.mixer, la.l_heads, la.l_dim, la.l_rot_dim, la.l_vdim, la.l_kv_rank, la.l_q_rank) == (hcfg.MIX_LATENT, 2, 8, 12, 20, 16, 0)
    assert (la.l_no_sink, la.r_half, la.r_dims, la.r_base, la.l_scale, la.l_window, la.l_gate) == (1, 0, 12, 300.0, 0.4, 19, 1)
    assert (la.x_experts, la.x_top, la.x_identity, la.x_groups, la.x_keep) == (3, 3, 1, 1, 1)
    assert [x.cache_elems_per_token() for x in (r, p, la)] == [0, 2 * (16 + 16), 16 + 12]


def test_what_the_configuration_leaves_out_does_not_exist():
    cfg = model_config([lat(size=None, mlp=moe(identity=None, groups=None)), par(scaling=None, mlp=None)])
    del cfg["logit_scale"]
    hc = HybridConfig.from_dict(cfg)
    a, b = hc.layers
    assert (a.l_window, a.x_identity, a.x_groups, a.x_keep, b.r_factor, b.ff_kind, hc.logit_scale) == (0, 0, 1, 1, 0.0, hcfg.FF_NONE, 1.0)
    names = plain.tensor_shapes(cfg)
    assert "l1.norm1b" in names and "l1.norm2" not in names and names["l0.mlp.router"] == (7, 40)


def test_config_reader_refuses_what_a_kernel_would_index_with():
    def bad(change, exc=ValueError):
        cfg = copy.deepcopy(SMALL)
        change(cfg["layers"])
        with pytest.raises(exc):
            HybridConfig.from_dict(cfg)
    bad(lambda c: c[0]["mixer"].update(decay=[0.5, 0.5]))
    bad(lambda c: c[0]["mixer"]["rot"].update(dims=7))
    bad(lambda c: c[0]["mixer"]["rot"].update(dims=14))
    bad(lambda c: c[1]["mixer"]["left"].update(kv_heads=3))
    bad(lambda c: c[1]["mixer"]["left"].update(vdim=12))
    bad(lambda c: c[1]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0))
    bad(lambda c: c[1]["mixer"]["right"].update(kv_heads=3))
    bad(lambda c: c[1]["mixer"]["right"].update(conv=17))
    bad(lambda c: c[2]["mixer"].update(mask={"size": -1}))
    bad(lambda c: c[2]["mixer"]["rot"].update(dims=10))
    bad(lambda c: c[2]["mlp"]["router"].update(groups={"count": 4, "keep": 1}))     # nine outputs
    bad(lambda c: c[2]["mlp"]["router"].update(groups={"count": 3, "keep": 4}))
    bad(lambda c: c[2]["mlp"]["router"].update(top=7))                              # two kept groups of three
    bad(lambda c: c[0].update(type="gla"), NotImplementedError)
    bad(lambda c: c[1]["mlp"].update(kind="dense"), NotImplementedError)


def test_registry_serves_it_through_the_hybrid_family(tmp_path):
    assert FAMILIES["Mafalorn"].name == "hybrid"
    (tmp_path / "config.json").write_text(json.dumps(SMALL))
    assert resolve(str(tmp_path)).name == "hybrid"
    assert family_of_config(HybridConfig.from_dict(SMALL)) is FAMILIES["Mafalorn"]


# ---- closed forms of the oracle --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("pairs", ["half", "neighbour"])
def test_rotation_by_hand(pairs):
    x = torch.zeros(4, 5, dtype=D)
    x[3] = t([1.0, 2.0, 3.0, 4.0, 5.0])[0]
    out = plain.rotate_all(x, {"base": 100.0, "dims": 4}, getattr(plain, pairs + "_pairs")(4))[3]
    for (i, j), f in zip([(0, 2), (1, 3)] if pairs == "half" else [(0, 1), (2, 3)], (1.0, 0.1)):
        a = 3.0 * f
        assert math.isclose(float(out[i]), float(x[3, i]) * math.cos(a) - float(x[3, j]) * math.sin(a), rel_tol=1e-12)
        assert math.isclose(float(out[j]), float(x[3, j]) * math.cos(a) + float(x[3, i]) * math.sin(a), rel_tol=1e-12)
    assert float(out[4]) == 5.0


def test_interpolated_frequencies_by_hand():
    rot = {"base": 10000.0, "dims": 8, "scaling": {"factor": 4.0, "original": 2000, "fast": 100.0, "slow": 1.0}}
    f = plain.frequencies(rot)
    at = lambda turns: 8 * math.log(2000 / (2 * math.pi * turns)) / (2 * math.log(10000.0))
    lo, hi = math.floor(at(100.0)), math.ceil(at(1.0))
    assert (lo, hi) == (0, 3)
    for i in range(4):
        plain_f, ramp = 10000.0 ** (-2 * i / 8), i / 3
        assert math.isclose(f[i], plain_f / 4.0 * ramp + plain_f * (1 - ramp), rel_tol=1e-12)
    assert math.isclose(plain.magnitude(rot), 0.1 * math.log(4.0) + 1.0)
    assert plain.magnitude({"base": 10.0, "dims": 4}) == 1.0
    # a range that collapses: every pair below it keeps its frequency, every pair above is divided
    rot["scaling"].update(fast=1.0, slow=1.0, original=2000)
    assert math.isclose(plain.frequencies(rot)[3], 10000.0 ** (-6 / 8) / 4.0, rel_tol=1e-12)


def test_engine_reads_the_same_rotation():
    spec = HybridConfig.from_dict(model_config([par()])).layers[0]
    assert {"factor": spec.r_factor, "original": spec.r_original, "fast": spec.r_fast, "slow": spec.r_slow} == {k: float(v) for k, v in SCALING.items()}


def test_retention_by_hand():
    one = t([1.0])
    p = {"q": one, "k": one, "v": t([1.0], [2.0]), "g": t([1.0], [1.0]), "o": torch.eye(2, dtype=D)}
    c = {"heads": 1, "dim": 1, "vdim": 2, "decay": [0.25], "rot": {"base": 10.0, "dims": 0}}
    out = plain.retention(t([1.0], [3.0]), p, c, 1e3)              # a large eps: the norm hardly depends on the read-out
    for row, (s, x) in zip(out, [(1.0, 1.0), ((0.25 + 9.0) * 3.0, 3.0)]):
        o = torch.tensor([s, 2.0 * s], dtype=D)
        assert torch.allclose(row, o / torch.sqrt((o * o).mean() + 1e3) * (x / (1.0 + math.exp(-x))))


def test_keys_are_scaled_and_heads_normed_without_a_weight():
    """dim 4: one key written at the first token, read at once: (q.k) / 2 times the value, divided by its root mean square."""
    p = {"q": t([1.0], [1.0], [0.0], [0.0]), "k": t([2.0], [0.0], [0.0], [0.0]), "v": t([3.0]), "g": t([1.0]), "o": t([1.0])}
    c = {"heads": 1, "dim": 4, "vdim": 1, "decay": [0.5], "rot": {"base": 10.0, "dims": 2}}
    out = plain.retention(t([1.0]), p, c, 7.0)
    o = 2.0 * 0.5 * 3.0
    assert math.isclose(float(out[0, 0]), o / math.sqrt(o * o + 7.0) / (1.0 + math.exp(-1.0)), rel_tol=1e-12)


def test_values_are_keys_before_their_rotation():
    """One head, equal keys; the scores differ by position, the values do not: the answer is the key itself times gate."""
    p = {"q": t([1.0], [0.5]), "k": t([0.3], [-0.8]), "g": t([0.0]), "o": torch.eye(2, dtype=D)}
    c = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 2.0, "rot": {"base": 50.0, "dims": 2}}
    out = plain.key_valued_attention(t([1.0], [1.0], [1.0]), p, c)
    assert torch.allclose(out, 0.5 * t([0.3, -0.8]).expand(3, 2))


def test_delta_rule_by_hand():
    p = {"q": t([1.0]), "k": t([1.0]), "v": t([2.0]), "q.conv": t([1.0]), "k.conv": t([1.0]), "v.conv": t([1.0]), "b": t([0.0]), "a": t([0.0]),
         "A_log": torch.zeros(1, dtype=D), "dt_bias": torch.zeros(1, dtype=D), "norm": torch.full((1,), 3.0, dtype=D), "g": t([1.0]), "o": t([1.0])}
    c = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "conv": 1}
    h = t([1.0], [2.0])
    silu = lambda z: z / (1.0 + math.exp(-z))
    unit = lambda z: z / math.sqrt(z * z + 1e-6)
    S, g = 0.0, math.exp(-math.log(2.0))                            # exp(-exp(0) softplus(0))
    out = plain.delta_rule(h, p, c, 1e2)
    for row, x in zip(out, (1.0, 2.0)):
        k = unit(silu(x))
        S *= g
        S += k * 0.5 * (silu(2.0 * x) - S * k)
        o = S * k
        assert math.isclose(float(row[0]), o / math.sqrt(o * o + 1e2) * 3.0 * silu(x), rel_tol=1e-9)


def test_convolution_by_hand():
    x = t([1.0], [10.0], [100.0])
    y = plain.short_conv(x, t([0.5, -1.0, 2.0]))
    want = t([2.0], [20.0 - 1.0], [200.0 - 10.0 + 0.5])
    assert torch.allclose(y, want / (1.0 + torch.exp(-want)))


def test_window_by_hand():
    assert [j for j in range(12) if plain.causal(9, j, 3)] == [7, 8, 9]
    assert [j for j in range(12) if plain.causal(1, j, 3)] == [0, 1]
    assert [j for j in range(12) if plain.causal(5, j)] == [0, 1, 2, 3, 4, 5]
    w = plain.softmax_seen(torch.zeros(4, 4, dtype=D), 2)
    assert torch.allclose(w, t([1, 0, 0, 0], [0.5, 0.5, 0, 0], [0, 0.5, 0.5, 0], [0, 0, 0.5, 0.5]).double())


def test_group_limited_routing_by_hand():
    router = torch.log(t([0.30], [0.10], [0.20], [0.15], [0.05], [0.20]))       # the scores for h = 1
    h = torch.ones(1, 1, dtype=D)
    r = {"top": 2, "groups": {"count": 3, "keep": 1}}
    none = torch.zeros(6, dtype=D)
    assert plain.route(h, router, none, r)[0] == [[0, 1]]                       # the best single output decides, not the sum
    c = torch.tensor([-0.9, -0.9, -0.75, -0.9, -0.8, -0.9], dtype=D)            # choice: -.6 -.8 | -.55 -.75 | -.75 -.7
    ids, wts = plain.route(h, router, c, r)
    assert ids == [[2, 3]] and torch.allclose(wts[0], torch.tensor([0.20, 0.15], dtype=D))
    ids, _ = plain.route(h, router, c, dict(r, groups={"count": 3, "keep": 2}))
    assert ids == [[2, 0]]
    ids, _ = plain.route(h, router, c, {"top": 3})
    assert ids == [[2, 0, 5]]


def test_identity_experts_pass_their_input():
    h = t([2.0, -1.0])
    router = torch.log(torch.tensor([[0.5], [0.3], [0.2]], dtype=D)) @ t([0.5, 0.0])      # h @ router.T = log scores
    p = {"router": router, "correction": torch.tensor([-9.0, 0.0, 0.0], dtype=D)}
    out = plain.experts(h, p, {"router": {"experts": 1, "identity": 2, "top": 2}})
    assert torch.allclose(out, (0.3 + 0.2) * h)


def test_norms_sit_on_both_sides_of_a_sublayer():
    """A mixer that writes nothing leaves the stream as it is; doubling its output projection does not change what is added."""
    cfg = model_config([ret(mlp=None)], eps=1e-12)
    w = {k: v.double() for k, v in plain.random_weights(cfg, 3).items()}
    base, a, b = [], [], []
    plain.forward(cfg, dict(w, **{"l0.mix.o": torch.zeros_like(w["l0.mix.o"])}), [3, 5, 8], layers_out=base)
    assert torch.allclose(base[0], w["embed"][[3, 5, 8]])
    plain.forward(cfg, w, [3, 5, 8], layers_out=a)
    plain.forward(cfg, dict(w, **{"l0.mix.o": 2.0 * w["l0.mix.o"]}), [3, 5, 8], layers_out=b)
    assert torch.allclose(a[0], b[0], atol=1e-9)
    add = (a[0] - base[0]) / w["l0.norm1b"]
    assert torch.allclose((add * add).mean(1), torch.ones(3, dtype=D), atol=1e-9)
