"""Mafalorn on the GPU against the plain fp64 restatement (oracle/mafalorn_plain.py): each mechanism alone, steps of the design
that must matter (a mistake planted in the oracle changes its answer, the engine agrees with the unchanged oracle), prefill
against token-by-token decoding, portions, unequal batches, reuse of pages and slots, a marked key far back, at page borders and
just inside / just outside the window (in prompts, in decoding, in portions, SIMT and tensor-core attention), the first tokens of
a sequence, long decoding, other sizes, and greedy generation through LLM.generate, the generate command line and the trace
replay."""
import copy

import numpy as np
import pytest
import torch

from oracle import mafalorn_plain as plain
from tests.mafalorn_helpers import (SMALL, TOL, Harness, close, delta_needle, key_value_needle, lat, latent_needle, model_config, moe,
                                    needle_tokens, oracle_logits, par, rand_tokens, rel_err, ret, retention_needle, row_errs, run, settled)

pytestmark = pytest.mark.gpu


def silent(w, *names):
    """Weights with these tensors set to zero."""
    return {k: (torch.zeros_like(v.float()) if k in names else v) for k, v in w.items()}


# ---- each mechanism alone ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["retention", "left", "right", "both", "latent", "no window", "experts"])
def test_mechanism_alone(which, dtype):
    tiny = ret(heads=1, dim=8, vdim=8, mlp=moe())
    cfg = model_config([{"retention": ret(mlp=None), "latent": lat(mlp=None), "no window": lat(size=None, mlp=None), "experts": tiny}.get(which, par(mlp=None))])
    toks = rand_tokens(45, cfg["vocab"], 3)
    w = plain.random_weights(cfg, 0)
    if which in ("left", "right"):
        w = silent(w, f"l0.mix.{'right' if which == 'left' else 'left'}.o")
    got, want = run(cfg, toks, dtype, weights=settled(w) if dtype == "bfloat16" else w)
    assert close(got, want, dtype)


@pytest.mark.parametrize("kw", [dict(experts=8, top=3, identity=4, groups=(4, 2)), dict(experts=1, top=1, identity=None, groups=None),
                                dict(experts=1, top=2, identity=1, groups=(1, 1)), dict(experts=5, top=5, ff=8, identity=0, groups=(5, 5)),
                                dict(experts=4, top=2, ff=10, identity=2, groups=(6, 2)), dict(experts=40, top=3, ff=9, identity=30, groups=(35, 4)),
                                dict(experts=12, top=3, ff=48, identity=4, groups=(2, 1)), dict(experts=60, top=6, ff=16, identity=0, groups=(3, 1))])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_router_shapes(kw, dtype):
    """One expert, every output chosen, groups of one output, more outputs and more groups than a warp, a group of identity experts
    only, a group across the border, expert sizes that the tensor-core product takes and ones it does not; many tokens so that
    the expert-sorted path runs, few so that the per-pair one does."""
    cfg = model_config([ret(heads=1, dim=8, vdim=8, mlp=moe(**kw)), ret(heads=2, dim=8, vdim=8, mlp=moe(**kw))])
    w = plain.random_weights(cfg, 0)
    toks = rand_tokens(80, cfg["vocab"], 4)
    got, want = run(cfg, toks, dtype, cuts=[60, 1, 7, 1], weights=settled(w) if dtype == "bfloat16" else w)
    assert close(got, want, dtype)


def test_only_identity_experts_chosen():
    """The correction sends every token to the group of identity experts: no row of any expert exists, in long and in short steps."""
    cfg = model_config([ret(mlp=moe(experts=2, top=2, identity=2, groups=(2, 1)))])
    w = plain.random_weights(cfg, 1)
    w["l0.mlp.correction"] = torch.tensor([-5.0, -5.0, -3.0, -3.0])       # choice scores are negative everywhere
    toks = rand_tokens(40, cfg["vocab"], 5)
    for dtype in ("float32", "bfloat16"):
        got, want = run(cfg, toks, dtype, cuts=[30, 1], weights=w)
        assert close(got, want, dtype)


# ---- steps of the design that must matter ----------------------------------------------------------------------------------
def _route_with(change):
    def wrong(h, router, correction, r, inner=plain.route):
        return change(inner, h, router, correction, r)
    return wrong


def _dropped_groups_count_as_zero(h, router, correction, r):
    s = torch.softmax(h @ router.T, 1)
    choice, gr = s + correction, r["groups"]
    per = s.shape[1] // gr["count"]
    ids = []
    for t in range(h.shape[0]):
        worth = choice[t].reshape(-1, per).max(1).values
        keep = torch.argsort(worth, descending=True, stable=True)[:gr["keep"]]
        c = torch.zeros_like(choice[t]).reshape(-1, per)
        c[keep] = choice[t].reshape(-1, per)[keep]
        ids.append(torch.argsort(c.flatten(), descending=True, stable=True)[:r["top"]].tolist())
    return ids, [s[t, i] for t, i in enumerate(ids)]


def _delta_reads_before_the_write(h, p, c, eps):
    T, H, G, D, Dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = plain.unit_vector(plain.short_conv(h @ p["q"].T, p["q.conv"]).reshape(T, G, D)) * D ** -0.5
    k = plain.unit_vector(plain.short_conv(h @ p["k"].T, p["k.conv"]).reshape(T, G, D))
    v = plain.short_conv(h @ p["v"].T, p["v.conv"]).reshape(T, H, Dv)
    beta, g = plain.sigmoid(h @ p["b"].T), plain.delta_decay(h, p)
    o = torch.zeros(T, H, Dv, dtype=h.dtype)
    for hh in range(H):
        S = torch.zeros(D, Dv, dtype=h.dtype)
        for t in range(T):
            S = g[t, hh] * S
            o[t, hh] = S.T @ q[t, hh // (H // G)]
            S = S + torch.outer(k[t, hh // (H // G)], beta[t, hh] * (v[t, hh] - S.T @ k[t, hh // (H // G)]))
    o = plain.unit_rms(o, eps) * p["norm"]
    return (o.reshape(T, H * Dv) * plain.silu(h @ p["g"].T)) @ p["o"].T


def _rotated_values(h, p, c):
    T, H, G, D = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    pairs = plain.half_pairs(int(c["rot"]["dims"]))
    q = plain.rotate_all((h @ p["q"].T).reshape(T, H, D), c["rot"], pairs)
    k = plain.rotate_all((h @ p["k"].T).reshape(T, G, D), c["rot"], pairs)
    gate = plain.sigmoid(h @ p["g"].T)
    out = [plain.softmax_seen(q[:, x] @ k[:, x // (H // G)].T * c["scale"]) @ k[:, x // (H // G)] * gate[:, x:x + 1] for x in range(H)]
    return torch.cat(out, 1) @ p["o"].T


def _halves(dims):
    return [(i, i + dims // 2) for i in range(dims // 2)]


def _neighbours(dims):
    return [(2 * i, 2 * i + 1) for i in range(dims // 2)]


PLANTED = {
    "decay per head": ("head_decays", lambda c, inner=plain.head_decays: inner(c).flip(0)),
    "pairing of halves": ("half_pairs", _neighbours),
    "pairing of neighbours": ("neighbour_pairs", _halves),
    "interpolated frequencies": ("frequencies", lambda rot, inner=plain.frequencies: inner({k: v for k, v in rot.items() if k != "scaling"})),
    "factor on cosine and sine": ("magnitude", lambda rot: 1.0),
    "values are unrotated keys": ("key_valued_attention", _rotated_values),
    "order of write and read-out": ("delta_rule", _delta_reads_before_the_write),
    "unit vectors": ("unit_vector", lambda x: x * 0.7),
    "activation behind the convolution": ("short_conv", lambda x, w, inner=plain.short_conv: torch.log(torch.exp(inner(x, w)) + 1.0)),
    "softplus": ("softplus", lambda z: torch.clamp(z, min=0.0)),
    "window length": ("causal", lambda i, j, size=None, inner=plain.causal: inner(i, j, None if size is None else size + 1)),
    "output gate": ("silu", plain.sigmoid),
    "sigmoid gates": ("sigmoid", lambda z: 0.5 + 0.25 * z),
    "group's score": ("group_score", sum),
    "correction": ("route", _route_with(lambda f, h, w, c, r: f(h, w, torch.zeros_like(c), r))),
    "groups": ("route", _route_with(lambda f, h, w, c, r: f(h, w, c, dict(r, groups=None)))),
    "plain weights": ("route", _route_with(lambda f, h, w, c, r: (lambda i, x: (i, [y / y.sum() for y in x]))(*f(h, w, c, r)))),
    "weights without the correction": ("route", _route_with(lambda f, h, w, c, r: (lambda i, x: (i, [y + c[j] for y, j in zip(x, i)]))(*f(h, w, c, r)))),
    "groups that are out": ("route", _dropped_groups_count_as_zero),
}


@pytest.mark.parametrize("what", sorted(PLANTED))
def test_step_matters_and_is_honoured(what, monkeypatch):
    m = moe(experts=7, top=3, identity=2, groups=(3, 2))
    cfg = model_config([ret(heads=2, dim=10, vdim=16, mlp=m), par(scale=0.6, mlp=m), lat(size=9, scale=0.6, mlp=m)])
    w = plain.random_weights(cfg, 9)
    for i in range(3):
        w[f"l{i}.mlp.correction"] = w[f"l{i}.mlp.correction"].float() * 4.0 - (0.9 if what == "groups that are out" else 0.0)
    toks = rand_tokens(48, cfg["vocab"], 10)
    want = oracle_logits(cfg, w, toks)
    name, wrong = PLANTED[what]
    monkeypatch.setattr(plain, name, wrong)
    assert rel_err(oracle_logits(cfg, w, toks)[20:], want[20:]) > 3e-3, "the oracle does not depend on it"
    monkeypatch.undo()
    got, _ = run(cfg, toks, "float32", cuts=[31, 2, 1], weights=w)
    assert rel_err(got, want) < TOL["float32"]


@pytest.mark.parametrize("what", ["left scale", "right scale", "score scale", "latent scale", "eps", "logit scale", "retention base", "rotated dimensions",
                                  "factor", "original", "fast", "slow", "decay", "head norm", "latent norm", "norm behind the mixer", "norm behind the experts",
                                  "decay bias", "A_log", "keep", "window"])
def test_constant_matters_and_is_honoured(what):
    cfg = model_config([ret(), par(scale=0.8), lat(scale=0.8), ret(mlp=None)], eps=0.3)
    w = plain.random_weights(cfg, 12)
    toks = rand_tokens(40, cfg["vocab"], 13)
    want = oracle_logits(cfg, w, toks)
    cfg2, w2 = copy.deepcopy(cfg), dict(w)
    m = [lc["mixer"] for lc in cfg2["layers"]]
    if what == "eps":
        cfg2["norm"]["eps"] = 0.2
    elif what == "logit scale":
        cfg2["logit_scale"] = 0.69
    elif what == "keep":
        cfg2["layers"][1]["mlp"]["router"]["groups"]["keep"] = 1
    elif what in ("factor", "original", "fast", "slow"):
        m[1]["left"]["rot"]["scaling"][what] *= {"factor": 1.3, "original": 2, "fast": 0.1, "slow": 3.0}[what]
    elif what in ("head norm", "latent norm", "norm behind the mixer", "norm behind the experts", "decay bias", "A_log"):
        name = {"head norm": "l1.mix.right.norm", "latent norm": "l2.mix.dkv.norm", "norm behind the mixer": "l1.norm1b",
                "norm behind the experts": "l0.norm2b", "decay bias": "l1.mix.right.dt_bias", "A_log": "l1.mix.right.A_log"}[what]
        w2[name] = w[name].float().flip(0)
    else:
        block, key, value = {"left scale": (m[1], "left_scale", 0.6), "right scale": (m[1], "right_scale", 1.2), "score scale": (m[1]["left"], "scale", 0.6),
                             "latent scale": (m[2], "scale", 0.6), "retention base": (m[0]["rot"], "base", 200.0), "window": (m[2]["mask"], "size", 12),
                             "rotated dimensions": (m[0]["rot"], "dims", 8), "decay": (m[0], "decay", [0.6, 0.9, 0.95])}[what]
        block[key] = value
    assert rel_err(oracle_logits(cfg2, w2, toks)[10:], want[10:]) > 3e-3, "the oracle does not depend on it"
    got, _ = run(cfg, toks, "float32", cuts=[23, 2, 1], weights=w)
    assert rel_err(got, want) < TOL["float32"]


# ---- prefill == decode, portions -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_equals_token_by_token(dtype):
    toks = rand_tokens(70, SMALL["vocab"], 5)
    w = plain.random_weights(SMALL, 0)
    w = settled(w) if dtype == "bfloat16" else w
    whole, want = run(SMALL, toks, dtype, weights=w)
    single, _ = run(SMALL, toks, dtype, cuts=[1], weights=w)
    assert close(whole, want, dtype)
    assert close(single, want, dtype)
    if dtype == "float32":
        assert close(single, whole)


@pytest.mark.parametrize("cuts", [[2], [3, 2, 7, 1, 16, 5], [17, 2, 2, 31], [33, 1]])
def test_portions(cuts):
    toks = rand_tokens(90, SMALL["vocab"], 7)
    got, want = run(SMALL, toks, "float32", cuts=cuts)
    assert close(got, want)


def test_step_larger_than_the_runner_capacity_is_cut():
    toks = rand_tokens(100, SMALL["vocab"], 8)
    got, want = run(SMALL, toks, "float32", max_step_tokens=32)
    assert close(got, want)


# ---- batches of unequal requests, reuse of pages and slots ------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_and_reuse(dtype):
    w = plain.random_weights(SMALL, 11)
    w = settled(w) if dtype == "bfloat16" else w
    V = SMALL["vocab"]
    reqs = {"a": rand_tokens(50, V, 1), "b": rand_tokens(7, V, 2), "c": rand_tokens(33, V, 3), "d": rand_tokens(1, V, 4),
            "e": rand_tokens(41, V, 5), "f": rand_tokens(20, V, 6)}
    ref = {k: oracle_logits(SMALL, w, v) for k, v in reqs.items()}
    hz = Harness(SMALL, w, dtype=dtype, page_size=16, num_pages=9, slots=3)          # a, c, e cannot be live together
    got = {k: [] for k in reqs}
    at = {k: 0 for k in reqs}

    def step(parts):
        ent = []
        for k, n in parts:
            n = min(n, len(reqs[k]) - at[k])
            ent.append((k, reqs[k][at[k]:at[k] + n], range(n)))
        out = hz.step(ent)
        o = 0
        for k, t, _ in ent:
            got[k].append(out[o:o + len(t)])
            o += len(t)
            at[k] += len(t)
            if at[k] == len(reqs[k]):
                hz.end(k)
    try:
        step([("a", 20), ("b", 3), ("d", 1)])           # d ends: its slot and page are free again
        step([("a", 1), ("b", 2), ("c", 9)])
        step([("c", 24), ("a", 1), ("b", 2)])           # c and b end
        step([("a", 12), ("e", 2)])
        step([("e", 17), ("a", 1), ("f", 5)])
        while at["a"] < 50 or at["e"] < 41 or at["f"] < 20:
            step([(k, 1 if k != "f" else 4) for k in ("a", "e", "f") if at[k] < len(reqs[k])])
        assert len(hz.sched.block_manager.free_block_ids) == 9 and len(hz.sched.state_manager.free_slots) == 3
    finally:
        hz.close()
    for k in reqs:
        assert close(np.concatenate(got[k], 0), ref[k], dtype), k


def test_slot_and_pages_used_again_start_from_the_empty_state():
    w = plain.random_weights(SMALL, 12)
    V = SMALL["vocab"]
    hz = Harness(SMALL, w, "float32", page_size=16, num_pages=4, slots=1)
    try:
        for i in range(3):
            toks = rand_tokens(40 + i, V, 20 + i)
            got = hz.feed("x", toks, cuts=[13, 1])
            hz.end("x")
            assert close(got, oracle_logits(SMALL, w, toks))
    finally:
        hz.close()


# ---- a key that must be found, or must not be: window, keys, states, page borders ---------------------------------------------------
CUTS = {"prompt": lambda n: [n], "decode": lambda n: [n - 30, 1], "portions": lambda n: [5, 2, 3, 17, 2, 6]}


def _find(cfg, w, n, needle_at, visible, how, dtype, page=16, max_step_tokens=512):
    toks, without = needle_tokens(n, needle_at)
    want = oracle_logits(cfg, w, toks)
    changed = rel_err(oracle_logits(cfg, w, without)[-1], want[-1])
    assert (changed > 0.3) if visible else (changed < 1e-9)                       # it decides, or it is hidden
    hz = Harness(cfg, w, dtype, page_size=page, num_pages=-(-n // page), slots=1, max_step_tokens=max_step_tokens)
    try:
        got = hz.feed("n", toks, cuts=CUTS[how](n))
    finally:
        hz.close()
    tol = TOL["float32"] if dtype == "float32" else 4e-2
    assert rel_err(got[-1], want[-1]) < tol
    assert rel_err(got, want) < tol


# asked from position 149 through a window of 24: it sees 126 .. 149
@pytest.mark.parametrize("needle_at", [0, 15, 16, 111, 112, 124, 125, 126, 127, 128, 143, 144, 148])
@pytest.mark.parametrize("how", list(CUTS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_marked_key_is_seen_exactly_inside_the_window(needle_at, how, dtype):
    cfg, w = latent_needle(size=24)
    _find(cfg, w, 150, needle_at, plain.causal(149, needle_at, 24), how, dtype)


@pytest.mark.parametrize("size,n", [(1, 40), (2, 41), (16, 50), (17, 48), (63, 128), (64, 129), (65, 130), (100, 201), (300, 700), (None, 150), (1000, 130)])
def test_windows_of_other_shapes(size, n):
    """A window of one token, of two, equal to the page, around a key tile, over several tiles and key splits, longer than the
    request, none at all; both tensor-core kernels (a cache row of 32 + 32 and one of 48 + 8)."""
    first = 0 if size is None else max(n - size, 0)
    for kw in (dict(rank=32, rot_dim=32, dim=24, heads=4, vdim=24), dict()):
        cfg, w = latent_needle(size=size, **kw)
        for needle_at in sorted({max(first - 1, 0), min(first, n - 2)}):
            for dtype in ("float32", "bfloat16"):
                for how in ("prompt", "decode"):
                    _find(cfg, w, n, needle_at, plain.causal(n - 1, needle_at, size), how, dtype, max_step_tokens=1024)


@pytest.mark.parametrize("needle_at", [0, 299, 300, 301, 311, 312, 320, 575, 576, 610])
def test_window_over_many_tiles_with_key_splits(needle_at):
    """612 tokens, a window of 312 (first seen position 300), in steps of at most 128 tokens: a full step leaves the splits joined,
    decoding cuts them."""
    cfg, w = latent_needle(heads=3, dim=24, rank=72, rot_dim=16, vdim=20, scale=0.5, size=312)
    for how in ("prompt", "decode"):
        _find(cfg, w, 612, needle_at, plain.causal(611, needle_at, 312), how, "bfloat16", page=64, max_step_tokens=128)


@pytest.mark.parametrize("needle_at", [0, 1, 15, 16, 63, 64, 120, 148])
@pytest.mark.parametrize("how", list(CUTS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mixer", ["left", "right", "retention"])
def test_marked_key_far_back_is_found(mixer, needle_at, how, dtype):
    cfg, w = {"left": key_value_needle, "right": delta_needle, "retention": retention_needle}[mixer]()
    _find(cfg, w, 150, needle_at, True, how, dtype)


@pytest.mark.parametrize("needle_at", [0, 255, 256, 511, 610])
def test_far_key_among_hundreds(needle_at):
    cfg, w = key_value_needle(heads=6, kv_heads=2, dim=40, rot_dims=16, scale=2.0)
    for how in ("prompt", "decode"):
        _find(cfg, w, 612, needle_at, True, how, "bfloat16", page=64, max_step_tokens=1024)


@pytest.mark.parametrize("which", ["latent", "left", "retention"])
def test_rotation_decides_where_keys_differ_only_by_position(which):
    """Only the rotated dimensions enter the scores, hundreds of tokens from the start."""
    if which == "latent":
        cfg = model_config([lat(heads=2, dim=8, rot_dim=16, rank=24, scale=1.2, base=1000.0, size=200, mlp=None)])
        w = plain.random_weights(cfg, 21)
        w["l0.mix.uk"] = torch.zeros_like(w["l0.mix.uk"].float())
        w["l0.mix.q"] = w["l0.mix.q"].float() * 3.0
    elif which == "left":
        cfg = model_config([par(dims=16, base=1000.0, scale=0.8, mlp=None)])
        w = silent(plain.random_weights(cfg, 22), "l0.mix.right.o")
    else:
        cfg = model_config([ret(dim=16, base=1000.0, decay=[0.995, 0.9, 0.999], mlp=None)])
        w = plain.random_weights(cfg, 23)
    toks = rand_tokens(500, cfg["vocab"], 22)
    for dtype, worst, mean in (("float32", TOL["float32"], TOL["float32"]), ("bfloat16", 1.2e-1, 1.5e-2)):      # sharp scores: bf16 keys and
        got, want = run(cfg, toks, dtype, cuts=[470, 1], weights=w, page_size=64, num_pages=8)                  # queries show in single rows
        e = row_errs(got, want)
        assert e.max() < worst and e.mean() < mean


def test_convolution_sees_its_taps_across_every_cut():
    """Content at one token shows in the next taps - 1 tokens: fed so that the cut falls before, on and behind it."""
    cfg, w = delta_needle(conv=4)
    w["l0.mix.right.v.conv"] = torch.tensor([[0.9, -0.7, 0.5, 1.0]]).repeat(w["l0.mix.right.v"].shape[0], 1)
    w["l0.mix.right.k.conv"] = torch.tensor([[0.3, 0.4, -0.5, 1.0]]).repeat(w["l0.mix.right.k"].shape[0], 1)
    toks, _ = needle_tokens(40, 20)
    toks[21] = toks[22] = toks[23] = 61
    want = oracle_logits(cfg, w, toks)
    for cuts in ([40], [21, 1], [20, 1, 2, 3], [19, 2, 2], [1]):
        for dtype in ("float32", "bfloat16"):
            hz = Harness(cfg, w, dtype, page_size=16, num_pages=3, slots=1)
            try:
                got = hz.feed("n", toks, cuts=cuts)
            finally:
                hz.close()
            assert rel_err(got, want) < (TOL["float32"] if dtype == "float32" else 4e-2)


# ---- the first tokens, long decoding, other sizes --------------------------------------------------------------------------------
@pytest.mark.parametrize("n", [1, 2, 3, 5])
def test_first_tokens(n):
    toks = rand_tokens(n, SMALL["vocab"], 40 + n)
    got, want = run(SMALL, toks, "float32")
    assert close(got, want)
    single, _ = run(SMALL, toks, "float32", cuts=[1])
    assert close(single, want)


def test_long_decoding():
    toks = rand_tokens(260, SMALL["vocab"], 50)
    got, want = run(SMALL, toks, "float32", cuts=[4, 1], num_pages=20)
    assert close(got, want)
    got, want = run(SMALL, toks, "bfloat16", cuts=[4, 1], num_pages=20, weights=settled(plain.random_weights(SMALL, 0)))
    assert close(got, want, "bfloat16")


OTHER = [
    # everything equal to one where it can be: heads, head sizes, a window of one, one tap, one expert, nothing rotated in one layer
    model_config([ret(heads=1, dim=1, vdim=1, dims=0, mlp=moe(1, 1, 1, None, None)),
                  par(heads=1, kv_heads=1, dim=2, dims=2, d_heads=1, d_kv_heads=1, d_dim=1, d_vdim=1, conv=1, mlp=None),
                  lat(heads=1, dim=1, rot_dim=2, vdim=1, rank=1, size=1, mlp=moe(1, 1, 3, 1, (2, 1)))], width=24, vocab=50),
    # sizes the tensor-core paths take, the wider attention tiles, unlike rotations
    model_config([ret(heads=4, dim=64, vdim=48, mlp=moe(16, 4, 32, 4, (5, 3))),
                  par(heads=4, kv_heads=4, dim=72, dims=48, scale=0.1, d_heads=6, d_kv_heads=3, d_dim=64, d_vdim=40, mlp=moe(12, 3, 40, 3, (5, 2))),
                  lat(heads=8, dim=24, rot_dim=16, vdim=40, rank=48, size=20), par(heads=2, kv_heads=1, dim=128, dims=64, scale=0.08, scaling=None, d_heads=2,
                                                                                   d_kv_heads=2, d_dim=128, d_vdim=104, conv=6, mlp=None),
                  lat(heads=4, dim=40, rot_dim=32, vdim=24, rank=32, size=33, mlp=None)], width=72, vocab=130, eps=1e-6),
    # nothing a multiple of 8; head sizes beyond a warp; partly rotated heads whose pairs are no multiple of a vector
    model_config([ret(heads=2, dim=33, vdim=70, dims=22, mlp=moe(3, 2, 13, 1, (2, 2))), lat(heads=5, dim=20, rot_dim=6, vdim=33, rank=37, size=7),
                  par(heads=6, kv_heads=2, dim=20, dims=10, d_heads=5, d_kv_heads=1, d_dim=33, d_vdim=70, conv=5, mlp=moe(6, 1, 11, 5, (1, 1))),
                  ret(heads=1, dim=144, vdim=9, dims=36, mlp=None)], width=44, vocab=61),
    # large recurrence heads (each register layout of both recurrences)
    model_config([ret(heads=1, dim=96, vdim=40, dims=96, mlp=None), ret(heads=2, dim=200, vdim=24, dims=104, mlp=None),
                  ret(heads=1, dim=400, vdim=16, dims=400, mlp=None), ret(heads=1, dim=640, vdim=12, dims=64, mlp=None),
                  par(dim=8, dims=4, d_heads=2, d_kv_heads=1, d_dim=96, d_vdim=24, mlp=None), par(dim=8, dims=4, d_heads=1, d_kv_heads=1, d_dim=200, d_vdim=40, mlp=None),
                  par(dim=8, dims=4, d_heads=2, d_kv_heads=2, d_dim=400, d_vdim=16, mlp=None), par(dim=8, dims=4, d_heads=1, d_kv_heads=1, d_dim=640, d_vdim=12, mlp=None)],
                 width=56, vocab=64),
]


@pytest.mark.parametrize("idx", range(len(OTHER)))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes(idx, dtype):
    cfg = OTHER[idx]
    toks = rand_tokens(60, cfg["vocab"], 60 + idx)
    w = plain.random_weights(cfg, 0)
    got, want = run(cfg, toks, dtype, cuts=[41, 3, 1], weights=settled(w) if dtype == "bfloat16" else w, page_size=32, num_pages=4)
    assert close(got, want, dtype)


# layer-sized models (the tensor-core products, attention tiles and sorted experts take over in the bf16 build): unlike head
# shapes, windows over several 64-token pages and inside one, feed-forwards beside every mixer
LAYER_SIZED = [
    model_config([lat(heads=4, dim=48, rot_dim=32, vdim=40, rank=96, scale=0.11, base=10000.0, size=100, mlp=moe(10, 2, 96, 2, (4, 2))),
                  ret(heads=5, dim=48, vdim=64, base=10000.0, mlp=moe(8, 2, 96, 4, (2, 1))),
                  par(heads=8, kv_heads=2, dim=40, dims=24, scale=0.16, base=10000.0, d_heads=6, d_kv_heads=3, d_dim=48, d_vdim=64, conv=4,
                      mlp=moe(9, 3, 64, 0, (3, 2))),
                  ret(heads=2, dim=128, vdim=96, dims=64, mlp=None), lat(heads=3, dim=40, rot_dim=24, vdim=56, rank=130, scale=0.12, size=48, mlp=moe(30, 5, 40, 10, (4, 2)))],
                 width=320, vocab=300),
    model_config([par(heads=3, kv_heads=1, dim=80, dims=80, scale=0.11, scaling=None, d_heads=2, d_kv_heads=2, d_dim=112, d_vdim=80, mlp=None),
                  ret(heads=3, dim=24, vdim=88, mlp=moe(7, 3, 50, 2, (3, 2))),
                  lat(heads=6, dim=40, rot_dim=24, vdim=40, rank=40, scale=0.12, base=5000.0, size=257, mlp=moe(6, 2, 72, 0, None))], width=200, vocab=333),
]


@pytest.mark.parametrize("idx", range(len(LAYER_SIZED)))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_sized_models_through_a_randomly_cut_mixed_schedule(idx, dtype):
    """Six requests, four slots, pages for the four longest only: portions of changing size beside single tokens, a request now
    and then left out of a step, the last 30 tokens of each one by one."""
    import random
    cfg = LAYER_SIZED[idx]
    w = plain.random_weights(cfg, 90 + idx)
    w = settled(w) if dtype == "bfloat16" else w
    V = cfg["vocab"]
    lens = [300, 230, 64, 5, 270, 129]
    reqs = {f"r{i}": rand_tokens(n, V, 91 + i) for i, n in enumerate(lens)}
    ref = {k: oracle_logits(cfg, w, v) for k, v in reqs.items()}
    pages = sum(-(-n // 64) for n in sorted(lens)[-4:])
    hz = Harness(cfg, w, dtype=dtype, page_size=64, num_pages=pages, slots=4, max_step_tokens=2048)
    rng = random.Random(7 + idx)
    got, at, live, waiting = {k: [] for k in reqs}, {k: 0 for k in reqs}, [], list(reqs)
    try:
        while live or waiting:
            while waiting and len(live) < 4:
                live.append(waiting.pop(0))
            ent = []
            for k in live:
                if len(live) > 1 and rng.random() < 0.15:
                    continue
                left = len(reqs[k]) - at[k]
                n = min(rng.choice([2, 3, 17, 64, 65, 100, 129]), left - 30) if left > 30 else 1
                ent.append((k, reqs[k][at[k]:at[k] + n], range(n)))
            if not ent:
                continue
            out = hz.step(ent)
            o = 0
            for k, t, _ in ent:
                got[k].append(out[o:o + len(t)])
                o += len(t)
                at[k] += len(t)
                if at[k] == len(reqs[k]):
                    hz.end(k)
                    live.remove(k)
        assert len(hz.sched.block_manager.free_block_ids) == pages and len(hz.sched.state_manager.free_slots) == 4
    finally:
        hz.close()
    e = np.concatenate([row_errs(np.concatenate(got[k], 0), ref[k]) for k in reqs])
    assert close(np.concatenate([np.concatenate(got[k], 0) for k in reqs]), np.concatenate([ref[k] for k in reqs]), dtype), (e.max(), np.median(e))


# ---- greedy generation through the engine's own entry points ------------------------------------------------------------------------
def _greedy_ok(cfg, w, prompt, ids):
    seq = list(prompt)
    for tok in ids:
        lg = oracle_logits(cfg, w, seq)[-1]
        assert tok == int(np.argmax(lg)) or lg.max() - lg[tok] < 1e-3 * (lg.max() - lg.min()), "not the oracle's greedy token"
        seq.append(tok)


def test_greedy_generation_through_llm_generate():
    from jacobiforcing_b200 import LLM, SamplingParams
    from jacobiforcing_b200.hybrid_config import HybridConfig
    w = plain.random_weights(SMALL, 70)
    llm = LLM(None, hf_config=HybridConfig.from_dict(SMALL), state_dict=w, dtype="float32", kvcache_block_size=16, num_kvcache_blocks=16,
              max_num_seqs=2, max_model_len=128, max_num_batched_tokens=24)
    V = SMALL["vocab"]
    prompts = [rand_tokens(30, V, 71), rand_tokens(5, V, 72), rand_tokens(17, V, 73)]      # three requests, two slots,
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True), use_tqdm=False)
    llm.exit()                                                                               # prompts cut at 24 tokens
    for prompt, out in zip(prompts, outs):
        assert len(out["token_ids"]) == 8
        _greedy_ok(SMALL, w, prompt, out["token_ids"])


def test_generate_command_line_and_trace_replay_on_a_checkpoint_directory(tmp_path):
    import json
    import os
    import subprocess
    import sys
    from tests.test_hybrid_host import _write_checkpoint
    w = plain.random_weights(SMALL, 75)
    _write_checkpoint(tmp_path, SMALL, w)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    prompt = rand_tokens(21, SMALL["vocab"], 76)
    out = subprocess.run([sys.executable, "-m", "jacobiforcing_b200.generate", "--model", str(tmp_path), "--prompt-ids",
                          ",".join(map(str, prompt)), "--max-tokens", "6", "--dtype", "float32", "--page-size", "16",
                          "--max-model-len", "64", "--max-num-batched-tokens", "64"], cwd=root, capture_output=True, text=True)
    assert out.returncode == 0, out.stderr[-2000:]
    _greedy_ok(SMALL, w, prompt, json.loads(out.stdout.strip().splitlines()[-1])["token_ids"])
    # trace replay: two requests, portions beside single tokens, one ends and its slot and pages are used again
    a, b = rand_tokens(30, SMALL["vocab"], 77), rand_tokens(9, SMALL["vocab"], 78)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": [0, 16]}, {"id": "b", "tokens": b[:2], "want": [1]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": [6]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[17:18], "want": [0]}, {"id": "c", "tokens": b, "want": [8]}], "end": ["c"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[18:], "want": []}], "end": ["a"]}]
    outdir = tmp_path / "out"
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(outdir), "--max-tokens", "128", "--page-size", "16"], input="\n".join(json.dumps(x) for x in steps) + "\n",
                       cwd=root, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    la, lb = oracle_logits(SMALL, w, a), oracle_logits(SMALL, w, b)
    V = SMALL["vocab"]
    g0 = np.fromfile(outdir / "0.f32", dtype="<f4").reshape(-1, V)
    g1 = np.fromfile(outdir / "1.f32", dtype="<f4").reshape(-1, V)
    g2 = np.fromfile(outdir / "2.f32", dtype="<f4").reshape(-1, V)
    assert not (outdir / "3.f32").exists()
    assert rel_err(g0, np.stack([la[0], la[16], lb[1]])) < TOL["float32"]
    assert rel_err(g1, lb[8:9]) < TOL["float32"]
    assert rel_err(g2, np.stack([la[17], lb[8]])) < TOL["float32"]
