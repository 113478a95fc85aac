"""Shared pieces of the Mafalorn tests: small configurations (sizes chosen unequal on purpose: key and value sizes differ, fewer
key heads than query heads, a window that is no multiple of the page), random bf16 weights from the plain oracle, one-layer
models in which one marked token decides the answer, and the error measures.  The engine is driven through
tests.hybrid_helpers.Harness (scheduler + runner)."""
from __future__ import annotations

import copy

import numpy as np
import torch

from oracle import mafalorn_plain as plain
from tests.hybrid_helpers import Harness, rand_tokens, rel_err  # noqa: F401  (re-exported)


def moe(experts=7, top=3, ff=24, identity=2, groups=(3, 2)):
    r = {"experts": experts, "top": top}
    if identity is not None:
        r["identity"] = identity
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def _mlp(mlp):
    return moe() if mlp == "default" else mlp


def ret(heads=3, dim=12, vdim=20, decay=None, base=400.0, dims=None, mlp="default"):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                                           "decay": list(decay) if decay else [1.0 - 2.0 ** (-2.0 - 1.3 * h) for h in range(heads)],
                                           "rot": {"base": base, "dims": dim if dims is None else dims}}, "mlp": _mlp(mlp)}


SCALING = {"factor": 5.0, "original": 40, "fast": 8.0, "slow": 0.5}


def par(heads=4, kv_heads=2, dim=16, scale=0.4, base=200.0, dims=12, scaling=SCALING, d_heads=4, d_kv_heads=2, d_dim=12, d_vdim=20, conv=3,
        left_scale=0.7, right_scale=1.3, mlp="default"):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(scaling)
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "rot": rot}, "left_scale": left_scale,
                      "right": {"heads": d_heads, "kv_heads": d_kv_heads, "dim": d_dim, "vdim": d_vdim, "conv": conv}, "right_scale": right_scale},
            "mlp": _mlp(mlp)}


def lat(heads=3, dim=16, rot_dim=8, vdim=12, rank=24, size=11, base=300.0, scale=0.4, mlp="default"):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if size is not None:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m, "mlp": _mlp(mlp)}


def model_config(layers, width=40, vocab=70, eps=2e-5, logit_scale=0.7):
    return {"architecture": "Mafalorn", "layers": copy.deepcopy(layers), "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "logit_scale": logit_scale}


# every mixer with and without a feed-forward, two layers of a kind with unlike sizes and rotations
SMALL = model_config([ret(mlp=moe(4, 1, 16, 2, (2, 1))), par(), lat(), ret(heads=2, dim=20, vdim=8, base=90.0, dims=16, mlp=None),
                      par(heads=6, kv_heads=2, dim=24, dims=24, scaling=None, d_heads=3, d_kv_heads=1, d_dim=20, d_vdim=12, conv=4, mlp=None),
                      lat(heads=2, dim=8, rot_dim=12, vdim=20, rank=16, size=19, mlp=moe(3, 3, 8, 1, None))])


def oracle_logits(config, weights, tokens, dtype=torch.float64):
    return plain.forward(config, weights, list(tokens), dtype=dtype).numpy()


def row_errs(got: np.ndarray, want: np.ndarray) -> np.ndarray:
    """Per row: root mean square of the centred difference over the centred reference."""
    got, want = np.atleast_2d(got).astype(np.float64), np.atleast_2d(want).astype(np.float64)
    d = got - want
    d = d - d.mean(1, keepdims=True)
    w = want - want.mean(1, keepdims=True)
    return np.sqrt((d ** 2).mean(1)) / np.sqrt((w ** 2).mean(1) + 1e-30)


TOL = {"float32": 2e-4, "bfloat16": 8e-2}


def close(got, want, dtype="float32") -> bool:
    """float32: every row within the tolerance.  bfloat16: one row in twenty (at least one) may lie outside, up to four times: a
    sublayer whose result happens to be small is normed up, rounding and all.  Runs of models with routers use `settled`
    weights there: rounding may choose another expert at a near tie, and every later row sees it through states and keys."""
    e = row_errs(got, want)
    if dtype == "float32":
        return bool(e.max() < TOL[dtype])
    return bool(np.sum(e >= TOL[dtype]) <= max(1, 0.05 * len(e)) and e.max() < 4 * TOL[dtype] and np.median(e) < TOL[dtype] / 1.5)


def settled(weights):
    """The same weights with corrections so large that they alone decide the choice of experts: no rounding can flip it."""
    return {k: (v.float() * 1000.0 if k.endswith(".correction") else v) for k, v in weights.items()}


def run(config, tokens, dtype="float32", cuts=None, seed=0, weights=None, **kw):
    w = weights if weights is not None else plain.random_weights(config, seed)
    hz = Harness(config, w, dtype=dtype, **kw)
    try:
        got = hz.feed("a", tokens, cuts)
    finally:
        hz.close()
    return got, oracle_logits(config, w, tokens)


# ---- one-layer models in which token 61 asks for token 60 ------------------------------------------------------------------------
# The stream's first quarter is a token's key address, the second quarter its query address, the second half its content.
# Only token 60 has a key address; token 61's query address is token 60's key address.  Everything that is not needed to
# find the marked token is zero, so its content decides the answer wherever it may be seen, and changes nothing elsewhere.
def _addresses(w, width, g):
    q4, half = width // 4, width // 2
    e = w["embed"].float()
    e[:, :half] = 0.0
    e[60, :q4] = torch.randn(q4, generator=g)
    e[61, q4:half] = e[60, :q4]
    e[60, half:] *= 3.0
    w["embed"] = e.to(torch.bfloat16)
    w["l0.norm1"] = torch.ones(width)
    return q4, half


def _set(w, name, t):
    w["l0.mix." + name] = t.to(torch.bfloat16).float()


def latent_needle(heads=2, dim=32, vdim=16, rank=48, rot_dim=8, size=24, width=64, scale=0.4):
    """The latent's first third holds the address, the rest the content; the rotated part is out of the way (zero)."""
    cfg = model_config([lat(heads=heads, dim=dim, vdim=vdim, rank=rank, rot_dim=rot_dim, size=size, scale=scale, mlp=None)], width=width, vocab=64)
    w = plain.random_weights(cfg, 33)
    g = torch.Generator().manual_seed(34)
    q4, half = _addresses(w, width, g)
    third = rank // 3
    m = torch.randn(third, q4, generator=g) * 2.0
    dkv = torch.zeros(rank + rot_dim, width)
    dkv[:third, :q4] = m
    dkv[third:rank, half:] = torch.randn(rank - third, half, generator=g) / half ** 0.5
    uk = torch.zeros(heads * dim, rank)
    uk[:, :third] = torch.randn(heads * dim, third, generator=g) / third ** 0.5
    uv = torch.zeros(heads * vdim, rank)
    uv[:, third:] = torch.randn(heads * vdim, rank - third, generator=g) / rank ** 0.5
    wq = torch.zeros(heads * (dim + rot_dim), width)
    for h in range(heads):
        wq[h * (dim + rot_dim):h * (dim + rot_dim) + dim, q4:half] = uk[h * dim:(h + 1) * dim, :third] @ m
    for k, v in {"q": wq, "dkv": dkv, "dkv.norm": torch.ones(rank), "uk": uk, "uv": uv}.items():
        _set(w, k, v)
    return cfg, w


def key_value_needle(heads=2, kv_heads=1, dim=32, rot_dims=8, width=64, scale=1.5):
    """The key's rotated dimensions are zero, half of the others hold the address, the rest content that no query reads; the
    right-hand mixer's output is zero."""
    cfg = model_config([par(heads=heads, kv_heads=kv_heads, dim=dim, dims=rot_dims, scale=scale, left_scale=1.0, mlp=None)], width=width, vocab=64)
    w = plain.random_weights(cfg, 37)
    g = torch.Generator().manual_seed(38)
    q4, half = _addresses(w, width, g)
    a = (dim - rot_dims) // 2                                    # address dimensions behind the rotated ones
    m = torch.randn(kv_heads, a, q4, generator=g)
    wk = torch.zeros(kv_heads, dim, width)
    wk[:, rot_dims:rot_dims + a, :q4] = m
    wk[:, rot_dims + a:, half:] = torch.randn(kv_heads, dim - rot_dims - a, half, generator=g) / half ** 0.5
    wq = torch.zeros(heads, dim, width)
    for h in range(heads):
        wq[h, rot_dims:rot_dims + a, q4:half] = m[h // (heads // kv_heads)]
    _set(w, "left.q", wq.reshape(-1, width))
    _set(w, "left.k", wk.reshape(-1, width))
    _set(w, "right.o", torch.zeros_like(w["l0.mix.right.o"].float()))
    return cfg, w


def retention_needle(heads=2, dim=16, vdim=24, width=64):
    """Decays near one and nothing rotated but two dimensions that stay zero, so the one key written stays readable far away."""
    cfg = model_config([ret(heads=heads, dim=dim, vdim=vdim, decay=[1.0 - 2.0 ** -10, 1.0][:heads], dims=2, mlp=None)], width=width, vocab=64)
    w = plain.random_weights(cfg, 35)
    g = torch.Generator().manual_seed(36)
    q4, half = _addresses(w, width, g)
    m = torch.randn(heads, dim, q4, generator=g)
    m[:, :2] = 0.0
    wk, wq = torch.zeros(heads * dim, width), torch.zeros(heads * dim, width)
    wk[:, :q4] = m.reshape(-1, q4)
    wq[:, q4:half] = m.reshape(-1, q4)
    wv = torch.zeros(heads * vdim, width)
    wv[:, half:] = torch.randn(heads * vdim, half, generator=g) / half ** 0.5
    _set(w, "q", wq)
    _set(w, "k", wk)
    _set(w, "v", wv)
    return cfg, w


def delta_needle(heads=2, kv_heads=1, dim=16, vdim=24, conv=3, width=64):
    """Decays near one, convolutions that pass the current token only; the left-hand mixer's output is zero."""
    cfg = model_config([par(d_heads=heads, d_kv_heads=kv_heads, d_dim=dim, d_vdim=vdim, conv=conv, right_scale=1.0, mlp=None)], width=width, vocab=64)
    w = plain.random_weights(cfg, 39)
    g = torch.Generator().manual_seed(40)
    q4, half = _addresses(w, width, g)
    m = torch.randn(kv_heads * dim, q4, generator=g)
    wk, wq = torch.zeros(kv_heads * dim, width), torch.zeros(kv_heads * dim, width)
    wk[:, :q4] = m
    wq[:, q4:half] = m
    wv = torch.zeros(heads * vdim, width)
    wv[:, half:] = torch.randn(heads * vdim, half, generator=g) / half ** 0.5
    for name, t in (("q", wq), ("k", wk), ("v", wv)):
        _set(w, f"right.{name}", t)
        taps = torch.zeros(t.shape[0], conv)
        taps[:, -1] = 1.0
        _set(w, f"right.{name}.conv", taps)
    _set(w, "right.A_log", torch.full((heads,), -9.0))
    _set(w, "right.a", torch.zeros(heads, width))
    _set(w, "right.dt_bias", torch.zeros(heads))
    _set(w, "left.o", torch.zeros_like(w["l0.mix.left.o"].float()))
    return cfg, w


def needle_tokens(n, needle_at):
    """(tokens with the marked token and the asking token last, the same without the marked token)."""
    toks = [2 + (i % 50) for i in range(n)]
    without = list(toks)
    toks[needle_at] = 60
    toks[-1] = without[-1] = 61
    return toks, without
