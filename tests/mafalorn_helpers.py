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


TOL = {"float32": 2e-4, "bfloat16": 6e-2}


def close(got, want, dtype="float32", skip=()) -> bool:
    """float32: every row within the tolerance.  bfloat16: the rows in `skip` are not judged (see near_ties); of the others a
    fifth may lie outside (typical rows are several times below the tolerance)."""
    e = row_errs(got, want)
    if dtype == "float32":
        return bool(e.max() < TOL[dtype])
    keep = np.ones(len(e), dtype=bool)
    keep[[i for i in skip if i < len(e)]] = False
    if not keep.any():
        return True
    e = e[keep]
    return bool(np.mean(e < TOL[dtype]) >= 0.8 and np.median(e) < TOL[dtype] / 2)


def near_ties(config, weights, tokens, margin=0.01):
    """Rows where the last chosen and the first rejected output, or the last kept and the first dropped group, lie closer than
    `margin` in the oracle: a run with rounding may choose the other one."""
    found = []
    inner = plain.route

    def watching(h, router, correction, r):
        choice = torch.softmax(h @ router.T, 1) + correction
        n, gr = choice.shape[1], r.get("groups") or {"count": 1, "keep": 1}
        worth = choice.reshape(-1, gr["count"], n // gr["count"]).max(2).values
        z, keep = torch.sort(worth, 1, descending=True)
        if gr["keep"] < gr["count"]:
            found.extend(torch.nonzero(z[:, gr["keep"] - 1] - z[:, gr["keep"]] < margin).flatten().tolist())
        for t in range(choice.shape[0]):
            c = torch.sort(choice[t].reshape(gr["count"], -1)[keep[t, :gr["keep"]]].flatten(), descending=True).values
            if r["top"] < len(c) and c[r["top"] - 1] - c[r["top"]] < margin:
                found.append(t)
        return inner(h, router, correction, r)
    plain.route = watching
    try:
        plain.forward(config, weights, list(tokens))
    finally:
        plain.route = inner
    return sorted(set(found))


def run(config, tokens, dtype="float32", cuts=None, seed=0, weights=None, **kw):
    w = weights if weights is not None else plain.random_weights(config, seed)
    hz = Harness(config, w, dtype=dtype, **kw)
    try:
        got = hz.feed("a", tokens, cuts)
    finally:
        hz.close()
    return got, oracle_logits(config, w, tokens)
