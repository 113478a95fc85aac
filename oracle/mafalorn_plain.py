"""Plain, slow restatement of the Mafalorn design: a decoder over one residual stream with an RMS norm (plain weight) on both
sides of every sublayer, x <- x + n1b(mixer(n1(x))), then x <- x + n2b(ff(n2(x))).  Mixers: retention (linear attention with
one fixed decay per head, rotated queries and keys), a pair of mixers side by side (softmax attention whose values are its
unrotated keys, with an interpolated rotation and one output gate per head, beside a gated delta rule with one decay per head),
and attention over a low-rank latent inside a sliding window with an element-wise output gate.  Feed-forward: gated silu
experts chosen inside the best groups by corrected softmax scores, some of which pass their input through.

One function per mechanism, whole sequences only, plain torch on the CPU: every token of a sequence from position 0, no
cache, no state hand-over, no batching.  It shares no code with the product path.

Notation: T tokens, W width, weights are [out, in] and applied as x @ w.T; `p` maps a sublayer's tensor leaf name ("q",
"right.k.conv", "dkv.norm", ...) to its tensor, `c` is the sublayer's block of the configuration, `eps` the norms' constant.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

DT = torch.float64


# ---- elementary pieces -------------------------------------------------------------------------------------------
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_vector(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# ---- rotations -----------------------------------------------------------------------------------------------------
def frequencies(rot: dict) -> List[float]:
    """base^(-2 i / dims); with a scaling, frequencies are interpolated between the pair indices where a pair turns `fast` and
    `slow` times over the original length."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f
    at = lambda turns: dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(at(float(sc["fast"]))), 0)
    hi = min(math.ceil(at(float(sc["slow"]))), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / float(sc["factor"]) * ramp + x * (1.0 - ramp))
    return out


def magnitude(rot: dict) -> float:
    sc = rot.get("scaling")
    return 0.1 * math.log(float(sc["factor"])) + 1.0 if sc else 1.0


def half_pairs(dims: int) -> List[tuple]:
    return [(i, i + dims // 2) for i in range(dims // 2)]


def neighbour_pairs(dims: int) -> List[tuple]:
    return [(2 * i, 2 * i + 1) for i in range(dims // 2)]


def rotate_all(x: torch.Tensor, rot: dict, pairs: List[tuple]) -> torch.Tensor:
    """x [T, ...]: row t turns by its position t; dimensions beyond the pairs pass unchanged."""
    out, m = x.clone(), magnitude(rot)
    pos = torch.arange(x.shape[0], dtype=DT).reshape([-1] + [1] * (x.ndim - 2))
    for (i, j), f in zip(pairs, frequencies(rot)):
        c, s = (torch.cos(pos * f) * m).to(x.dtype), (torch.sin(pos * f) * m).to(x.dtype)
        out[..., i] = x[..., i] * c - x[..., j] * s
        out[..., j] = x[..., j] * c + x[..., i] * s
    return out


# ---- retention -----------------------------------------------------------------------------------------------------
def head_decays(c: dict) -> torch.Tensor:
    return torch.tensor([float(x) for x in c["decay"]], dtype=DT)


def retention(h: torch.Tensor, p: Dict[str, torch.Tensor], c: dict, eps: float) -> torch.Tensor:
    T, H, D, Dv = h.shape[0], c["heads"], c["dim"], c["vdim"]
    pairs = half_pairs(int(c["rot"]["dims"]))
    q = rotate_all((h @ p["q"].T).reshape(T, H, D), c["rot"], pairs)
    k = rotate_all((h @ p["k"].T).reshape(T, H, D), c["rot"], pairs) * D ** -0.5
    v = (h @ p["v"].T).reshape(T, H, Dv)
    a = head_decays(c).to(h.dtype)[:, None, None]
    S = torch.zeros(H, D, Dv, dtype=h.dtype)
    o = torch.zeros(T, H, Dv, dtype=h.dtype)
    for t in range(T):
        S = a * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)                       # the read-out sees the current token's write
    return (unit_rms(o, eps).reshape(T, H * Dv) * silu(h @ p["g"].T)) @ p["o"].T


# ---- attention whose values are its unrotated keys -------------------------------------------------------------------
def causal(i, j, size: Optional[int] = None):
    """Whether position i sees position j (numbers or tensors)."""
    return j <= i if size is None else (j <= i) & (i - j < size)


def softmax_seen(s: torch.Tensor, size: Optional[int] = None) -> torch.Tensor:
    at = torch.arange(s.shape[0])
    s = torch.where(causal(at[:, None], at[None, :], size), s, torch.tensor(-math.inf, dtype=s.dtype))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def key_valued_attention(h: torch.Tensor, p: Dict[str, torch.Tensor], c: dict) -> torch.Tensor:
    T, H, G, D = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    pairs = half_pairs(int(c["rot"]["dims"]))
    k = (h @ p["k"].T).reshape(T, G, D)
    q = rotate_all((h @ p["q"].T).reshape(T, H, D), c["rot"], pairs)
    kr = rotate_all(k, c["rot"], pairs)
    gate = sigmoid(h @ p["g"].T)                                       # one number per head
    out = []
    for hh in range(H):
        g = hh // (H // G)
        w = softmax_seen(q[:, hh] @ kr[:, g].T * float(c["scale"]))
        out.append(w @ k[:, g] * gate[:, hh:hh + 1])                   # the value is the key before its rotation
    return torch.cat(out, 1) @ p["o"].T


# ---- gated delta rule, one decay per head ----------------------------------------------------------------------------
def short_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """silu of a causal convolution over time per channel; w [channels, taps], the last tap is the current token's."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for i in range(taps):
            s = t - (taps - 1) + i
            if s >= 0:
                y[t] += w[:, i] * x[s]
    return silu(y)


def delta_decay(h: torch.Tensor, p: Dict[str, torch.Tensor]) -> torch.Tensor:
    return torch.exp(-torch.exp(p["A_log"]) * softplus(h @ p["a"].T + p["dt_bias"]))


def delta_rule(h: torch.Tensor, p: Dict[str, torch.Tensor], c: dict, eps: float) -> torch.Tensor:
    T, H, G, D, Dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = unit_vector(short_conv(h @ p["q"].T, p["q.conv"]).reshape(T, G, D)) * D ** -0.5
    k = unit_vector(short_conv(h @ p["k"].T, p["k.conv"]).reshape(T, G, D))
    v = short_conv(h @ p["v"].T, p["v.conv"]).reshape(T, H, Dv)
    beta, g = sigmoid(h @ p["b"].T), delta_decay(h, p)
    o = torch.zeros(T, H, Dv, dtype=h.dtype)
    for hh in range(H):
        gh = hh // (H // G)
        S = torch.zeros(D, Dv, dtype=h.dtype)
        for t in range(T):
            S = g[t, hh] * S
            u = beta[t, hh] * (v[t, hh] - S.T @ k[t, gh])
            S = S + torch.outer(k[t, gh], u)
            o[t, hh] = S.T @ q[t, gh]                                  # after the write
    o = unit_rms(o, eps) * p["norm"]
    return (o.reshape(T, H * Dv) * silu(h @ p["g"].T)) @ p["o"].T


def side_by_side(h: torch.Tensor, p: Dict[str, torch.Tensor], c: dict, eps: float) -> torch.Tensor:
    part = lambda side: {k[len(side) + 1:]: v for k, v in p.items() if k.startswith(side + ".")}
    return (float(c["left_scale"]) * key_valued_attention(h, part("left"), c["left"]) +
            float(c["right_scale"]) * delta_rule(h, part("right"), c["right"], eps))


# ---- attention over a latent inside a window ----------------------------------------------------------------------------
def latent_attention(h: torch.Tensor, p: Dict[str, torch.Tensor], c: dict, eps: float) -> torch.Tensor:
    T, H, D, Rt, Dv, K = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    pairs = neighbour_pairs(int(c["rot"]["dims"]))
    q = (h @ p["q"].T).reshape(T, H, D + Rt)
    d = h @ p["dkv"].T
    lat = unit_rms(d[:, :K], eps) * p["dkv.norm"]
    kr = rotate_all(d[:, K:], c["rot"], pairs)
    qr = rotate_all(q[:, :, D:], c["rot"], pairs)
    kn = (lat @ p["uk"].T).reshape(T, H, D)
    v = (lat @ p["uv"].T).reshape(T, H, Dv)
    size = (c.get("mask") or {}).get("size")
    out = []
    for hh in range(H):
        s = (q[:, hh, :D] @ kn[:, hh].T + qr[:, hh] @ kr.T) * float(c["scale"])
        out.append(softmax_seen(s, size) @ v[:, hh])
    return (torch.cat(out, 1) * sigmoid(h @ p["g"].T)) @ p["o"].T


# ---- feed-forward -----------------------------------------------------------------------------------------------------
def gated(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def group_score(choice: List[float]) -> float:
    return max(choice)


def route(h: torch.Tensor, router: torch.Tensor, correction: torch.Tensor, r: dict):
    """Per token: the best groups by group_score of the choice scores (softmax score + correction), in them the outputs with the
    largest choice scores (ties to the lower index); weights = the plain scores, not renormalised."""
    z = h @ router.T
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    choice = s + correction
    n, top = z.shape[1], int(r["top"])
    gr = r.get("groups") or {"count": 1, "keep": 1}
    per = n // int(gr["count"])
    ids = []
    for t in range(h.shape[0]):
        c = [float(x) for x in choice[t]]
        worth = [group_score(c[g * per:(g + 1) * per]) for g in range(int(gr["count"]))]
        kept = sorted(range(len(worth)), key=lambda g: (-worth[g], g))[:int(gr["keep"])]
        open_ = [e for g in kept for e in range(g * per, (g + 1) * per)]
        ids.append(sorted(open_, key=lambda e: (-c[e], e))[:top])
    return ids, [torch.stack([s[t, e] for e in ids[t]]) for t in range(h.shape[0])]


def experts(h: torch.Tensor, p: Dict[str, torch.Tensor], c: dict) -> torch.Tensor:
    n = int(c["router"]["experts"])
    ids, wts = route(h, p["router"], p["correction"], c["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(ids[t], wts[t]):
            out[t] += w * (h[t] if e >= n else gated(h[t], p[f"e{e}.gate"], p[f"e{e}.up"], p[f"e{e}.down"]))
    return out


# ---- the model -----------------------------------------------------------------------------------------------------------------
MIXERS = {"retention": retention, "parallel": side_by_side, "latent_attention": latent_attention}


def sub(weights: Dict[str, torch.Tensor], prefix: str, dtype) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(dtype) for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=DT, layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from position 0.  layers_out: receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    norm = lambda y, name: unit_rms(y, eps) * weights[name].to(dtype)
    x = weights["embed"].to(dtype)[tokens]
    for i, lc in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + norm(MIXERS[lc["type"]](norm(x, p + "norm1"), sub(weights, p + "mix.", dtype), lc["mixer"], eps), p + "norm1b")
        if lc.get("mlp") is not None:
            x = x + norm(experts(norm(x, p + "norm2"), sub(weights, p + "mlp.", dtype), lc["mlp"]), p + "norm2b")
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ weights["head"].to(dtype).T * float(cfg.get("logit_scale", 1.0))


# ---- tensors of a configuration, random weights -----------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W, V = int(cfg["width"]), int(cfg["vocab"])
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, lc in enumerate(cfg["layers"]):
        p, m, c = f"l{i}.", f"l{i}.mix.", lc["mixer"]
        out.update({p + "norm1": (W,), p + "norm1b": (W,)})
        if lc["type"] == "retention":
            H, D, Dv = c["heads"], c["dim"], c["vdim"]
            out.update({m + "q": (H * D, W), m + "k": (H * D, W), m + "v": (H * Dv, W), m + "g": (H * Dv, W), m + "o": (W, H * Dv)})
        elif lc["type"] == "latent_attention":
            H, D, Rt, Dv, K = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
            out.update({m + "q": (H * (D + Rt), W), m + "dkv": (K + Rt, W), m + "dkv.norm": (K,), m + "uk": (H * D, K), m + "uv": (H * Dv, K),
                        m + "g": (H * Dv, W), m + "o": (W, H * Dv)})
        else:
            a, d = c["left"], c["right"]
            nq, nk = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            out.update({m + "left.q": (nq, W), m + "left.k": (nk, W), m + "left.g": (a["heads"], W), m + "left.o": (W, a["heads"] * a["vdim"])})
            H, nk, nv, t = d["heads"], d["kv_heads"] * d["dim"], d["heads"] * d["vdim"], d["conv"]
            for name, n in (("q", nk), ("k", nk), ("v", nv)):
                out.update({m + f"right.{name}": (n, W), m + f"right.{name}.conv": (n, t)})
            out.update({m + "right.b": (H, W), m + "right.a": (H, W), m + "right.A_log": (H,), m + "right.dt_bias": (H,),
                        m + "right.norm": (d["vdim"],), m + "right.g": (nv, W), m + "right.o": (W, nv)})
        mlp = lc.get("mlp")
        if mlp is None:
            continue
        out.update({p + "norm2": (W,), p + "norm2b": (W,)})
        r, ff = mlp["router"], mlp["expert"]["ff"]
        n = int(r["experts"]) + int(r.get("identity", 0))
        out.update({p + "mlp.router": (n, W), p + "mlp.correction": (n,)})
        for e in range(int(r["experts"])):
            out.update({p + f"mlp.e{e}.gate": (ff, W), p + f"mlp.e{e}.up": (ff, W), p + f"mlp.e{e}.down": (W, ff)})
    return out


def random_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bf16 weights: matrices ~ N(0, 1 / in) (routers three times that, so that the choice is rarely close), norm
    weights near one, decays that keep the delta rule's state for some tens of tokens, corrections that change the choice now
    and then and make some choice scores negative."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and name[1].isdigit() else name
        if leaf == "embed":
            t = torch.randn(shape, generator=g)
        elif leaf.endswith(".conv"):
            t = torch.randn(shape, generator=g) * 0.5
            t[:, -1] += 1.0
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[1])
            if leaf == "mlp.router":
                t = t * 3.0
        elif leaf == "mix.right.A_log":
            t = -2.0 + 0.5 * torch.randn(shape, generator=g)
        elif leaf == "mix.right.dt_bias":
            t = -1.0 + torch.randn(shape, generator=g)
        elif leaf == "mlp.correction":
            t = torch.randn(shape, generator=g) * 0.05
        else:
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        out[name] = t.to(torch.bfloat16)
    return out
