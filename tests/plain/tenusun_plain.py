"""A plain, slow implementation of the Tenusun decoder in NumPy float64: one function per
mechanism, whole sequences at once, no cache. It shares no code with the library and is the
oracle of the library's tests.

The design. x = c E[token], logits = E N(x) with the table itself. Every layer norms what a
sublayer reads and what it gives back: x += N1b(mixer(N1(x))), x += N2b(ff(N2(x))), all of them
layer norms with a weight and a bias.

Mixers. Latent attention: queries through a normed latent, keys and values out of one normed
latent c per token and one rotated key part that all heads share, a window, a plain softmax.
Attention: grouped heads with value rows of their own size, q and k rotated with frequencies
stretched by wavelength, a softmax whose denominator has one more term exp(0), values blended
with those of the first layer that blends, (1 - l) v + l v_first, and a gate
sigmoid(W_g h) for every value of the concatenated heads.

Feed-forwards: W_d (g sigmoid(1.702 g) (u + 1)) with g = min(W_g h, limit) and u = W_u h cut to
[-limit, limit]; or experts W_d (silu(W_g h) * W_u h), chosen by sigmoid scores plus a
correction among the best groups of neighbouring experts (a group counts its two best), weighted
by the scores alone.

``w``: a dict name -> float64 array. ``config``: the dict of config.json. ``rnd`` is applied to
what a 16-bit implementation keeps in 16 bits (the default keeps float64).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import numpy as np


# ---------------------------------------------------------------------------- small functions
def exact(a):
    return a


def bfloat16(a):
    """a rounded to the nearest bfloat16 (ties to even), as float64."""
    bits = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    bits = (bits + 0x7FFF + ((bits >> 16) & 1)) & 0xFFFF0000
    return bits.astype(np.uint32).view(np.float32).astype(np.float64).reshape(np.shape(a))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def layer_norm(x, w, b, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


# ---------------------------------------------------------------------------- positions
def rotary_frequencies(rot) -> Tuple[np.ndarray, float]:
    """The angle per position of every pair, and the factor of cosine and sine."""
    n, base = int(rot["dims"]), float(rot["base"])
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def where(turns):        # the pair (as a fraction) that makes so many turns over `original`
        return n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * ramp + fi * (1.0 - ramp))
    return np.array(out), 0.1 * math.log(s["factor"]) + 1.0


def rotate_halves(x, positions, rot):
    """x [T, heads, size]: value i of the first ``dims`` turns with value i + dims / 2."""
    f, amp = rotary_frequencies(rot)
    n = 2 * len(f)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = amp * np.cos(angle)[:, None, :], amp * np.sin(angle)[:, None, :]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., n:]], axis=-1)


def visible(T: int, size: Optional[int]):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size else True)


# ---------------------------------------------------------------------------- softmaxes
def softmax_rows(s, mask, extra_term: bool):
    """Row by row over the visible keys; ``extra_term``: one more term exp(0) below."""
    s = np.where(mask, s, -np.inf)
    top = s.max(axis=1, keepdims=True)
    if extra_term:
        top = np.maximum(top, 0.0)
    e = np.exp(s - top)
    return e / (e.sum(axis=1, keepdims=True) + (np.exp(-top) if extra_term else 0.0))


# ---------------------------------------------------------------------------- mixers
def latent_attention(h, w, p, m, eps, rnd=exact):
    """h [T, width] -> [T, width]; ``p`` the tensors' prefix, ``m`` the mixer's sizes."""
    T = h.shape[0]
    H, d, r, vd, kvr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    cq = rnd(rms_norm(rnd(h @ w[p + "dq"].T), w[p + "dq.norm"], eps))
    q = rnd(cq @ w[p + "uq"].T).reshape(T, H, d + r)
    both = rnd(h @ w[p + "dkv"].T)
    c = rnd(rms_norm(both[:, :kvr], w[p + "dkv.norm"], eps))
    kr = rnd(rotate_halves(both[:, None, kvr:], np.arange(T), rot))[:, 0]
    qr = rnd(rotate_halves(q[..., d:], np.arange(T), rot))
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, vd)
    mask = visible(T, (m.get("mask") or {}).get("size"))
    heads = []
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        heads.append(rnd(softmax_rows(s, mask, False) @ v[:, i]))
    return np.concatenate(heads, axis=1) @ w[p + "o"].T


def blend(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, w, p, m, first_values=None, rnd=exact):
    """h [T, width] -> ([T, width], the layer's own values [T, G vd] before any blending).
    ``first_values``: what this layer's values are blended with, or None."""
    T = h.shape[0]
    H, G, d, vd = m["heads"], m.get("kv_heads") or m["heads"], m["dim"], m["vdim"]
    q = rnd(h @ w[p + "q"].T).reshape(T, H, d)
    k = rnd(h @ w[p + "k"].T).reshape(T, G, d)
    own = rnd(h @ w[p + "v"].T)
    v = own if first_values is None else rnd(blend(own, first_values, float(w[p + "vmix"])))
    v = v.reshape(T, G, vd)
    if m.get("rot"):
        q = rnd(rotate_halves(q, np.arange(T), m["rot"]))
        k = rnd(rotate_halves(k, np.arange(T), m["rot"]))
    mask = visible(T, None)
    heads = []
    for i in range(H):
        g = i // (H // G)
        heads.append(softmax_rows((q[:, i] @ k[:, g].T) * m["scale"], mask, True) @ v[:, g])
    gate = sigmoid(rnd(h @ w[p + "g"].T))
    return rnd(np.concatenate(heads, axis=1) * gate) @ w[p + "o"].T, own


# ---------------------------------------------------------------------------- feed-forwards
def clamped_dense(h, w, p, limit, rnd=exact):
    g = np.minimum(h @ w[p + "gate"].T, limit)
    u = np.clip(h @ w[p + "up"].T, -limit, limit)
    return rnd(g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choose(z, correction, top, count, keep) -> Tuple[List[int], List[float]]:
    """The experts of one token's router logits z [E] and their weights (ties: the lower)."""
    chosen, weights, _ = choose_with_margin(z, correction, top, count, keep)
    return chosen, weights


def choose_with_margin(z, correction, top, count, keep):
    """Also how close the call was: the least that a choice score (or a group's score) lies above
    the first one left out."""
    s = sigmoid(z)
    score = s + correction
    size = len(z) // count
    totals = [sum(sorted(score[g * size:(g + 1) * size])[-2:]) for g in range(count)]
    groups = sorted(range(count), key=lambda g: (-totals[g], g))
    kept = groups[:keep]
    ranked = sorted((e for e in range(len(z)) if e // size in kept), key=lambda e: (-score[e], e))
    chosen = ranked[:top]
    margin = np.inf
    if keep < count:
        margin = min(margin, totals[groups[keep - 1]] - totals[groups[keep]])
    if top < len(ranked):
        margin = min(margin, score[ranked[top - 1]] - score[ranked[top]])
    return chosen, [float(s[e]) for e in chosen], float(margin)


class Routing:
    """What a test wants to know of the routers' choices, or to settle about them.

    ``margins[(layer, t)]``: how close the call was. ``forced[(layer, t)]``: the experts that
    another implementation chose there; they replace the plain choice where the two differ and the
    margin is below ``close`` (a computation in 16 bits may fall on either side of such a call);
    where the margin is larger the difference is an error (unless ``strict`` is off)."""

    def __init__(self, forced=None, close: float = 0.05, strict: bool = True):
        self.forced, self.close, self.strict = forced or {}, close, strict
        self.margins: Dict = {}

    def settle(self, layer, t, chosen, weights, margin, z):
        self.margins[(layer, t)] = margin
        theirs = self.forced.get((layer, t))
        if theirs is None or set(theirs) == set(chosen):
            return chosen, weights
        if self.strict and margin >= self.close:
            raise AssertionError(f"layer {layer}, token {t}: experts {sorted(theirs)} were chosen, "
                                 f"{sorted(chosen)} expected, at a margin of {margin:.3g}")
        return list(theirs), [float(v) for v in sigmoid(z[list(theirs)])]


def routed_experts(h, w, p, mlp, rnd=exact, routing: Optional[Routing] = None, layer: int = 0):
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ w[p + "router"].T
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, weights, margin = choose_with_margin(z[t], w[p + "correction"], r["top"],
                                                     groups["count"], groups["keep"])
        if routing is not None:
            chosen, weights = routing.settle(layer, t, chosen, weights, margin, z[t])
        for e, s in zip(chosen, weights):
            q = f"{p}e{e}."
            a = rnd(silu(w[q + "gate"] @ h[t]) * (w[q + "up"] @ h[t]))
            out[t] += s * (w[q + "down"] @ a)
    return out


# ---------------------------------------------------------------------------- the model
def forward(config, w: Dict[str, np.ndarray], tokens, rnd=exact,
            states: Optional[list] = None, routing: Optional[Routing] = None) -> np.ndarray:
    """Logits [T, vocab] of a whole sequence; ``states`` receives the residual after every
    layer; ``routing``: what a test knows or wants to know of the routers' choices."""
    eps = float(config["norm"]["eps"])

    def norm(x, name):
        return layer_norm(x, w[name], w[name + ".b"], eps)

    x = w["embed"][np.asarray(tokens)] * float((config.get("embedding") or {}).get("scale", 1.0))
    first_values = None
    for i, layer in enumerate(config["layers"]):
        l, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        h = rnd(norm(x, l + "norm1"))
        if layer["type"] == "latent_attention":
            y = latent_attention(h, w, l + "mix.", m, eps, rnd)
        else:
            blends = bool(m.get("v_mix"))
            y, own = attention(h, w, l + "mix.", m, first_values if blends else None, rnd)
            if blends and first_values is None:
                first_values = own
        x = x + norm(y, l + "norm1b")
        if mlp is not None:
            h = rnd(norm(x, l + "norm2"))
            if mlp.get("kind", "dense") == "dense":
                y = clamped_dense(h, w, l + "mlp.", float(mlp["limit"]), rnd)
            else:
                y = routed_experts(h, w, l + "mlp.", mlp, rnd, routing, i)
            x = x + norm(y, l + "norm2b")
        if states is not None:
            states.append(x.copy())
    return rnd(norm(x, "final.norm")) @ w["embed"].T
