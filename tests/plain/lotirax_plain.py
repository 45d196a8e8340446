"""A plain, slow implementation of the Lotirax decoder in NumPy float64: one function per
mechanism, whole sequences at once, no cache. It shares no code with the library and is the
oracle of the library's tests.

The design. x = E[token]. Every layer reads its input through one norm and adds both of its
sublayers at once: h = N1(x), x += m (l1 * mixer(h) + l2 * ff(h)), N(x) = x / sqrt(mean(x^2) +
eps) * (1 + w), l1 and l2 vectors, m a number for the model. A run of layers [start, stop) may
be passed ``times`` times with the same weights; before every pass x = W_in [x ; x0] + step[t]
with the embedding's output x0.

The mixer is differential attention: every head has two maps (a query and a key each) over the
same values. q, k, v have biases; q and k are normed per map with a weight shared by all heads
and maps, then the first ``dims`` of each map's values turn (pairs i, i + dims / 2; frequencies
stretched by wavelength, cosine and sine amplified). Each map is a softmax over the last
``size`` positions; o = a_1 - lambda a_2, over its root mean square, times (1 - diff), with
lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff.

Feed-forwards: W_d (silu(W_g h) * W_u h), or experts W_d relu(W_u h)^2 that a table names for
every token id, each with the weight 1 / top, and one shared expert of the same form.

``w``: a dict name -> float64 array (tables: integers). ``config``: the dict of config.json.
``rnd`` is applied to what a 16-bit implementation keeps in 16 bits (the default keeps
float64).
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


def silu(z):
    return z / (1.0 + np.exp(-z))


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_one_plus(x, w, eps):
    return unit_rms(x, eps) * (1.0 + w)


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


# ---------------------------------------------------------------------------- attention
def visible(T: int, size: Optional[int]):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size else True)


def softmax_attention(q, k, v, scale, mask):
    """q [T, d], k [T, d], v [T, vd] of one map."""
    s = np.where(mask, (q @ k.T) * scale, -np.inf)
    e = np.exp(s - s.max(axis=1, keepdims=True))
    return (e / e.sum(axis=1, keepdims=True)) @ v


def map_weight(w, p, diff) -> float:
    """lambda, what the second map is taken off with."""
    return (math.exp(float(np.sum(w[p + "lq1"] * w[p + "lk1"])))
            - math.exp(float(np.sum(w[p + "lq2"] * w[p + "lk2"]))) + diff)


def combine_maps(a1, a2, lam, diff, eps):
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, w, p, m, eps, rnd=exact):
    """h [T, width] -> [T, width]; ``p`` the tensors' prefix, ``m`` the mixer's sizes."""
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G, vd = m.get("kv_heads") or H, m.get("vdim") or d
    q = rnd(h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, 2 * H, d)
    k = rnd(h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, 2 * G, d)
    v = rnd(h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, vd)
    q = unit_rms(q, eps) * w[p + "q.norm"]
    k = unit_rms(k, eps) * w[p + "k.norm"]
    if m.get("rot"):
        q, k = rotate_halves(q, range(T), m["rot"]), rotate_halves(k, range(T), m["rot"])
    q, k = rnd(q), rnd(k)
    mask = visible(T, (m.get("mask") or {}).get("size"))
    lam = map_weight(w, p, m["diff"])
    heads = []
    for n in range(H):
        g = n // (H // G)
        a = [softmax_attention(q[:, 2 * n + i], k[:, 2 * g + i], v[:, g], m["scale"], mask)
             for i in range(2)]
        heads.append(combine_maps(a[0], a[1], lam, m["diff"], eps))
    return rnd(np.concatenate(heads, axis=1)) @ w[p + "o"].T


# ---------------------------------------------------------------------------- feed-forwards
def gated_feed_forward(h, w, p, rnd=exact):
    return rnd(silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p, rnd=exact):
    return rnd(relu_squared(h @ w[p + "up"].T)) @ w[p + "down"].T


def table_experts(h, ids, w, p, mlp, rnd=exact):
    """The experts that the table names for the token ids, and the shared one."""
    top = mlp["router"]["top"]
    y = np.zeros_like(h)
    for t, token in enumerate(ids):
        for e in w[p + "table"][token]:
            y[t] += expert(h[t:t + 1], w, f"{p}e{int(e)}.", rnd)[0] / top
    if mlp.get("shared"):
        y = y + expert(h, w, p + "shared.", rnd)
    return y


# ---------------------------------------------------------------------------- the decoder
def layer_runs(config) -> List[Tuple[int, int]]:
    """(layer, pass that this run opens or -1) in the order in which they run."""
    n = len(config["layers"])
    if not config.get("loop"):
        return [(i, -1) for i in range(n)]
    lp = config["loop"]
    out = [(i, -1) for i in range(lp["start"])]
    for t in range(lp["times"]):
        out += [(i, t if i == lp["start"] else -1) for i in range(lp["start"], lp["stop"])]
    return out + [(i, -1) for i in range(lp["stop"], n)]


def pass_start(x, x0, w, t, rnd=exact):
    return rnd(np.concatenate([x, x0], axis=1)) @ w["loop.in"].T + w["loop.step"][t]


def layer(x, ids, w, p, spec, eps, mult, rnd=exact):
    h = rnd(norm_one_plus(x, w[p + "norm1"], eps))
    add = w[p + "ls1"] * differential_attention(h, w, p + "mix.", spec["mixer"], eps, rnd)
    mlp = spec.get("mlp")
    if mlp:
        if mlp.get("kind") == "moe":
            y = table_experts(h, ids, w, p + "mlp.", mlp, rnd)
        else:
            y = gated_feed_forward(h, w, p + "mlp.", rnd)
        add = add + w[p + "ls2"] * y
    return x + mult * add


def forward(config, w: Dict[str, np.ndarray], tokens, rnd=exact, states: Optional[list] = None):
    """The logits [T, vocab] of a whole sequence; ``states`` receives the residual after every
    layer run."""
    eps = config["norm"]["eps"]
    tokens = np.asarray(tokens)
    x = x0 = w["embed"][tokens]
    for i, t in layer_runs(config):
        if t >= 0:
            x = pass_start(x, x0, w, t, rnd)
        x = layer(x, tokens, w, f"l{i}.", config["layers"][i], eps, config["residual_mult"], rnd)
        if states is not None:
            states.append(x)
    return rnd(norm_one_plus(x, w["final.norm"], eps)) @ w["embed"].T


def greedy(config, w, prompt, n: int) -> List[int]:
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(np.argmax(forward(config, w, ids)[-1])))
    return ids[len(prompt):]
