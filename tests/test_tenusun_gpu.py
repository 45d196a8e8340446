"""The Tenusun family on a B200 against the plain implementation, in float32 and bfloat16: each
mechanism alone (with weights or inputs made so that a fault shows), then the engine on four small
models of other sizes: whole prompts with the residual after every layer, prompts against
token-by-token decoding, portions down to two tokens, unequal batches against each request alone,
slots and pages used again, the first tokens, long decoding past windows and page borders, decode
graphs, and greedy generation through the entry point."""
import os

import numpy as np
import pytest
import torch

from mormot2_ai_b200 import Engine, Entry, LlmClient, PartSpec, Runtime, TenusunConfig
from mormot2_ai_b200 import kernels as K
from mormot2_ai_b200.cache.pages import PAGE, pages_for
from mormot2_ai_b200.cache.storage import CacheLine
from mormot2_ai_b200.parts import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITIONS
from mormot2_ai_b200.parts.block import settle
from mormot2_ai_b200.weights import random_tensors
from tests.gpu_helpers import DEV, make_step
from tests.plain import tenusun_plain as plain
from tests.tenusun_models import SMALL, SmallModel, _att, _lat, _rot

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module", params=sorted(SMALL))
def small(request, tmp_path_factory):
    return SmallModel(request.param, str(tmp_path_factory.mktemp("tenusun_" + request.param)))


@pytest.fixture(scope="module")
def small_a(tmp_path_factory):
    return SmallModel("A", str(tmp_path_factory.mktemp("tenusun_A_only")))


class Choices:
    """The experts that an engine's routers chose, by slot, layer and position, read through the
    routed feed-forward's probe. In 16 bits a router may fall on the other side of a close call
    than the plain implementation; the plain one then takes the engine's choice THERE
    (``plain.Routing``), and a different choice anywhere else fails the test."""

    def __init__(self, eng):
        from mormot2_ai_b200.parts.moe import RoutedExperts
        self.layers = [i for i, l in enumerate(eng.model.layers)
                       if isinstance(l.feed_forward, RoutedExperts)]
        self.calls, self.by_slot = 0, {}
        for i in self.layers:
            eng.model.layers[i].feed_forward.probe = self.seen
        eng.use_graphs = False

    def seen(self, part, step, ids):
        layer = self.layers[self.calls % len(self.layers)]      # routers run in the layers' order
        self.calls += 1
        rows, at = ids.cpu().numpy(), 0
        for slot, past, new in zip(step.host_slots, step.host_past, step.host_new):
            kept = self.by_slot.setdefault(slot, {})
            for j in range(new):
                kept[(layer, past + j)] = rows[at + j].tolist()
            at += new


def expected(model, eng, slot, ids, dtype, states=None, alone=None):
    """The plain logits and those that 16-bit rounding alone gives, both with the engine's side of
    close calls (and the choices that the engine made in the slot are forgotten)."""
    forced = eng.choices.by_slot.pop(slot, {}) if eng.choices is not None else {}
    return (model.reference(ids, states, plain.Routing(forced)),
            model.rounded(ids, dtype, forced, alone))


# The bounds of this family's comparisons, set from what was measured. float32: the largest
# difference of a logit over the largest logit. bfloat16: per position, the largest difference of
# a logit over the spread of the plain logits, bounded in the median, the ninth decile and the
# worst position of a comparison, and never tighter than three times what the plain
# implementation itself moves by when it rounds what a 16-bit run rounds.
F32_TOL = 2e-5
BF16_TOL = {"median": 0.04, "decile": 0.08, "worst": 0.2}


def spread_errors(got, want):
    rows = np.abs(got - want).reshape(-1, want.shape[-1]).max(axis=1) / want.std()
    return np.median(rows), np.quantile(rows, 0.9), rows.max(), len(rows)


def check(got, want, dtype, what, rounded=None):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape, (got.shape, want.shape)
    record = os.environ.get("MORMOT_TOL_RECORD")
    if dtype == "float32":
        err = np.abs(got - want).max() / max(1.0, np.abs(want).max())
        if record:
            with open(record, "a") as f:
                f.write(f"float32\t{err:.3e}\t{what}\n")
        assert err <= F32_TOL, f"{what}: relative error {err:.3g} (float32)"
        return
    med, dec, worst, n = spread_errors(got, want)
    tol = dict(BF16_TOL)
    if rounded is not None:
        r = spread_errors(np.asarray(rounded, dtype=np.float64), want)
        tol = {k: max(tol[k], 3.0 * r[i]) for i, k in enumerate(("median", "decile", "worst"))}
    if record:
        with open(record, "a") as f:
            f.write(f"bfloat16\t{med:.3f}\t{dec:.3f}\t{worst:.3f}\t{n}\t{what}\t{tol}\n")
    assert worst <= tol["worst"], f"{what}: a position off by {worst:.3g} of the spread"
    if n >= 8:
        assert med <= tol["median"] and dec <= tol["decile"], \
            f"{what}: median {med:.3g}, ninth decile {dec:.3g} of the spread (bfloat16)"


def close(got, want, dtype, what):
    """Both divided by the largest expected value."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    err = np.abs(got - want).max() / max(1e-6, np.abs(want).max())
    assert err <= (2e-5 if dtype == "float32" else 2e-2), f"{what}: {err:.3g}"


def part_weights(part, seed=0, std=0.1):
    w = random_tensors(part.tensors(), seed, std=std, norm_std=0.2, dtype=torch.bfloat16)
    return w, {k: v.double().numpy() for k, v in w.items()}


def to_dev(w, dtype):
    return {k: v.to(TORCH[dtype]).to(DEV) for k, v in w.items()}


def rounded(a, dtype):
    return torch.tensor(np.asarray(a), dtype=torch.float32).to(TORCH[dtype]).double().numpy()


def line_of(n_slots, max_len, nkv, head_dim, vd, dtype, seed=0):
    """A cache line that keeps all pages, scrambled over the pool."""
    per = pages_for(max_len)
    n_pages = n_slots * per + 3
    ids = np.random.default_rng(seed).permutation(n_pages)[:n_slots * per]
    table = torch.tensor(ids.reshape(n_slots, per), dtype=torch.int32, device=DEV)
    k = torch.zeros((n_pages, nkv, PAGE, head_dim), dtype=dtype, device=DEV)
    v = torch.zeros((n_pages, nkv, PAGE, vd), dtype=dtype, device=DEV)
    return CacheLine(k, v, table, per, 0, 0, nkv, head_dim, 0 if vd == head_dim else vd)


# ---------------------------------------------------------------------------- mechanisms
def f32(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32, device=DEV)


def normed(x, kind, w, b, eps):
    if kind == "layer":
        return plain.layer_norm(x, w, b, eps)
    return plain.rms_norm(x, w, eps) + b


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [64, 70, 512, 1536, 5120, 12288])
def test_norms_on_both_sides_of_a_sublayer(dtype, H):
    """x += N_out(sum of the parts), h = N_in(x): both kinds, parts that lie one after another or
    row by row, with and without either half; rows whose mean is far from zero."""
    T, eps, cd = 5, 1e-4, TORCH[dtype]
    rng = np.random.default_rng(H)
    x = rng.normal(size=(T, H)) + 3.0 * rng.normal(size=(T, 1))
    w1, w2 = 1.0 + 0.3 * rng.normal(size=(2, H))
    b1, b2 = rng.normal(size=(2, H))
    stored = rng.normal(size=(T, H)) * 0.1 + 40.0       # far from zero: the deviations are small
    split = rng.normal(size=(3, T, H))
    rows = rng.normal(size=(T, 11, H))                  # row t * 11 + k: more than one round of loads
    for kind1, kind2 in (("layer", "layer"), ("rms", "layer"), ("layer", "rms")):
        for y, total in ((f32(stored), stored), (f32(split), split.sum(0)),
                         (f32(rows).transpose(0, 1), rows.sum(1))):
            for weights in (torch.float32, cd):
                ws = [torch.tensor(a, device=DEV).to(weights) for a in (w1, b1, w2, b2)]
                v = [a.double().cpu().numpy() for a in ws]
                want = x + normed(total, kind1, v[0], v[1], eps)
                xd, h = f32(x), torch.empty((T, H), dtype=cd, device=DEV)
                K.norm_step(xd, y, (ws[0], ws[1], kind1, eps), h, (ws[2], ws[3], kind2, eps))
                tight = np.abs(xd.double().cpu().numpy() - want).max() / np.abs(want).max()
                assert tight < 2e-4, (kind1, tight)     # 40 + 0.1 n in float32 keeps that much of n
                close(h.double().cpu().numpy(), normed(xd.double().cpu().numpy(), kind2, v[2], v[3], eps),
                      dtype, f"{kind1}, {kind2}")
                xd = f32(x)
                K.norm_step(xd, y, (ws[0], None, kind1, eps))     # settled, no bias
                no_bias = x + normed(total, kind1, v[0], 0.0, eps)
                assert np.abs(xd.double().cpu().numpy() - no_bias).max() < 2e-4 * np.abs(no_bias).max()
    for kind in ("layer", "rms"):                       # the norm alone, of some rows
        pick = [4, 0, 0, 2]
        h = torch.empty((4, H), dtype=cd, device=DEV)
        K.norm_step(f32(x), h=h, in_norm=(f32(w1), f32(b1), kind, eps),
                    rows=torch.tensor(pick, dtype=torch.int32, device=DEV))
        close(h.double().cpu().numpy(), normed(x[pick], kind, w1, b1, eps), dtype, f"rows, {kind}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_norms_over_many_rows(dtype):
    T, H, eps = 300, 4096, 1e-6
    rng = np.random.default_rng(3)
    x, y, w, b = (rng.normal(size=s) for s in ((T, H), (2, T, H), (H,), (H,)))
    xd, h = f32(x), torch.empty((T, H), dtype=TORCH[dtype], device=DEV)
    K.norm_step(xd, f32(y), (f32(w), f32(b), "layer", eps), h, (f32(b), f32(w), "layer", eps))
    want = x + plain.layer_norm(y.sum(0), w, b, eps)
    close(xd.cpu().numpy(), want, "float32", "residual")
    close(h.double().cpu().numpy(), plain.layer_norm(want, b, w, eps), dtype, "operand")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nh,nkv,dim,vd,rot", [
    (4, 2, 18, 10, _rot(12, 500.0, 3.0)), (3, 1, 7, 5, _rot(4, 20.0)), (2, 1, 130, 300, None),
    (4, 2, 64, 40, _rot(32, 1e4, 8.0, 128)), (5, 5, 128, 64, _rot(128, 1e4)), (6, 2, 72, 8, _rot(16, 90.0, 2.0))])
def test_rotation_blend_and_gates_of_a_products_rows(dtype, nh, nkv, dim, vd, rot):
    cd = TORCH[dtype]
    rng = np.random.default_rng(dim)
    gate_n = nh * vd
    at_v = (nh + nkv) * dim
    width = at_v + nkv * vd + gate_n
    seqs = [(1, 0, [0] * 3, []), (0, 60, [0] * 6, []), (2, 1000, [0], [])]
    if dim >= 64:
        seqs.append((3, 50, [0] * 130, []))
    pos = np.concatenate([np.arange(past, past + len(t)) for _, past, t, _ in seqs])
    slots = np.concatenate([[slot] * len(t) for slot, _, t, _ in seqs])
    step, T = make_step(seqs), len(pos)
    position = None
    if rot:
        params = {"theta": rot["base"], "rot_dim": rot["dims"]}
        if rot.get("scaling"):
            position = POSITIONS.build(PartSpec("rope_yarn", {**params, **rot["scaling"]}))
        else:
            position = POSITIONS.build(PartSpec("rope_half", {**params, "rounding": "once"}))
        position.bind({}, Runtime(cd))
    freq, n_rot = position.frequencies() if position else (None, 0)
    amp = position.amplitude if position else 1.0
    lam = f32([0.3])
    tol = 8e-3 if dtype == "bfloat16" else 2e-4           # angles in float32
    for form in ("stored", "split"):
        for mix in (None, "first", "blend"):
            parts = rng.normal(size=(3, T, width))
            rows = parts.sum(0)
            if form == "stored":
                rows = rounded(rows, dtype)
                given = torch.tensor(rows, dtype=cd, device=DEV)
            else:
                given = f32(parts)
            q, k = rows[:, :nh * dim].reshape(T, -1, dim), rows[:, nh * dim:at_v].reshape(T, -1, dim)
            v = rows[:, at_v:at_v + nkv * vd]
            if rot:
                q, k = plain.rotate_halves(q, pos, rot), plain.rotate_halves(k, pos, rot)
            other = rounded(rng.normal(size=(T, nkv * vd)), dtype)
            first = torch.tensor(other, dtype=cd, device=DEV) if mix else None
            line = line_of(4, 1024, nkv, dim, vd, cd)
            gate = torch.empty((T, gate_n), dtype=cd, device=DEV) if form == "split" else None
            q_out = given if form == "stored" else torch.empty((T, nh * dim), dtype=cd, device=DEV)
            K.rope_store(given, freq, n_rot, amp, step, line, nh, nkv, dim, vd, q_out, first,
                         lam if mix == "blend" else None, gate)
            if mix == "first":
                close(first.double().cpu().numpy(), v, dtype, "the first layer's values")
            elif mix == "blend":
                assert np.array_equal(first.double().cpu().numpy(), other)
                v = plain.blend(v, other, 0.3)
            got = q_out.double().cpu().numpy()
            if form == "stored":                          # the other columns are left alone
                assert np.array_equal(got[:, at_v:], rows[:, at_v:])
            else:
                close(gate.double().cpu().numpy(), rows[:, at_v + nkv * vd:], dtype, "gates")
            err = np.abs(got[:, :nh * dim].reshape(T, -1, dim) - q).max() / np.abs(q).max()
            assert err < tol, (form, mix, err)
            table = line.page_table.cpu()
            for t in range(T):
                page = int(table[slots[t], pos[t] // PAGE])
                kc = line.k[page, :, pos[t] % PAGE].double().cpu().numpy()
                vc = line.v[page, :, pos[t] % PAGE].double().cpu().numpy()
                assert np.abs(kc - k[t]).max() / np.abs(k).max() < tol, (form, mix, t)
                assert np.abs(vc.reshape(-1) - v[t]).max() / np.abs(v).max() < (
                    1e-2 if dtype == "bfloat16" else 1e-6), (form, mix, t)


def attention_reference(q, keys, vals, gates, pos, nkv, scale, window):
    """q [T, nh, d] at positions ``pos``, keys [N, nkv, d], vals [N, nkv, vd], gates [T, nh, vd]."""
    T, nh = q.shape[:2]
    out = np.zeros((T, nh, vals.shape[-1]))
    for t in range(T):
        lo = max(0, pos[t] + 1 - window) if window else 0
        for h in range(nh):
            g = h // (nh // nkv)
            s = keys[lo:pos[t] + 1, g] @ q[t, h] * scale
            p = plain.softmax_rows(s[None], np.ones((1, len(s)), dtype=bool), True)[0]
            out[t, h] = (p @ vals[lo:pos[t] + 1, g]) * plain.sigmoid(gates[t, h])
    return out


def fill(line, slot, keys, vals):
    table = line.page_table.cpu().numpy()
    for p in range(0, len(keys), PAGE):
        page = int(table[slot, p // PAGE])
        n = min(PAGE, len(keys) - p)
        line.k[page, :, :n] = torch.tensor(keys[p:p + n]).transpose(0, 1).to(line.k.dtype).to(DEV)
        line.v[page, :, :n] = torch.tensor(vals[p:p + n]).transpose(0, 1).to(line.v.dtype).to(DEV)


SIZES = [(4, 2, 18, 10), (2, 2, 16, 24), (6, 1, 48, 72), (3, 3, 64, 128), (4, 1, 64, 64), (20, 1, 40, 56),
         (2, 1, 72, 136), (4, 2, 128, 64), (3, 1, 128, 128), (17, 1, 8, 8), (2, 1, 120, 104), (2, 1, 130, 250)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nh,nkv,dim,vd", SIZES)
def test_loud_keys_against_the_sink(dtype, nh, nkv, dim, vd):
    """One key whose score stands out, at page borders, far back and at a window's edge, for tokens
    of a prompt and decoded ones: it decides the head's output where it is visible, shrunk by the
    sink's share, and must not be felt where it is not; a gate for every value. The other scores
    lie so low that the sink takes most of what the loud key leaves."""
    cd, scale = TORCH[dtype], 0.25
    rt = Runtime(cd)
    N = 330
    rng = np.random.default_rng(dim + vd)
    sink = torch.zeros((nh,), dtype=torch.float32, device=DEV)
    direction = rng.normal(size=dim)
    direction /= np.linalg.norm(direction)
    for window in (0, 5, 64, 65, 200):
        for loud in (0, 1, 63, 64, 127, 128, 200, 256):
            keys = rng.normal(size=(N, nkv, dim)) * 0.2 - direction * 5.0
            vals = rounded(rng.normal(size=(N, nkv, vd)), "bfloat16")
            q = rng.normal(size=(N, nh, dim)) * 0.2 + direction * 5.0
            keys[loud] = direction * (2.0 if loud % 2 else 4.0)       # e^2.5 or e^5 against one
            keys, q = rounded(keys, "bfloat16"), rounded(q, "bfloat16")
            gates = rounded(rng.normal(size=(N, nh, vd)), "bfloat16")
            line = line_of(2, N, nkv, dim, vd, cd, seed=loud)
            fill(line, 1, keys, vals)
            edge = loud + (window or 200)                      # the first token that misses it
            places = sorted({p for p in (loud, loud + 1, edge - 1, edge, edge + 1, N - 1) if loud <= p < N})
            a = places[0]
            want = attention_reference(q[places], keys, vals, gates[places], places, nkv, scale, window)
            alone = attention_reference(q[places[:1]], keys, vals, gates[places[:1]], places[:1], nkv,
                                        scale, window)
            size = np.abs(alone).max()

            def run(step, rows, gate_rows):
                n = len(rows)
                # q and the gates in one row, as the product leaves them
                pad = -(-nh * dim // 8) * 8
                both = torch.zeros((n, pad + nh * vd), dtype=cd, device=DEV)
                both[:, :nh * dim] = torch.tensor(rows.reshape(n, -1)).to(cd).to(DEV)
                both[:, pad:] = torch.tensor(gate_rows.reshape(n, -1)).to(cd).to(DEV)
                out = torch.full((n, nh * vd), 9.0, dtype=cd, device=DEV)
                rt.attention(both, both.shape[1], out, step, line, nh, nkv, dim, window, scale, vd=vd,
                             sink=sink, gate=both[:, pad:], gate_stride=both.shape[1], gate_dim=vd)
                return out.double().cpu().numpy().reshape(n, nh, vd)

            got = run(make_step([(1, a, [0] * (N - a), [])]), q[a:], gates[a:])[[p - a for p in places]]
            err = np.abs(got - want).max() / size
            assert err <= (3e-5 if dtype == "float32" else 2e-2), (window, loud, "prompt", err)
            for i, p in enumerate(places):
                got = run(make_step([(1, p, [0], [])]), q[p:p + 1], gates[p:p + 1])[0]
                err = np.abs(got - want[i]).max() / size
                assert err <= (3e-5 if dtype == "float32" else 2e-2), (window, loud, p, err)
    rt.check()


def test_decode_splits_through_scratch_with_a_gate_per_value():
    """The form of a long sequence: more splits than a cluster holds, added up by a second kernel."""
    rt = Runtime(torch.bfloat16)
    rng = np.random.default_rng(2)
    for nh, nkv, dim, vd in ((4, 2, 128, 64), (6, 2, 40, 24), (2, 1, 128, 128)):
        N, scale = 1500, 0.2
        keys, vals = (rounded(rng.normal(size=(N, nkv, d)), "bfloat16") for d in (dim, vd))
        q, gates = (rounded(rng.normal(size=(1, nh, d)), "bfloat16") for d in (dim, vd))
        line = line_of(1, N, nkv, dim, vd, torch.bfloat16)
        fill(line, 0, keys, vals)
        out = torch.empty((1, nh * vd), dtype=torch.bfloat16, device=DEV)
        qd = torch.tensor(q.reshape(1, -1)).to(torch.bfloat16).to(DEV)
        gd = torch.tensor(gates.reshape(1, -1)).to(torch.bfloat16).to(DEV)
        sink = torch.zeros((nh,), dtype=torch.float32, device=DEV)
        for splits in (1, 3, 19):
            K.attention_decode(qd, nh * dim, out, make_step([(0, N - 1, [0], [])]), line, nh, nkv, dim, 0,
                               scale, splits, rt.attention_scratch, rt.error_word, sink, gate=gd,
                               gate_stride=nh * vd, gate_dim=vd, vd=vd)
            want = attention_reference(q, keys, vals, gates, [N - 1], nkv, scale, 0)
            close(out.double().cpu().numpy().reshape(nh, vd), want[0], "bfloat16", f"{splits} splits")
    rt.check()


def run_mixer(mixer, hs, cuts, hidden, dtype, line, memos=None):
    """Feeds each sequence of ``hs`` (float arrays [n, hidden]) through the mixer in the
    portions that ``cuts`` names (all sequences of a step together), from slots 2, 0, 1, ...;
    returns the mixer's output per sequence. ``memos``: what every step's parts have kept (a list
    that is filled, or used again)."""
    slots = [2, 0, 1, 3][:len(hs)]
    outs = [[] for _ in hs]
    for n, (lo, hi) in enumerate(cuts):
        seqs, rows = [], []
        for b, h in enumerate(hs):
            a, e = min(lo, len(h)), min(hi, len(h))
            if e > a:
                seqs.append((slots[b], a, [0] * (e - a), []))
                rows.append((b, a, e))
        if not seqs:
            continue
        step = make_step(seqs)
        if memos is not None:
            if n < len(memos):
                step.memo = memos[n]
            else:
                memos.append(step.memo)
        h = torch.tensor(np.concatenate([hs[b][a:e] for b, a, e in rows])).to(TORCH[dtype]).to(DEV)
        for store in (True, False):             # into a place of its own, and added onto one
            x = torch.full((h.shape[0], hidden), 0.5, device=DEV)
            pending = mixer.forward(h, x, step, line, None, True, store=store)
            if pending is not None:             # split sums that the next kernel would add
                if store:
                    x.zero_()
                settle(x, pending)
            got, at = x.cpu().double().numpy() - (0.0 if store else 0.5), 0
            if store:
                for b, a, e in rows:
                    outs[b].append(got[at:at + e - a])
                    at += e - a
                kept = got
            else:
                assert np.abs(got - kept).max() <= 1e-4 * max(1.0, np.abs(kept).max())
    return [np.concatenate(o) for o in outs]


CUTS = [[(0, 150)], [(0, 2), (2, 4), (4, 64), (64, 66), (66, 150)],
        [(0, 60)] + [(t, t + 1) for t in range(60, 72)]]


def mixer_of(layer, hidden, rt, first=False, eps=1e-4):
    cfg = TenusunConfig.from_dict({"architecture": "Tenusun", "vocab": 9, "width": hidden,
                                   "norm": {"eps": eps}, "layers": [layer]})
    positions = {}
    spec = cfg._mixer(layer, positions, first)
    positions = {k: POSITIONS.build(v) for k, v in positions.items()}
    for p in positions.values():
        p.bind({}, rt)
    return MIXERS.build(spec, "x.", positions=positions)


MIXES = [(_att(4, 2, 22, 10, 0.3, _rot(12, 500.0, 3.0), True), 72), (_att(3, 1, 40, 24, 0.2, _rot(32, 90.0), True), 64),
         (_att(2, 2, 128, 64, 0.1, _rot(64, 1e4, 8.0, 128), True), 96), (_att(8, 1, 64, 128, 0.15, None, True), 128)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer,hidden", MIXES, ids=[str(i) for i in range(len(MIXES))])
def test_attention_as_a_mixer_and_values_blended_across_layers(dtype, layer, hidden):
    """Two layers of three unequal sequences, in whole portions, small ones and single tokens: the
    first keeps its values of the step, the second blends them with its own."""
    m = layer["mixer"]
    rt = Runtime(TORCH[dtype])
    one, two = mixer_of(layer, hidden, rt, first=True), mixer_of(layer, hidden, rt)
    rng = np.random.default_rng(7)
    hs = [[rounded(rng.normal(size=(n, hidden)), dtype) for n in (150, 3, 67)] for _ in range(2)]
    bound = []
    for mixer, seed in ((one, 11), (two, 12)):
        w, wp = part_weights(mixer, seed=seed, std=0.2)
        wp.setdefault("x.mix.vmix", np.float64(0.5))
        mixer.bind(to_dev(w, dtype), rt)
        bound.append(wp)
    want, moved = ([], []), ([], [])
    for b in range(3):
        for out, rnd in ((want, plain.exact), (moved, plain.bfloat16)):
            y, own = plain.attention(hs[0][b], bound[0], "x.mix.", m, None, rnd)
            out[0].append(y)
            out[1].append(plain.attention(hs[1][b], bound[1], "x.mix.", m, own, rnd)[0])
    assert float(bound[1]["x.mix.vmix"]) > 0.05
    for cuts in CUTS:
        memos = []
        for i, mixer in enumerate((one, two)):
            line = line_of(4, 192, m["kv_heads"], m["dim"], m["vdim"], TORCH[dtype], seed=3)
            got = run_mixer(mixer, hs[i], cuts, hidden, dtype, line, memos)
            for g, wnt, mv in zip(got, want[i], moved[i]):
                check(g, wnt[:len(g)], dtype, f"layer {i}, cuts {cuts[:4]}",
                      mv[:len(g)] if dtype == "bfloat16" else None)
    rt.check()


LATENTS = [(_lat(3, 18, 10, 14, 26, 30, 0.25, 21, 90.0), 72), (_lat(4, 48, 32, 40, 72, 64, 0.12, 65, 1e4), 96),
           (_lat(1, 16, 16, 8, 24, 48, 0.2, 64, 50.0), 64), (_lat(6, 24, 0, 32, 16, 32, 0.2, 0, 50.0), 64),
           # sizes for which long steps form keys and values per head
           (_lat(3, 64, 32, 64, 72, 64, 0.12, 65, 1e4), 96), (_lat(2, 128, 64, 128, 40, 48, 0.08, 200, 1e3), 64),
           (_lat(5, 64, 0, 128, 32, 80, 0.15, 0, 50.0), 64), (_lat(1, 128, 8, 64, 24, 40, 0.1, 1, 90.0), 64),
           (_lat(2, 64, 48, 64, 40, 128, 0.1, 300, 1e3), 64)]


def loud_pair(w, m, hidden, eps, rng):
    """Two inputs of which the second's queries like the first's keys more than anything else (by
    the unrotated part of the scores, in one head)."""
    c = rng.normal(size=(900, hidden))
    H, d = m["heads"], m["dim"]
    cq = plain.rms_norm(c @ w["x.mix.dq"].T, w["x.mix.dq.norm"], eps)
    q = (cq @ w["x.mix.uq"].T).reshape(900, H, -1)[..., :d]
    ckv = plain.rms_norm(c @ w["x.mix.dkv"].T[:, :m["kv_rank"]], w["x.mix.dkv.norm"], eps)
    k = (ckv @ w["x.mix.uk"].T).reshape(900, H, d)
    best = np.einsum("ihd,jhd->hij", q, k).max(axis=0)
    i, j = np.unravel_index(best.argmax(), best.shape)
    return c[j], c[i]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer,hidden", LATENTS, ids=[str(i) for i in range(len(LATENTS))])
def test_latent_attention_in_a_window(dtype, layer, hidden, monkeypatch):
    """One key that some queries like more than all others: queries at the last position that sees
    it and at the first that does not."""
    m, eps = layer["mixer"], 1e-4
    rt = Runtime(TORCH[dtype])
    mixer = mixer_of(layer, hidden, rt, eps=eps)
    w, wp = part_weights(mixer, seed=5, std=0.25)
    mixer.bind(to_dev(w, dtype), rt)
    rng = np.random.default_rng(9)
    formed = mixer.sizes_expand()
    N = 600 if formed else 150          # long enough for several tiles of rows
    hs = [rng.normal(size=(n, hidden)) for n in (N, 3, 67)]
    size = (m.get("mask") or {}).get("size")
    key, query = loud_pair(wp, m, hidden, eps, rng)
    hs[0][10] = key
    for n in (10 + (size or 70) - 1, 10 + (size or 70)):
        if n != 10:
            hs[0][n] = query
    hs = [rounded(h, dtype) for h in hs]
    want = [plain.latent_attention(h, wp, "x.mix.", m, eps) for h in hs]
    moved = [plain.latent_attention(h, wp, "x.mix.", m, eps, rnd=plain.bfloat16) for h in hs]
    if size:        # a window one position off would show
        for other, at in [(size + 1, 10 + size)] + [(size - 1, 10 + size - 1)] * (size > 1):
            off = plain.latent_attention(hs[0], wp, "x.mix.", dict(m, mask={"size": other}), eps)
            assert np.abs(off[at] - want[0][at]).max() > 0.2 * want[0].std(), (other, at)
    calls, kernel = [], K.latent_prefill_tc
    monkeypatch.setattr(K, "latent_prefill_tc", lambda *a, **k: (calls.append(1), kernel(*a, **k))[1])
    cuts_of = CUTS if not formed else [
        [(0, N)], [(0, 2), (2, 4), (4, 64), (64, 66), (66, N)], [(0, 300), (300, 429), (429, N)],
        [(0, 560)] + [(t, t + 1) for t in range(560, 568)]]
    for cuts in cuts_of:
        line = line_of(4, N + 42, 1, m["kv_rank"] + m["rot_dim"], m["kv_rank"] + m["rot_dim"], TORCH[dtype], seed=3)
        got = run_mixer(mixer, hs, cuts, hidden, dtype, line)
        for g, wnt, mv in zip(got, want, moved):
            check(g, wnt[:len(g)], dtype, f"cuts {cuts[:4]}", mv[:len(g)] if dtype == "bfloat16" else None)
    # two calls (stored, and added) for each of the six long portions
    assert len(calls) == (12 if formed and dtype == "bfloat16" else 0)
    rt.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ff,limit", [(64, 96, 0.7), (70, 90, 1.6), (256, 520, 2.5), (72, 34, 0.3)])
def test_the_clamped_feed_forward(dtype, hidden, ff, limit):
    """Inputs so large that gate and up pass the limit on both sides."""
    part = FEED_FORWARDS.build(PartSpec("gated_mlp", {
        "hidden_size": hidden, "intermediate_size": ff, "activation": "clamped_swish", "limit": limit,
        "names": {"gate": "gate", "up": "up", "down": "down"}}), "y.")
    w, wp = part_weights(part, seed=ff, std=2.0 / np.sqrt(hidden))
    rt = Runtime(TORCH[dtype])
    part.bind(to_dev(w, dtype), rt)
    rng = np.random.default_rng(ff)
    for T in (1, 5, 17, 70, 300):
        h = rounded(rng.normal(size=(T, hidden)), dtype)
        want = plain.clamped_dense(h, wp, "y.", limit)
        z = h @ wp["y.gate"].T
        assert (z > limit).mean() > 0.05 and (z < -limit).mean() > 0.05
        hd, step = torch.tensor(h).to(TORCH[dtype]).to(DEV), make_step([(0, 0, [0] * T, [])])
        for store in (True, False):
            x = torch.full((T, hidden), 0.5, device=DEV)
            pending = part.forward(hd, x, step, store=store)
            if pending is not None:
                if store:
                    x.zero_()
                settle(x, pending)
            close(x.cpu().numpy() - (0.0 if store else 0.5), want, dtype, f"{T} tokens, store {store}")
    rt.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,top,ff,hidden,groups", [
    (10, 3, 26, 72, (5, 2)), (6, 1, 14, 30, (3, 1)), (32, 6, 64, 128, (8, 3)), (12, 12, 32, 64, None),
    (256, 8, 32, 64, (32, 5)), (9, 3, 40, 48, (1, 1)), (5, 2, 96, 64, (5, 3)), (64, 4, 32, 64, (2, 1))])
def test_experts_chosen_by_scores_among_groups(dtype, experts, top, ff, hidden, groups):
    """The choice itself (exactly, for logits that are no close call), with corrections that make
    choice scores negative, and the experts' weighted sum."""
    count, keep = groups or (1, 1)
    part = FEED_FORWARDS.build(PartSpec("routed_experts", {
        "hidden_size": hidden, "experts": experts, "top": top, "intermediate_size": ff,
        "activation": "silu", "weights": "sigmoid", "groups": count, "keep_groups": keep,
        "shared_gate": False,
        "names": {"router": "router", "correction": "correction", "expert": "e{}.", "shared": "shared.",
                  "gate": "gate", "up": "up", "down": "down"}}), "y.")
    w, wp = part_weights(part, seed=experts, std=0.2)
    rng = np.random.default_rng(ff)
    w["y.correction"] = torch.tensor(rng.normal(size=experts) * 0.7).to(torch.bfloat16)
    wp["y.correction"] = w["y.correction"].double().numpy()
    rt = Runtime(TORCH[dtype])
    part.bind(to_dev(w, dtype), rt)
    seen = []
    part.probe = lambda p, step, ids: seen.append(ids.cpu().numpy().copy())
    mlp = {"router": {"top": top, "groups": {"count": count, "keep": keep}}}
    for T in (1, 2, 7, 9, 40, 65, 300):
        h = rounded(rng.normal(size=(T, hidden)), dtype)
        z = h @ wp["y.router"].T
        # a close call (of experts or of groups) may go either way after rounding: no such token
        for t in range(T):
            s = plain.sigmoid(z[t]) + wp["y.correction"]
            chosen = plain.choose(z[t], wp["y.correction"], top, count, keep)[0]
            for _ in range(3):
                near = plain.choose(z[t] + rng.normal(size=experts) * 1e-3, wp["y.correction"], top, count, keep)[0]
                if sorted(near) != sorted(chosen):
                    h[t] = h[t - 1] if t else h[t] * 0.0
                    break
        z = h @ wp["y.router"].T
        want = plain.routed_experts(h, wp, "y.", mlp)
        hd, step = torch.tensor(h).to(TORCH[dtype]).to(DEV), make_step([(0, 0, [0] * T, [])])
        y = part.forward_parts(hd, step)
        assert y.shape == (top, T, hidden)
        close(y.double().sum(0).cpu().numpy(), want, dtype, f"{T} tokens")
        for t in range(T):
            if np.abs(h[t]).max() > 0:
                assert sorted(seen[-1][t]) == sorted(plain.choose(z[t], wp["y.correction"], top, count, keep)[0]), t
        x = torch.full((T, hidden), 0.5, device=DEV)
        part.forward(hd, x, step)
        close(x.cpu().numpy() - 0.5, want, dtype, f"{T} tokens, added")
    rt.check()


@pytest.mark.parametrize("parts", [1, 3])
def test_router_ties_and_groups_of_one_kernel_and_of_two(parts):
    """Equal scores: the lower expert and the lower group; the fused kernel of few tokens and the
    two kernels of many make the same choice."""
    rng = np.random.default_rng(parts)
    E, top, count, keep, T = 24, 5, 6, 3, 50
    # many equal logits, whose sums of two are equal only where the two are
    z = np.concatenate([rng.choice([0.0, 1.0, 3.0], size=(1, T, E)), np.zeros((parts - 1, T, E))])
    corr = np.zeros(E)
    want = [plain.choose(z[:, t].sum(0), corr, top, count, keep) for t in range(T)]
    zd = f32(z) if parts > 1 else f32(z[0])
    for fused in (True, False):
        ids = torch.empty((T, top), dtype=torch.int32, device=DEV)
        w = torch.empty((T, top), dtype=torch.float32, device=DEV)
        if fused:
            max_tiles = T * top // 8 + 1 + E
            plan = torch.empty((2 + E + T * top + 2 * max_tiles,), dtype=torch.int32, device=DEV)
            K.moe_route_plan(zd, E, top, E, ids, w, None, 8, max_tiles, plan, K.ROUTE_SIGMOID, f32(corr),
                             1.5, E, count, keep)
        else:
            K.moe_route(zd, E, top, E, ids, w, None, K.ROUTE_SIGMOID, f32(corr), 1.5, count, keep)
        for t in range(T):
            assert ids[t].tolist() == want[t][0], (fused, t)
            assert np.allclose(w[t].cpu().numpy(), 1.5 * np.array(want[t][1]), rtol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("with_ff", [True, False])
def test_a_block_that_norms_both_sides(dtype, with_ff):
    """Sublayers that are known functions (one gives rows that are still to be added up), three
    blocks in a row: what is pending is normed and added by the next block's kernel."""
    H, T = 48, 6
    rt = Runtime(TORCH[dtype])

    class Known:
        def forward(self, h, x, *args):
            x += 2.0 * h.float() + 1.0

    class Rows:
        def forward_parts(self, h, step):
            return torch.stack([h.float(), -4.0 * h.float() ** 2], dim=1).transpose(0, 1)

    norms = {n: NORMS.build(PartSpec("layernorm", {"name": n, "size": H, "eps": 1e-4, "bias": True}))
             for n in ("mixer", "mixer_out", "feed_forward", "feed_forward_out")}
    block = BLOCKS.build(PartSpec("sandwich_residual", {"feed_forward": with_ff}), "", mixer=Known(),
                         feed_forward=Rows(), norms=norms)
    wp = {}
    for i, part in enumerate(norms.values()):
        w, p = part_weights(part, seed=i, std=0.5)
        part.bind(to_dev(w, dtype), rt)
        wp.update(p)
    block.bind({}, rt)
    norm = lambda x, n: plain.layer_norm(x, wp[n], wp[n + ".b"], 1e-4)
    x = np.random.default_rng(0).normal(size=(T, H))
    xd, step, want, pending = f32(x), make_step([(0, 0, [0] * T, [])]), x, None
    for _ in range(3):
        h = rounded(norm(want, "mixer"), dtype)
        want = want + norm(2.0 * h + 1.0, "mixer_out")
        if with_ff:
            h = rounded(norm(want, "feed_forward"), dtype)
            want = want + norm(h - 4.0 * h ** 2, "feed_forward_out")
        pending = block.forward(xd, step, None, None, True, pending=pending)
    settle(xd, pending)
    close(xd.cpu().numpy(), want, dtype, "three blocks")


# ---------------------------------------------------------------------------- the engine
def engine_of(model, dtype, **kw):
    kw.setdefault("max_tokens", 2048)
    eng = Engine.from_folder(model.folder, dtype=dtype, **kw)
    eng.choices = Choices(eng) if dtype == "bfloat16" else None
    return eng


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompts_and_states_after_every_layer_run(small, dtype):
    eng = engine_of(small, dtype)
    for n in small.prompt_lens:
        ids = small.tokens(n, seed=n)
        states = []
        eng.on_state = lambda name, x: states.append((name, x.cpu().numpy().copy()))
        slot = eng.open()
        out = eng.step([Entry(slot, ids, list(range(n)))]).cpu().numpy()
        eng.on_state = None
        eng.close(slot)
        want_states, alone = [], []     # alone: how far rounding alone moves each state
        want, moved = expected(small, eng, slot, ids, dtype, want_states, alone)
        check(out, want, dtype, f"{small.name}: whole prompt of {n}", moved)
        slot = eng.open()           # and without anyone looking at the residual in between
        out = eng.step([Entry(slot, ids, list(range(n)))]).cpu().numpy()
        eng.close(slot)
        check(out, expected(small, eng, slot, ids, dtype)[0], dtype,
              f"{small.name}: whole prompt of {n}, sums left pending", moved)
        runs = [x for name, x in states if name.startswith("run")]
        assert len(runs) == len(want_states) == small.runs
        for i, (got, ref) in enumerate(zip(runs, want_states)):
            err = np.abs(got - ref).max() / max(1.0, np.abs(ref).max())
            bound = F32_TOL
            if dtype == "bfloat16":
                bound = max(0.02, 3.0 * np.abs(alone[i] - ref).max() / max(1.0, np.abs(ref).max()))
            assert err <= bound, (n, i, err)
    eng.rt.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_against_token_by_token_decoding(small, dtype):
    """The last tokens one by one through the cache, across a page border and past every window,
    and a sequence that is decoded from its second token on."""
    eng = engine_of(small, dtype)
    for n, head in ((75, 58), (12, 1), (170, 126)):
        ids = small.tokens(n, seed=100 + n)
        slot = eng.open()
        got = [eng.step([Entry(slot, ids[:head], [head - 1])]).cpu().numpy()]
        for t in range(head, n):
            got.append(eng.step([Entry(slot, [ids[t]])]).cpu().numpy().copy())
        assert eng.length(slot) == n
        eng.close(slot)
        want, moved = expected(small, eng, slot, ids, dtype)
        check(np.concatenate(got), want[head - 1:], dtype,
              f"{n} tokens after a prompt of {head}", None if moved is None else moved[head - 1:])
    eng.rt.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [2, 7, 64])
def test_portions_of_prompts(small, dtype, chunk):
    eng = engine_of(small, dtype, prefill_chunk=chunk)
    n = 131
    ids = small.tokens(n, seed=500 + chunk)
    slot = eng.open()
    want = [0, 1, 62, 63, 64, 65, n - 1]
    out = eng.step([Entry(slot, ids, want)]).cpu().numpy()
    eng.close(slot)
    ref, moved = expected(small, eng, slot, ids, dtype)
    check(out, ref[want], dtype, f"{n} tokens in passes of {chunk}",
          None if moved is None else moved[want])
    slot = eng.open()
    got = [eng.step([Entry(slot, ids[a:b], list(range(b - a)))]).cpu().numpy()
           for a, b in ((0, 3), (3, 5), (5, 66), (66, n))]
    eng.close(slot)
    ref, moved = expected(small, eng, slot, ids, dtype)
    check(np.concatenate(got), ref, dtype, "steps of 3, 2, 61 and 65 tokens", moved)
    eng.rt.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batches_against_each_alone_with_reuse(small, dtype):
    """Batches of unequal requests, one after another in three slots and just enough pages:
    every logit equals that of the request's own whole pass; slots and pages are given back
    and used again."""
    lens = small.prompt_lens + [2, 65, 33]
    decode = [small.decode_steps, 3, 1, small.decode_steps, 5, 2, 4][:len(lens)]
    lens = lens[:len(decode)]
    pages = max(sum(-(-(n + d) // 64) for n, d in list(zip(lens, decode))[b0:b0 + 3])
                for b0 in range(0, len(lens), 3))
    eng = engine_of(small, dtype, max_tokens=64 * pages, max_slots=3)
    reqs = [small.tokens(n + d, seed=200 + i) for i, (n, d) in enumerate(zip(lens, decode))]
    for b0 in range(0, len(reqs), 3):
        idx = list(range(b0, min(b0 + 3, len(reqs))))
        slots = {i: eng.open() for i in idx}
        mine = dict(slots)
        got = {i: {} for i in idx}
        out = eng.step([Entry(slots[i], reqs[i][:lens[i]]) for i in idx]).cpu().numpy()
        for row, i in enumerate(idx):
            got[i][lens[i] - 1] = out[row:row + 1]
        at = {i: lens[i] for i in idx}
        while True:
            for i in [i for i in idx if i in slots and at[i] == len(reqs[i])]:
                eng.close(slots.pop(i))
            live = [i for i in idx if i in slots]
            if not live:
                break
            out = eng.step([Entry(slots[i], [reqs[i][at[i]]]) for i in live]).cpu().numpy()
            for row, i in enumerate(live):
                got[i][at[i]] = out[row:row + 1].copy()
                at[i] += 1
        for i in idx:
            ref, moved = expected(small, eng, mine[i], reqs[i], dtype)
            places = sorted(got[i])
            check(np.concatenate([got[i][t] for t in places]), ref[places], dtype, f"request {i}",
                  None if moved is None else moved[places])
    assert all(eng.book.held_pages(g) == 0 for g in range(len(eng.plans)))
    assert eng.book.slots.free == 3
    assert eng.faults() == []
    eng.rt.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_batch_mates_do_not_matter(small, dtype):
    eng = engine_of(small, dtype)
    a = small.tokens(70, seed=1)
    others = [small.tokens(n, seed=2 + n) for n in (3, 129)]
    s = eng.open()
    alone = [eng.step([Entry(s, a[:66], [0, 64, 65])]).cpu().numpy()]
    alone += [eng.step([Entry(s, [t])]).cpu().numpy().copy() for t in a[66:]]
    eng.close(s)
    slots = [eng.open() for _ in range(3)]
    out = eng.step([Entry(slots[0], others[0], []), Entry(slots[1], a[:66], [0, 64, 65]),
                    Entry(slots[2], others[1], [])]).cpu().numpy()
    tol = 1e-5 if dtype == "float32" else 3e-2
    scale = np.abs(alone[0]).max()
    assert np.abs(out - alone[0]).max() <= tol * scale
    for k, t in enumerate(a[66:]):
        out = eng.step([Entry(slots[0], [5]), Entry(slots[1], [t]), Entry(slots[2], [7])])
        assert np.abs(out.cpu().numpy()[1:2] - alone[1 + k]).max() <= tol * scale
    eng.rt.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_from_the_first_token(small_a, dtype):
    small = small_a
    eng = engine_of(small, dtype, max_tokens=512)
    ids = small.tokens(200, seed=300)
    slot = eng.open()
    got = [eng.step([Entry(slot, [t])]).cpu().numpy().copy() for t in ids]
    eng.close(slot)
    want, moved = expected(small, eng, slot, ids, dtype)
    check(np.concatenate(got), want, dtype, "200 tokens one by one", moved)
    eng.rt.check()


def test_decode_graphs_replay_what_was_computed(small_a):
    """A replayed step blends with the values of its own pass."""
    small = small_a
    ids = [small.tokens(40 + 3 * i, seed=600 + i) for i in range(2)]
    for dtype in DTYPES:
        outs = {}
        for graphs in (True, False):
            eng = engine_of(small, dtype, max_tokens=1024)
            if eng.choices is not None:
                for i in eng.choices.layers:        # nobody looks at the choices here
                    eng.model.layers[i].feed_forward.probe = None
            eng.use_graphs = graphs
            slots = [eng.open() for _ in ids]
            eng.step([Entry(s, r[:30], []) for s, r in zip(slots, ids)])
            outs[graphs] = [eng.step([Entry(s, [r[t]]) for s, r in zip(slots, ids)]).cpu().numpy().copy()
                            for t in range(30, 40)]
            assert len(eng.graphs) == (1 if graphs else 0)
            eng.rt.check()
        for a, b in zip(outs[True], outs[False]):
            assert np.array_equal(a, b)
        if dtype == "float32":
            for row, r in enumerate(ids):
                check(np.concatenate([o[row:row + 1] for o in outs[True]]),
                      small.reference(r)[30:40], dtype, f"row {row}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_generation_runs_pick_what_single_steps_pick(small, dtype):
    """The generation loop decodes in runs whose token ids and positions move on in device
    memory; a sequence alone must get the very tokens that the step function gives it one step
    at a time (the same kernels on the same numbers)."""
    client = LlmClient(small.folder, dtype=dtype, max_batch=2, cache_tokens=1024)
    eng = client.engine
    for n in (1, 70):
        p = small.tokens(n, seed=900 + n)
        got = client.generate([p], max_tokens=8, temperature=0.0, stop=[])[0]
        slot = eng.open()
        logits = eng.step([Entry(slot, p)]).cpu().numpy()
        want = []
        for _ in range(8):
            want.append(int(logits[-1].argmax()))
            logits = eng.step([Entry(slot, [want[-1]])]).cpu().numpy()
        eng.close(slot)
        assert got == want, (n, got, want)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_point(small, dtype):
    client = LlmClient(small.folder, dtype=dtype, max_batch=3, cache_tokens=1024)
    prompts = [small.tokens(n, seed=800 + n) for n in (4, 70, 17, 1)]
    steps = small.decode_steps
    got = client.generate(prompts, max_tokens=steps, temperature=0.0, stop=[])
    for p, tokens in zip(prompts, got):
        assert len(tokens) == steps
        ids = list(p)
        for i, a in enumerate(tokens):
            routing = plain.Routing()
            logits = small.reference(ids, routing=routing)[-1]
            if dtype == "bfloat16" and min(routing.margins.values(), default=1.0) < routing.close:
                break          # a router's close call: 16 bits may take the other side from here on
            order = np.argsort(-logits, kind="stable")
            if a != int(order[0]):
                # a 16-bit run may leave the plain choice at a near tie only
                margin = float(logits[order[0]] - logits[order[1]])
                assert dtype == "bfloat16" and margin < 0.06 * logits.std(), (i, a, margin)
                break
            ids.append(a)
    assert all(client.engine.book.held_pages(g) == 0 for g in range(len(client.engine.plans)))


def test_steps_replayed_through_the_trace_runner(small_a, tmp_path):
    """``bin/trace_run`` as a user runs it: requests of unequal lengths start in one step, go on
    by one token together, and the shorter ones end earlier."""
    import json
    import subprocess
    import sys
    from tests.conftest import ROOT
    small = small_a
    reqs = {f"q{i}": small.tokens(n, seed=950 + i) for i, n in enumerate((3, 75, 133))}
    at = {r: len(ids) - 2 - i for i, (r, ids) in enumerate(reqs.items())}
    steps = [{"step": 0, "end": [], "entries": [
        {"id": r, "tokens": ids[:at[r]], "want": [at[r] - 1]} for r, ids in reqs.items()]}]
    expect = {0: [(r, at[r] - 1) for r in reqs]}
    live = list(reqs)
    while live:
        n = len(steps)
        expect[n] = [(r, at[r]) for r in live]
        entries = [{"id": r, "tokens": [reqs[r][at[r]]], "want": [0]} for r in live]
        for r in live:
            at[r] += 1
        ended = [r for r in live if at[r] == len(reqs[r])]
        steps.append({"step": n, "entries": entries, "end": ended})
        live = [r for r in live if r not in ended]
    for dtype in DTYPES:
        out = tmp_path / dtype
        p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model",
                            small.folder, "--dtype", dtype, "--out", str(out), "--max-tokens",
                            str(sum(len(ids) for ids in reqs.values()))],
                           input="".join(json.dumps(s) + "\n" for s in steps),
                           capture_output=True, text=True, timeout=900)
        assert p.returncode == 0, p.stderr[-3000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == \
            [f"done {s['step']}" for s in steps]
        refs = {r: small.reference(ids) for r, ids in reqs.items()}
        moved = {r: small.rounded(ids, dtype) for r, ids in reqs.items()}
        for step, wanted in expect.items():
            got = np.fromfile(str(out / f"{step}.f32"), dtype="<f4").reshape(-1, small.doc["vocab"])
            check(got, np.stack([refs[r][t] for r, t in wanted]), dtype, f"step {step}",
                  None if dtype != "bfloat16" else np.stack([moved[r][t] for r, t in wanted]))
