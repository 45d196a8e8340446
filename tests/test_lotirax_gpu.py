"""The Lotirax family on a B200 against the plain implementation, in float32 and bfloat16:
each mechanism alone (with weights or inputs made so that a fault shows), then the engine on
four small models of other sizes: whole prompts with the residual after every layer run,
prompts against token-by-token decoding, portions down to two tokens, unequal batches against
each request alone, slots and pages used again, the first tokens, long decoding past windows
and page borders, decode graphs, and greedy generation through the entry point."""
import os
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from mormot2_ai_b200 import Engine, Entry, LlmClient, LotiraxConfig, PartSpec, Runtime, WeightsError
from mormot2_ai_b200 import kernels as K
from mormot2_ai_b200.cache.pages import PAGE, pages_for
from mormot2_ai_b200.cache.storage import CacheLine
from mormot2_ai_b200.parts import BLOCKS, ENTRIES, FEED_FORWARDS, MIXERS, NORMS, POSITIONS
from mormot2_ai_b200.parts.block import BranchSums, settle
from mormot2_ai_b200.weights import random_tensors
from tests.gpu_helpers import DEV, make_step
from tests.lotirax_models import SMALL, SmallModel, _att, _rot
from tests.plain import lotirax_plain as plain

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module", params=sorted(SMALL))
def small(request, tmp_path_factory):
    return SmallModel(request.param, str(tmp_path_factory.mktemp("lotirax_" + request.param)))


@pytest.fixture(scope="module")
def small_a(tmp_path_factory):
    return SmallModel("A", str(tmp_path_factory.mktemp("lotirax_A_only")))


# The bounds of this family's comparisons, set from what was measured. float32: the largest
# difference of a logit over the largest logit. bfloat16: per position, the largest difference of
# a logit over the spread of the plain logits, bounded in the median, the ninth decile and the
# worst position of a comparison, and never tighter than three times what the plain
# implementation itself moves by when it rounds what a 16-bit run rounds.
F32_TOL = 1e-5
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
    return w, {k: v.numpy() if v.dtype == torch.int32 else v.double().numpy() for k, v in w.items()}


def to_dev(w, dtype):
    return {k: (v if v.dtype == torch.int32 else v.to(TORCH[dtype])).to(DEV) for k, v in w.items()}


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
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [64, 70, 1536, 5120])
def test_scaled_sums_of_sublayers_and_the_norm_after_them(dtype, H):
    T = 5
    rng = np.random.default_rng(H)
    f32 = lambda a: torch.tensor(a, dtype=torch.float32, device=DEV)
    x = rng.normal(size=(T, H))
    parts = rng.normal(size=(3, T, H))
    rows = rng.normal(size=(T, 2, H))           # row t * 2 + k: two parts a token
    stored = rng.normal(size=(T, H))
    s1, s2, w = rng.normal(size=(3, H))
    terms = [(f32(parts), 0.7, f32(s1)), (f32(rows).transpose(0, 1), 0.5, f32(s2)),
             (f32(stored), 1.5, None)]
    want = x + 0.7 * s1 * parts.sum(0) + 0.5 * s2 * rows.sum(1) + 1.5 * stored
    for n in range(4):
        part = x.copy()
        for y, f, s in [(parts.sum(0), 0.7, s1), (rows.sum(1), 0.5, s2), (stored, 1.5, 1.0)][:n]:
            part = part + f * s * y
        xd, out = f32(x), torch.empty((T, H), dtype=TORCH[dtype], device=DEV)
        K.branch_norm(xd, terms[:n], f32(w), 1e-5, out)
        close(xd.cpu().numpy(), part, "float32", f"{n} terms")
        close(out.double().cpu().numpy(), plain.unit_rms(part, 1e-5) * w, dtype, f"norm after {n}")
    many = rng.normal(size=(9, T, H))           # more parts than one round of loads
    xd, out = f32(x), torch.empty((T, H), dtype=TORCH[dtype], device=DEV)
    K.branch_norm(xd, [(f32(many), 0.2, f32(s1)), terms[2]], f32(w), 1e-5, out)
    part = x + 0.2 * s1 * many.sum(0) + 1.5 * stored
    close(xd.cpu().numpy(), part, "float32", "nine parts and one")
    close(out.double().cpu().numpy(), plain.unit_rms(part, 1e-5) * w, dtype, "norm after ten parts")
    xd = f32(x)
    K.branch_norm(xd, terms)                    # without a norm
    close(xd.cpu().numpy(), want, "float32", "settled")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [24, 30, 128])
def test_a_pass_starts_from_the_projection_and_its_vector(dtype, size):
    rt = Runtime(TORCH[dtype])
    for row in range(3):
        part = ENTRIES.build(PartSpec("pass_projection", {
            "names": {"in": "in", "step": "step"}, "rows": 3, "row": row, "size": size}))
        w, wp = part_weights(part, seed=4, std=0.3)
        part.bind(to_dev(w, dtype), rt)
        rng = np.random.default_rng(row)
        for T in (1, 3, 90):
            x = rng.normal(size=(T, size))
            table, ids = rounded(rng.normal(size=(11, size)), "bfloat16"), rng.integers(0, 11, T)
            x0 = table[ids] * 0.7
            y, scale = rng.normal(size=(2, T, size)), rng.normal(size=size)
            f32 = lambda a: torch.tensor(a, dtype=torch.float32, device=DEV)
            xd = f32(x)
            emb = SimpleNamespace(table=torch.tensor(table, device=DEV).to(TORCH[dtype]), scale=0.7)
            step = make_step([(0, 0, ids.tolist(), [])])
            pending = part.forward(xd, step, emb,
                                   pending=BranchSums([(f32(y), 0.3, f32(scale))]))
            settle(xd, pending)
            want = plain.pass_start(x + 0.3 * scale * y.sum(0), x0,
                                    {"loop.in": wp["in"], "loop.step": wp["step"]}, row)
            close(xd.cpu().numpy(), want, dtype, f"pass {row}, {T} tokens")
    rt.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nh,nkv,dim,vd,rot", [
    (4, 2, 18, 10, _rot(12, 500.0, 3.0)), (3, 1, 7, 5, _rot(4, 20.0)), (5, 5, 64, 128, _rot(64, 1e4, 8.0, 128)),
    (2, 1, 130, 300, None), (2, 2, 128, 64, _rot(100, 900.0))])
def test_biases_norms_and_rotation_of_two_maps(dtype, nh, nkv, dim, vd, rot):
    if vd > 256 and dim % 2:
        pytest.skip("value rows of odd sizes end at 256")
    eps, cd = 1e-3, TORCH[dtype]
    rng = np.random.default_rng(dim)
    width = 2 * (nh + nkv) * dim + nkv * vd
    seqs = [(1, 0, [0] * 3, []), (0, 60, [0] * 6, []), (2, 1000, [0], [])]
    if dim >= 64:                    # enough tokens for the form of long steps
        seqs.append((3, 50, [0] * 130, []))
    pos = np.concatenate([np.arange(past, past + len(t)) for _, past, t, _ in seqs])
    slots = np.concatenate([[slot] * len(t) for slot, _, t, _ in seqs])
    step, T = make_step(seqs), len(pos)
    bias, wq, wk = rng.normal(size=width), *(1.0 + 0.3 * rng.normal(size=(2, dim)))
    f32 = lambda a: torch.tensor(a, dtype=torch.float32, device=DEV)
    position = None
    if rot:
        params = {"theta": rot["base"], "rot_dim": rot["dims"]}
        if rot.get("scaling"):
            position = POSITIONS.build(PartSpec("rope_yarn", {**params, **rot["scaling"]}))
        else:
            position = POSITIONS.build(PartSpec("rope_half", {**params, "rounding": "once"}))
        position.bind({}, Runtime(cd))
    for form in ("stored", "split", "no bias"):
        parts = rng.normal(size=(3, T, width))
        rows = parts.sum(0)
        if form != "split":
            rows = rounded(rows, dtype)
            given = torch.tensor(rows, dtype=cd, device=DEV)
        else:
            given = f32(parts)
        full = rows + (bias if form != "no bias" else 0.0)
        q, k, v = np.split(full, [2 * nh * dim, 2 * (nh + nkv) * dim], axis=1)
        q = plain.unit_rms(q.reshape(T, -1, dim), eps) * wq
        k = plain.unit_rms(k.reshape(T, -1, dim), eps) * wk
        if rot:
            q, k = plain.rotate_halves(q, pos, rot), plain.rotate_halves(k, pos, rot)
        line = line_of(4, 1024, nkv, 2 * dim, vd, cd)
        q_out = torch.empty((T, 2 * nh * dim), dtype=cd, device=DEV)
        freq, n_rot = position.frequencies() if position else (None, 0)
        K.maps_norm_rope_store(given, f32(bias) if form != "no bias" else None, f32(wq), f32(wk),
                               eps, freq, n_rot, position.amplitude if position else 1.0, step,
                               line, nh, nkv, 2, dim, vd, q_out)
        loose = "bfloat16" if dtype == "bfloat16" else "float32"
        err = np.abs(q_out.double().cpu().numpy().reshape(T, -1, dim) - q).max() / np.abs(q).max()
        assert err < (8e-3 if loose == "bfloat16" else 2e-4), (form, err)   # angles in float32
        table = line.page_table.cpu()
        for t in range(T):
            page = int(table[slots[t], pos[t] // PAGE])
            kc = line.k[page, :, pos[t] % PAGE].double().cpu().numpy()
            vc = line.v[page, :, pos[t] % PAGE].double().cpu().numpy()
            err = np.abs(kc.reshape(-1, dim) - k[t]).max() / np.abs(k).max()
            assert err < (8e-3 if loose == "bfloat16" else 2e-4), (form, t, err)
            close(vc.reshape(-1), v[t], dtype, f"{form}: value {t}")


def attention_reference(q, keys, vals, pos, nkv, scale, lam, factor, eps, window):
    """q [T, nh, 2, d] at positions ``pos``, keys [N, nkv, 2, d], vals [N, nkv, vd]."""
    T, nh = q.shape[:2]
    out = np.zeros((T, nh, vals.shape[-1]))
    for t in range(T):
        lo = max(0, pos[t] + 1 - window) if window else 0
        for h in range(nh):
            g = h // (nh // nkv)
            a = []
            for m in range(2):
                s = keys[lo:pos[t] + 1, g, m] @ q[t, h, m] * scale
                e = np.exp(s - s.max())
                a.append((e / e.sum()) @ vals[lo:pos[t] + 1, g])
            out[t, h] = plain.combine_maps(a[0], a[1], lam, 0.0, eps) * factor
    return out


def fill(line, slot, keys, vals):
    table = line.page_table.cpu().numpy()
    for p in range(0, len(keys), PAGE):
        page = int(table[slot, p // PAGE])
        n = min(PAGE, len(keys) - p)
        line.k[page, :, :n] = torch.tensor(keys[p:p + n]).flatten(2).transpose(0, 1).to(line.k.dtype).to(DEV)
        line.v[page, :, :n] = torch.tensor(vals[p:p + n]).transpose(0, 1).to(line.v.dtype).to(DEV)


SIZES = [(4, 2, 18, 10), (2, 2, 16, 24), (6, 1, 48, 72), (3, 3, 64, 128), (4, 1, 64, 64),
         (2, 1, 72, 136), (20, 1, 40, 56), (1, 1, 128, 256), (2, 1, 130, 300)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nh,nkv,dim,vd", SIZES)
def test_loud_keys_just_inside_and_just_outside_the_window(dtype, nh, nkv, dim, vd):
    """One key whose score in one of the maps stands out, at the window's edge, at page borders
    and far back, for tokens of a prompt and decoded ones: it decides the head's output where
    it is visible and must not be felt where it is not."""
    cd, scale, lam, factor, eps = TORCH[dtype], 0.25, 0.6, 0.35, 1e-5
    rt = Runtime(cd)
    N = 330
    rng = np.random.default_rng(dim + vd)
    direction = rng.normal(size=dim)
    direction /= np.linalg.norm(direction)
    for window in (0, 5, 64, 65, 200):
        for loud in (0, 1, 63, 64, 127, 128, 200, 256):
            keys = rounded(rng.normal(size=(N, nkv, 2, dim)) * 0.3, "bfloat16")
            vals = rounded(rng.normal(size=(N, nkv, vd)), "bfloat16")
            q = rng.normal(size=(N, nh, 2, dim)) * 0.3
            m = loud % 2                                       # the map in which it is loud
            keys[loud, :, m] = rounded(direction * 8.0, "bfloat16")
            q[:, :, m] += direction * 8.0
            q = rounded(q, "bfloat16")
            line = line_of(2, N, nkv, 2 * dim, vd, cd, seed=loud)
            fill(line, 1, keys, vals)
            edge = loud + (window or 200)                      # the first token that misses it
            places = sorted({p for p in (loud, loud + 1, edge - 1, edge, edge + 1, N - 1) if loud <= p < N})
            a = places[0]
            # a prompt's portion that ends at the last token, and single decoded tokens
            step = make_step([(1, a, [0] * (N - a), [])])
            qd = torch.tensor(q[a:].reshape(N - a, -1), dtype=cd, device=DEV)
            out = torch.full((N - a, nh * vd), 9.0, dtype=cd, device=DEV)
            rt.differential_attention(qd, out, step, line, nh, nkv, dim, vd, window, scale, lam,
                                      factor, eps)
            want = attention_reference(q[places], keys, vals, places, nkv, scale, lam, factor, eps, window)
            got = out.double().cpu().numpy().reshape(N - a, nh, vd)[[p - a for p in places]]
            close(got, want, dtype, f"window {window}, loud {loud}, prompt")
            for i, p in enumerate(places):
                step = make_step([(1, p, [0], [])])
                qd = torch.tensor(q[p].reshape(1, -1), dtype=cd, device=DEV)
                o1 = torch.full((1, nh * vd), 9.0, dtype=cd, device=DEV)
                rt.differential_attention(qd, o1, step, line, nh, nkv, dim, vd, window, scale, lam,
                                          factor, eps)
                close(o1.double().cpu().numpy().reshape(nh, vd), want[i], dtype,
                      f"window {window}, loud {loud}, decoded at {p}")
    rt.check()


def run_mixer(mixer, hs, cuts, hidden, dtype, line):
    """Feeds each sequence of ``hs`` (float arrays [n, hidden]) through the mixer in the
    portions that ``cuts`` names (all sequences of a step together), from slots 2, 0, 1, ...;
    returns what the mixer added to the residual, per sequence."""
    slots = [2, 0, 1, 3][:len(hs)]
    outs = [[] for _ in hs]
    for lo, hi in cuts:
        seqs, rows = [], []
        for b, h in enumerate(hs):
            a, e = min(lo, len(h)), min(hi, len(h))
            if e > a:
                seqs.append((slots[b], a, [0] * (e - a), []))
                rows.append((b, a, e))
        if not seqs:
            continue
        step = make_step(seqs)
        h = torch.tensor(np.concatenate([hs[b][a:e] for b, a, e in rows])).to(TORCH[dtype]).to(DEV)
        x = torch.full((h.shape[0], hidden), 0.5, device=DEV)
        pending = mixer.forward(h, x, step, line, None, True)
        if pending is not None:                 # split sums that the next norm would add
            settle(x, pending)
        got, at = x.cpu().double().numpy() - 0.5, 0
        for b, a, e in rows:
            outs[b].append(got[at:at + e - a])
            at += e - a
    return [np.concatenate(o) for o in outs]


MIXES = [(_att(4, 2, 18, 10, 0.4, 0.3, 21, _rot(12, 500.0, 3.0)), 72),
         (_att(2, 2, 64, 128, 0.2, 0.7, 65, _rot(64, 1e4, 8.0, 128)), 96),
         (_att(8, 1, 32, 48, 0.3, 0.5, 0, _rot(20, 300.0)), 64),
         (_att(1, 1, 128, 160, 0.1, 0.4, 50, None), 56)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer,hidden", MIXES, ids=[str(i) for i in range(len(MIXES))])
def test_differential_attention_as_a_mixer(dtype, layer, hidden):
    """Whole portions, small ones and single tokens of three unequal sequences."""
    eps, m = 1e-4, layer["mixer"]
    cfg = LotiraxConfig.from_dict({"architecture": "Lotirax", "vocab": 9, "width": hidden,
                                   "norm": {"eps": eps}, "layers": [layer]})
    positions = {}
    spec = cfg._mixer(m, positions)
    rt = Runtime(TORCH[dtype])
    positions = {k: POSITIONS.build(v) for k, v in positions.items()}
    for p in positions.values():
        p.bind({}, rt)
    mixer = MIXERS.build(spec, "x.", positions=positions)
    w, wp = part_weights(mixer, seed=11, std=0.2)
    for n, t in w.items():
        if n.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t.mul_(2.0)
    wp = {k: v.double().numpy() for k, v in w.items()}
    mixer.bind(to_dev(w, dtype), rt)
    assert abs(mixer.lam - plain.map_weight(wp, "x.mix.", m["diff"])) < 1e-6
    rng = np.random.default_rng(7)
    hs = [rounded(rng.normal(size=(n, hidden)), dtype) for n in (150, 3, 67)]
    want = [plain.differential_attention(h, wp, "x.mix.", m, eps) for h in hs]
    moved = [plain.differential_attention(h, wp, "x.mix.", m, eps, rnd=plain.bfloat16) for h in hs]
    for cuts in ([(0, 150)], [(0, 2), (2, 4), (4, 64), (64, 66), (66, 150)],
                 [(0, 60)] + [(t, t + 1) for t in range(60, 72)]):
        line = line_of(4, 192, m["kv_heads"], 2 * m["dim"], m["vdim"], TORCH[dtype], seed=3)
        got = run_mixer(mixer, hs, cuts, hidden, dtype, line)
        for g, wnt, mv in zip(got, want, moved):
            check(g, wnt[:len(g)], dtype, f"cuts {cuts[:4]}", mv[:len(g)] if dtype == "bfloat16" else None)
    rt.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,top,ff,shared,hidden", [
    (5, 2, 26, 34, 72), (3, 1, 14, 0, 30), (9, 4, 64, 96, 128), (16, 1, 96, 32, 64), (4, 4, 40, 8, 48)])
def test_experts_that_a_table_names(dtype, experts, top, ff, shared, hidden):
    vocab = 60
    part = FEED_FORWARDS.build(PartSpec("table_experts", {
        "hidden_size": hidden, "vocab_size": vocab, "experts": experts, "top": top,
        "intermediate_size": ff, "shared_size": shared, "activation": "relu_squared",
        "names": {"table": "table", "expert": "e{}.", "shared": "shared.", "up": "up",
                  "down": "down"}}), "y.")
    w, wp = part_weights(part, seed=experts, std=0.3)
    rt = Runtime(TORCH[dtype])
    part.bind(to_dev(w, dtype), rt)
    rng = np.random.default_rng(ff)
    mlp = {"router": {"top": top}, "shared": {"ff": shared} if shared else None}
    for T in (1, 2, 7, 8, 9, 40, 300):
        ids = rng.integers(0, vocab, T)
        if T == 40:
            ids[:] = 17                          # every token asks for the same experts
        h = rounded(rng.normal(size=(T, hidden)), dtype)
        x = torch.full((T, hidden), 0.5, device=DEV)
        step = make_step([(0, 0, ids.tolist(), [])])
        for again in range(2):                   # the second time the step's lists are there
            part.forward(torch.tensor(h).to(TORCH[dtype]).to(DEV), x, step)
        want = 0.5 + 2.0 * plain.table_experts(h, ids, wp, "y.", mlp)
        close(x.cpu().numpy(), want, dtype, f"{T} tokens")
    rt.check()


def test_a_table_that_names_no_expert_is_refused():
    part = FEED_FORWARDS.build(PartSpec("table_experts", {
        "hidden_size": 16, "vocab_size": 8, "experts": 3, "top": 1, "intermediate_size": 8,
        "activation": "relu_squared",
        "names": {"table": "table", "expert": "e{}.", "shared": "shared.", "up": "up",
                  "down": "down"}}))
    w, _ = part_weights(part)
    for bad in (-1, 3):
        wrong = dict(to_dev(w, "float32"))
        wrong["table"] = wrong["table"].clone()
        wrong["table"][5, 0] = bad
        with pytest.raises(WeightsError):
            part.bind(wrong, Runtime(torch.float32))


@pytest.mark.parametrize("dtype", DTYPES)
def test_sublayers_side_by_side_with_their_scales(dtype):
    """A block whose sublayers are known functions: what it leaves for the residual is
    factor * (scale_1 * mixer + scale_2 * feed-forward) of one norm's output."""
    H, T = 48, 6
    rt = Runtime(TORCH[dtype])

    class Known:
        def __init__(self, factor):
            self.factor = factor

        def forward(self, h, x, *args):
            x += self.factor * h.float()

    norm = NORMS.build(PartSpec("rmsnorm", {"name": "n", "size": H, "eps": 1e-4, "one_plus": True}))
    block = BLOCKS.build(PartSpec("parallel_residual", {
        "hidden_size": H, "factor": 0.3, "scales": {"mixer": "s1", "feed_forward": "s2"}}), "",
        mixer=Known(2.0), feed_forward=Known(-5.0), norms={"input": norm})
    w, wp = {}, {}
    for part in (norm, block):
        a, b = part_weights(part, seed=1, std=0.5)
        w.update(a), wp.update(b)
    for part in (norm, block):
        part.bind(to_dev(w, dtype), rt)
    rng = np.random.default_rng(0)
    x = rng.normal(size=(T, H))
    xd = torch.tensor(x, dtype=torch.float32, device=DEV)
    step = make_step([(0, 0, [0] * T, [])])
    want = x
    pending = None
    for _ in range(3):                            # the next block's norm adds what is pending
        h = rounded(plain.norm_one_plus(want, wp["n"], 1e-4), dtype)
        want = want + 0.3 * (wp["s1"] * 2.0 * h + wp["s2"] * -5.0 * h)
        pending = block.forward(xd, step, None, None, True, pending=pending)
    settle(xd, pending)
    close(xd.cpu().numpy(), want, dtype, "three blocks")


# ---------------------------------------------------------------------------- the engine
def engine_of(model, dtype, **kw):
    kw.setdefault("max_tokens", 2048)
    return Engine.from_folder(model.folder, dtype=dtype, **kw)


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
        want_states = []
        want, moved = small.reference(ids, want_states), small.rounded(ids, dtype)
        check(out, want, dtype, f"{small.name}: whole prompt of {n}", moved)
        slot = eng.open()           # and without anyone looking at the residual in between
        check(eng.step([Entry(slot, ids, list(range(n)))]).cpu().numpy(), want, dtype,
              f"{small.name}: whole prompt of {n}, sums left pending", moved)
        eng.close(slot)
        runs = [x for name, x in states if name.startswith("run")]
        assert len(runs) == len(want_states) == small.runs
        alone = []                  # how far rounding alone moves each state (bfloat16)
        if dtype == "bfloat16":
            small.plain.forward(small.plain_config, small.weights, ids, rnd=small.plain.bfloat16,
                                states=alone)
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
        moved = small.rounded(ids, dtype)
        check(np.concatenate(got), small.reference(ids)[head - 1:], dtype,
              f"{n} tokens after a prompt of {head}", None if moved is None else moved[head - 1:])
    eng.rt.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [2, 7, 64])
def test_portions_of_prompts(small, dtype, chunk):
    eng = engine_of(small, dtype, prefill_chunk=chunk)
    n = 131
    ids = small.tokens(n, seed=500 + chunk)
    ref, moved = small.reference(ids), small.rounded(ids, dtype)
    slot = eng.open()
    want = [0, 1, 62, 63, 64, 65, n - 1]
    out = eng.step([Entry(slot, ids, want)]).cpu().numpy()
    eng.close(slot)
    check(out, ref[want], dtype, f"{n} tokens in passes of {chunk}",
          None if moved is None else moved[want])
    slot = eng.open()
    got = [eng.step([Entry(slot, ids[a:b], list(range(b - a)))]).cpu().numpy()
           for a, b in ((0, 3), (3, 5), (5, 66), (66, n))]
    eng.close(slot)
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
            ref, moved = small.reference(reqs[i]), small.rounded(reqs[i], dtype)
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
    check(np.concatenate(got), small.reference(ids), dtype, "200 tokens one by one",
          small.rounded(ids, dtype))
    eng.rt.check()


def test_decode_graphs_replay_what_was_computed(small_a):
    """A replayed step looks its tokens' experts up anew and reads the lists of its own pass."""
    small = small_a
    ids = [small.tokens(40 + 3 * i, seed=600 + i) for i in range(2)]
    for dtype in DTYPES:
        outs = {}
        for graphs in (True, False):
            eng = engine_of(small, dtype, max_tokens=1024)
            assert eng.use_graphs
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
            logits = small.reference(ids)[-1]
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
