"""The Lotirax family without a GPU: the registry, the model as data (looped layers with cache
lines of their own and the projection that opens a pass), tensor names and shapes, defaults of
absent keys, refusals, tables of random models, and the plain implementation's own
consistency."""
import json
import math

import numpy as np
import pytest
import torch

from mormot2_ai_b200 import ConfigError, DecoderModel, LotiraxConfig, architectures
from mormot2_ai_b200.config.registry import family_of
from mormot2_ai_b200.parts.position import yarn_inverse_frequencies
from mormot2_ai_b200.weights import random_tensors
from tests.lotirax_models import SMALL, _rot, small_doc
from tests.plain import lotirax_plain as plain


def test_registry_and_round_trip():
    assert "Lotirax" in architectures()
    for name in SMALL:
        doc = small_doc(name)
        assert family_of(doc) is LotiraxConfig
        c = LotiraxConfig.from_dict(doc)
        again = LotiraxConfig.from_dict(json.loads(json.dumps(c.to_dict())))
        assert again == c
        assert c.vocab_size == doc["vocab"] and c.hidden_size == doc["width"]
        assert c.num_hidden_layers == len(doc["layers"])


def test_passes_have_lines_of_their_own_and_start_with_a_projection():
    c = LotiraxConfig.from_dict(small_doc("C"))
    spec = c.to_model_spec()
    assert [r.layer for r in spec.schedule] == [0, 1, 2, 1, 2, 1, 2]
    assert [r.cache_line for r in spec.schedule] == list(range(7))
    opened = [(i, r.before.params["row"]) for i, r in enumerate(spec.schedule) if r.before]
    assert opened == [(1, 0), (3, 1), (5, 2)]
    assert all(spec.schedule[i].before.kind == "pass_projection" for i, _ in opened)
    assert c.order() == plain.layer_runs(small_doc("C"))
    assert LotiraxConfig.from_dict(small_doc("D")).order() == [(0, 0), (1, -1), (2, -1)]


def test_tensor_names_shapes_and_lines():
    model = DecoderModel(LotiraxConfig.from_dict(small_doc("A")).to_model_spec())
    shapes = {t.name: t.shape for t in model.tensors()}
    W = 72
    assert shapes["embed"] == (150, W) and shapes["loop.in"] == (W, 2 * W)
    assert shapes["loop.step"] == (2, W) and shapes["final.norm"] == (W,)
    assert shapes["l0.mix.q"] == (4 * 2 * 18, W) and shapes["l0.mix.q.b"] == (4 * 2 * 18,)
    assert shapes["l0.mix.k"] == (2 * 2 * 18, W) and shapes["l0.mix.k.b"] == (2 * 2 * 18,)
    assert shapes["l0.mix.v"] == (2 * 10, W) and shapes["l0.mix.v.b"] == (2 * 10,)
    assert shapes["l0.mix.q.norm"] == shapes["l0.mix.lk2"] == (18,)
    assert shapes["l0.mix.o"] == (W, 4 * 10)
    assert shapes["l0.norm1"] == shapes["l0.ls1"] == shapes["l0.ls2"] == (W,)
    assert "l0.norm2" not in shapes
    assert shapes["l0.mlp.table"] == (150, 2) and shapes["l0.mlp.e4.up"] == (26, W)
    assert shapes["l0.mlp.e0.down"] == (W, 26) and "l0.mlp.e5.up" not in shapes
    assert shapes["l0.mlp.shared.up"] == (34, W) and "l2.mlp.shared.up" not in shapes
    assert shapes["l1.mlp.gate"] == (90, W) and shapes["l1.mlp.down"] == (W, 90)
    # a line keeps the two maps of a key head in one row, values in rows of their own size
    need = model.line_needs[0]
    assert (need.kv_heads, need.head_dim, need.v_dim, need.window) == (2, 36, 10, 21)
    assert model.line_needs[2] == need and not model.state_needs
    # value rows as long as two maps need no pool of their own
    c = DecoderModel(LotiraxConfig.from_dict(small_doc("C")).to_model_spec()).line_needs
    assert c[0].head_dim == 128 and c[0].v_dim == 0 and c[1].v_dim == 64


def test_absent_keys_and_a_layer_without_feed_forward():
    c = LotiraxConfig.from_dict(small_doc("B"))
    assert c.residual_mult == 1.0 and c.loop is None
    spec = c.to_model_spec()
    assert spec.layers[0].mixer.params["window"] == 0
    assert spec.layers[1].feed_forward.kind == "none"
    kinds = {k: p.kind for k, p in spec.positions.items()}
    assert sorted(kinds.values()) == ["rope_half", "rope_half", "rope_yarn"]
    needs = {t.name: t for t in DecoderModel(spec).tensors()}
    assert needs["l1.ls2"].optional and not needs["l0.ls2"].optional
    assert needs["loop.in"].optional and needs["loop.step"].shape == (-1, 40)
    assert needs["head"].must_equal == "embed" and needs["head"].optional
    none = LotiraxConfig.from_dict(small_doc("D")).to_model_spec()
    assert none.layers[2].mixer.params["position"] == ""
    doc = small_doc("B")
    for key in ("kv_heads", "vdim"):
        del doc["layers"][1]["mixer"][key]
    p = LotiraxConfig.from_dict(doc).to_model_spec().layers[1].mixer.params
    assert p["kv_heads"] == 2 and p["vdim"] == 12
    # equal rotations are one encoding of the model
    a = LotiraxConfig.from_dict(small_doc("A")).to_model_spec()
    assert len(a.positions) == 2
    assert a.layers[0].mixer.params["position"] == a.layers[2].mixer.params["position"]


@pytest.mark.parametrize("change,text", [
    (lambda d: d["layers"][0].update(type="other"), "not known"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "key/value heads"),
    (lambda d: d["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=20), "rotating"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=5), "rotating"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(base=0), "base"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(slow=0), "slow"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("factor"), "factor"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda d: d["layers"][0]["mlp"].pop("expert"), "expert"),
    (lambda d: d["layers"][0].update(mlp={"kind": "routed", "ff": 8}), "feed-forward kind"),
    (lambda d: d["loop"].update(stop=0), "stop"),
    (lambda d: d["loop"].update(stop=4), "stop"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_refusals(change, text):
    doc = small_doc("A")
    change(doc)
    with pytest.raises(ConfigError) as e:
        LotiraxConfig.from_dict(doc).to_model_spec()
    assert text in str(e.value)


def _weights(doc, seed):
    model = DecoderModel(LotiraxConfig.from_dict(doc).to_model_spec())
    w = random_tensors(model.tensors(), seed, std=0.15, norm_std=0.2)
    return {k: v.numpy() if v.dtype == torch.int32 else v.double().numpy() for k, v in w.items()}


def test_tables_of_a_random_model_name_different_experts():
    w = _weights(small_doc("A"), 5)
    for name, experts, top in (("l0.mlp.table", 5, 2), ("l2.mlp.table", 7, 3)):
        t = w[name]
        assert t.dtype == np.int32 and t.shape == (150, top)
        assert t.min() == 0 and t.max() == experts - 1
        assert all(len(set(row)) == top for row in t.tolist())


@pytest.mark.parametrize("rot", [_rot(12, 500.0, 3.0), _rot(64, 1e4, 8.0, 128), _rot(10, 90.0, 2.0, 30),
                                 _rot(6, 10.0, 1.5, 4000, 32.0, 1.0), _rot(2, 7.0, 2.0, 9, 1.0, 0.9)])
def test_scaled_frequencies_are_the_encoding_s(rot):
    f, amp = plain.rotary_frequencies(rot)
    s = rot["scaling"]
    got = yarn_inverse_frequencies(rot["base"], rot["dims"], s["factor"], s["original"], s["fast"],
                                   s["slow"])
    assert np.allclose(got, f, rtol=1e-6)
    assert math.isclose(amp, 0.1 * math.log(s["factor"]) + 1.0)


@pytest.mark.parametrize("name", ["A", "B"])
def test_the_plain_implementation_is_causal(name):
    """A prefix gives the logits that the whole sequence gives at its positions."""
    doc = dict(small_doc(name))
    doc.setdefault("residual_mult", 1.0)
    w = _weights(doc, 3)
    ids = np.random.default_rng(1).integers(0, doc["vocab"], 40).tolist()
    whole = plain.forward(doc, w, ids)
    assert np.allclose(plain.forward(doc, w, ids[:17]), whole[:17], rtol=1e-9, atol=1e-9)
    assert np.isfinite(whole).all()


def test_plain_windows_and_the_maps_difference():
    m = plain.visible(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[1].tolist()[:2] == [True, True]
    assert plain.visible(4, None)[3].all() and not plain.visible(4, 2)[3, 1]
    # equal maps: what is left is (1 - lambda) a, whose size the norm takes away again
    a = np.array([[3.0, -4.0]])
    out = plain.combine_maps(a, a, 0.25, 0.4, 0.0)
    assert np.allclose(out, 0.6 * a / math.sqrt(12.5))
    w = {"lq1": np.array([1.0, 0.0]), "lk1": np.array([0.5, 9.0]), "lq2": np.zeros(2), "lk2": np.zeros(2)}
    assert math.isclose(plain.map_weight(w, "", 0.3), math.exp(0.5) - 1.0 + 0.3)


def test_plain_turns_pairs_half_a_rotation_apart():
    x = np.zeros((2, 1, 5))
    x[:, 0, 0], x[:, 0, 4] = 1.0, 7.0
    out = plain.rotate_halves(x, [0, 2], {"dims": 4, "base": 100.0})
    assert np.allclose(out[0], x[0])
    assert np.allclose(out[1, 0], [math.cos(2.0), 0.0, math.sin(2.0), 0.0, 7.0])
