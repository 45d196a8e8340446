"""The Tenusun family without a GPU: the registry, the model as data (norms on both sides of a
sublayer, which layer's values the others are blended with), tensor names and shapes, defaults of
absent keys, refusals, and the plain implementation's own consistency."""
import json
import math

import numpy as np
import pytest

from mormot2_ai_b200 import ConfigError, DecoderModel, PartSpec, TenusunConfig, architectures
from mormot2_ai_b200.config.registry import family_of
from mormot2_ai_b200.parts import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITIONS
from mormot2_ai_b200.weights import random_tensors
from tests.plain import tenusun_plain as plain
from tests.tenusun_models import SMALL, sharpen, small_doc


def test_registry_and_round_trip():
    assert "Tenusun" in architectures()
    for name in SMALL:
        doc = small_doc(name)
        assert family_of(doc) is TenusunConfig
        c = TenusunConfig.from_dict(doc)
        again = TenusunConfig.from_dict(json.loads(json.dumps(c.to_dict())))
        assert again == c
        assert c.vocab_size == doc["vocab"] and c.hidden_size == doc["width"]
        assert c.num_hidden_layers == len(doc["layers"])


def test_tensor_names_shapes_and_lines():
    model = DecoderModel(TenusunConfig.from_dict(small_doc("A")).to_model_spec())
    shapes = {t.name: t.shape for t in model.tensors()}
    W = 70
    for n in ("l0.norm1", "l0.norm1b", "l3.norm2", "l3.norm2b", "final.norm"):
        assert shapes[n] == shapes[n + ".b"] == (W,)
    assert shapes["embed"] == (150, W)
    assert shapes["l0.mix.dq"] == (26, W) and shapes["l0.mix.dq.norm"] == (26,)
    assert shapes["l0.mix.uq"] == (3 * 28, 26) and shapes["l0.mix.dkv"] == (40, W)
    assert shapes["l0.mix.uk"] == (3 * 18, 30) and shapes["l0.mix.uv"] == (3 * 14, 30)
    assert shapes["l0.mix.o"] == (W, 3 * 14) and "l0.mix.g" not in shapes
    assert shapes["l1.mix.q"] == (4 * 22, W) and shapes["l1.mix.k"] == (2 * 22, W)
    assert shapes["l1.mix.v"] == (2 * 10, W) and shapes["l1.mix.g"] == (4 * 10, W)
    assert shapes["l1.mix.vmix"] == () and "l2.mix.vmix" not in shapes
    assert shapes["l0.mlp.router"] == (10, W) and shapes["l0.mlp.correction"] == (10,)
    assert shapes["l0.mlp.e9.gate"] == (26, W) and shapes["l0.mlp.e0.down"] == (W, 26)
    assert shapes["l1.mlp.gate"] == (90, W) and "l0.mlp.shared.up" not in shapes
    # one row a token for the latent, keys and values of their own sizes for the others
    need = model.line_needs[0]
    assert (need.kv_heads, need.head_dim, need.planes, need.window) == (1, 40, 1, 21)
    need = model.line_needs[1]
    assert (need.kv_heads, need.head_dim, need.v_dim, need.window) == (2, 22, 10, 0)
    assert model.line_needs[3].v_dim == 0 and not model.state_needs


def test_the_first_layer_that_blends_keeps_its_own_values():
    spec = TenusunConfig.from_dict(small_doc("A")).to_model_spec()
    mixes = [l.mixer.params.get("value_mix") for l in spec.layers]
    assert mixes == [None, "first", None, "blend", None, "blend"]
    needs = {t.name: t for t in DecoderModel(spec).tensors()}
    assert needs["l1.mix.vmix"].optional and not needs["l3.mix.vmix"].optional
    assert all(l.mixer.params.get("value_mix") is None
               for l in TenusunConfig.from_dict(small_doc("B")).to_model_spec().layers)


def test_absent_keys_and_a_layer_without_feed_forward():
    spec = TenusunConfig.from_dict(small_doc("B")).to_model_spec()
    assert spec.embedding.params["scale"] == 1.0
    assert spec.layers[0].mixer.params["position"] == ""
    assert spec.layers[1].mixer.params["window"] == 0
    assert spec.layers[1].feed_forward.kind == "none"
    assert spec.layers[1].block.params["feed_forward"] is False
    assert spec.layers[0].feed_forward.params["groups"] == 1
    needs = {t.name: t for t in DecoderModel(spec).tensors()}
    for n in ("l1.norm2", "l1.norm2.b", "l1.norm2b", "l1.norm2b.b"):
        assert needs[n].optional and not needs[n.replace("l1", "l0")].optional
    assert needs["head"].must_equal == "embed" and needs["head"].optional
    doc = small_doc("B")
    for key in ("kv_heads", "vdim"):
        del doc["layers"][2]["mixer"][key]
    p = TenusunConfig.from_dict(doc).to_model_spec().layers[2].mixer.params
    assert p["kv_heads"] == 3 and p["v_dim"] == 12
    # equal rotations are one encoding of the model
    a = TenusunConfig.from_dict(small_doc("A")).to_model_spec()
    assert len(a.positions) == 5
    assert a.layers[1].mixer.params["position"] == a.layers[5].mixer.params["position"]


@pytest.mark.parametrize("change,text", [
    (lambda d: d["layers"][0].update(type="other"), "not known"),
    (lambda d: d["layers"][1]["mixer"].update(kv_heads=3), "key/value heads"),
    (lambda d: d["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda d: d["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=12), "rotating"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=5), "rotating"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(base=0), "base"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].update(slow=0), "slow"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("factor"), "factor"),
    (lambda d: d["layers"][5]["mixer"].update(vdim=12), "blended"),
    (lambda d: d["layers"][1]["mlp"].pop("limit"), "limit"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=11), "top"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=5), "groups"),
    (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=3), "groups"),
    (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=6), "keep"),
    (lambda d: d["layers"][0]["mlp"].pop("expert"), "expert"),
    (lambda d: d["layers"][0].update(mlp={"kind": "routed", "ff": 8}), "feed-forward kind"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_refusals(change, text):
    doc = small_doc("A")
    change(doc)
    with pytest.raises(ConfigError) as e:
        TenusunConfig.from_dict(doc).to_model_spec()
    assert text in str(e.value)


def test_parts_refuse_what_does_not_go_together():
    names = {"q": "q", "k": "k", "v": "v", "o": "o", "g": "g"}
    base = {"hidden_size": 16, "heads": 2, "kv_heads": 1, "head_dim": 8, "scale": 1.0}
    bad = [dict(base, names=names, gate="value", head_norm="unit_after_rotation", head_norm_eps=1e-6),
           dict(base, names=names, gate="token"), dict(base, names=names, value_mix="last"),
           dict(base, names=names, gate="value", shared_kv=True)]
    for p in bad:
        with pytest.raises(ConfigError):
            MIXERS.build(PartSpec("gqa_attention", p))
    yarn = POSITIONS.build(PartSpec("rope_yarn", {"theta": 100.0, "rot_dim": 8, "factor": 2.0,
                                                  "original": 32, "fast": 4.0, "slow": 1.0}))
    with pytest.raises(ConfigError):        # the kernels that norm heads know no amplitude
        MIXERS.build(PartSpec("gqa_attention", dict(base, names=dict(names, q_norm="a", k_norm="b"),
                                                    position="r", head_norm_eps=1e-6)),
                     "", positions={"r": yarn})
    moe = {"hidden_size": 16, "experts": 12, "top": 3, "intermediate_size": 8, "shared_gate": False,
           "names": {"router": "r", "expert": "e{}.", "shared": "s.", "gate": "g", "up": "u", "down": "d"}}
    FEED_FORWARDS.build(PartSpec("routed_experts", dict(moe, weights="sigmoid", groups=4, keep_groups=1)))
    for more in ({"weights": "softmax_of_chosen", "groups": 3}, {"weights": "sigmoid", "groups": 5},
                 {"weights": "sigmoid", "groups": 6, "keep_groups": 1}):
        with pytest.raises(ConfigError):
            FEED_FORWARDS.build(PartSpec("routed_experts", dict(moe, **more)))
    norm = NORMS.build(PartSpec("layernorm", {"name": "n", "size": 8, "eps": 1e-6, "bias": True}))
    tanh = NORMS.build(PartSpec("dynamic_tanh", {"name": "n", "size": 8}))
    with pytest.raises(ConfigError):
        BLOCKS.build(PartSpec("sandwich_residual", {"feed_forward": False}), "", mixer=None,
                     feed_forward=None, norms={"mixer": norm, "mixer_out": tanh})


def _weights(doc, seed):
    model = DecoderModel(TenusunConfig.from_dict(doc).to_model_spec())
    w = sharpen(random_tensors(model.tensors(), seed, std=0.15, norm_std=0.2), 0.15)
    w.setdefault("l1.mix.vmix", np.float64(0.9))
    return {k: np.asarray(v if isinstance(v, float) else v.double().numpy()) if hasattr(v, "double")
            else np.asarray(v) for k, v in w.items()}


@pytest.mark.parametrize("name", ["A", "B"])
def test_the_plain_implementation_is_causal(name):
    """A prefix gives the logits that the whole sequence gives at its positions."""
    doc = small_doc(name)
    w = _weights(doc, 3)
    ids = np.random.default_rng(1).integers(0, doc["vocab"], 40).tolist()
    whole = plain.forward(doc, w, ids)
    assert np.allclose(plain.forward(doc, w, ids[:17]), whole[:17], rtol=1e-9, atol=1e-9)
    assert np.isfinite(whole).all()


def test_every_mechanism_of_the_plain_implementation_counts():
    """Taking one away changes the logits: the sharpened random weights let none of them hide."""
    doc = small_doc("A")
    w = _weights(doc, 4)
    ids = np.random.default_rng(2).integers(0, doc["vocab"], 60).tolist()
    base = plain.forward(doc, w, ids)

    def moved(change_doc=None, change_w=None):
        d, v = small_doc("A"), dict(w)
        if change_doc:
            change_doc(d)
        if change_w:
            change_w(v)
        return np.abs(plain.forward(d, v, ids) - base).max() / base.std()

    assert moved(lambda d: d["layers"][3]["mixer"].pop("v_mix")) > 0.05
    assert moved(None, lambda v: v.update({"l1.mix.vmix": np.float64(0.1)})) == 0.0   # unused
    assert moved(None, lambda v: v.update({"l3.mix.vmix": v["l3.mix.vmix"] * 0.5})) > 0.02
    assert moved(lambda d: d["layers"][0]["mixer"]["mask"].update(size=22)) > 0.02
    assert moved(lambda d: d["layers"][1]["mixer"]["rot"].pop("scaling")) > 0.02
    assert moved(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=5)) > 0.05
    assert moved(lambda d: d["layers"][1]["mlp"].update(limit=0.9)) > 0.01
    assert moved(None, lambda v: v.update({"l0.mlp.correction": v["l0.mlp.correction"] * 0})) > 0.05
    for n in ("l0.norm1.b", "l1.norm1b.b", "l3.norm2.b", "l4.norm2b.b", "final.norm.b"):
        assert moved(None, lambda v: v.update({n: v[n] * 0})) > 0.02, n


def test_plain_softmax_with_one_more_term():
    s = np.array([[1.0, -2.0, 9.0], [-700.0, -800.0, 5.0]])
    mask = np.array([[True, True, False], [True, True, False]])
    p = plain.softmax_rows(s, mask, True)
    assert np.allclose(p[0, :2], np.exp([1.0, -2.0]) / (1.0 + np.exp(1.0) + np.exp(-2.0)))
    assert p[0, 2] == 0.0 and np.abs(p[1]).max() < 1e-300     # far below the sink: nothing is left
    assert np.allclose(plain.softmax_rows(s, mask, False).sum(axis=1), 1.0)


def test_plain_choice_among_groups():
    # scores s = sigmoid(z) are all 1/2: the corrections decide, the weights do not see them
    corr = np.array([0.9, -3.0, -3.0, 0.4, 0.45, -3.0, 0.5, 0.0, 0.1])
    chosen, weights = plain.choose(np.zeros(9), corr, 2, 3, 1)
    assert chosen == [3, 4] or chosen == [4, 3]          # 0.4 + 0.45 beats 0.9 - 3 and 0.5 + 0.1
    assert weights == [0.5, 0.5]
    # negative choice scores: an expert of a kept group still beats one of a group that is not
    corr = np.array([-2.0, -2.1, -9.0, -1.0, -9.0, -9.0])
    chosen, _ = plain.choose(np.zeros(6), corr, 2, 2, 1)
    assert chosen == [0, 1]
    assert plain.choose(np.zeros(4), np.zeros(4), 2, 1, 1)[0] == [0, 1]       # ties: the lower
    z = np.array([2.0, -1.0, 0.0, 3.0])
    chosen, weights = plain.choose(z, np.zeros(4), 3, 1, 1)
    assert chosen == [3, 0, 2] and np.allclose(weights, 1 / (1 + np.exp(-z[[3, 0, 2]])))


def test_plain_clamped_form_and_blend():
    one = np.eye(1)
    h = np.array([[5.0], [-5.0], [0.5]])
    w = {"gate": one, "up": one, "down": one}
    out = plain.clamped_dense(h, w, "", 2.0)[:, 0]
    f = lambda g, u: g / (1 + math.exp(-1.702 * g)) * (u + 1)
    assert np.allclose(out, [f(2.0, 2.0), f(-5.0, -2.0), f(0.5, 0.5)])
    assert np.allclose(plain.blend(np.array([1.0]), np.array([5.0]), 0.25), [2.0])


def test_plain_turns_pairs_half_a_rotation_apart():
    x = np.zeros((2, 1, 5))
    x[:, 0, 0], x[:, 0, 4] = 1.0, 7.0
    out = plain.rotate_halves(x, [0, 2], {"dims": 4, "base": 100.0})
    assert np.allclose(out[0], x[0])
    assert np.allclose(out[1, 0], [math.cos(2.0), 0.0, math.sin(2.0), 0.0, 7.0])
