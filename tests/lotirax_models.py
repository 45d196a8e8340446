"""Small Lotirax configurations for the tests, their random model folders and the plain
implementation's view of them.

A: a loop of two passes over the first two layers; sizes that are no multiples of four; fewer
   rotating values than a map has; key/value groups; a window that decoding passes; two and
   three experts a token, with and without a shared one.
B: no loop, no residual factor, no window in the first layer, no frequency scaling; one head;
   as many key/value heads as heads; one expert a token; a layer without feed-forward.
C: sizes that the tcgen05 kernel takes (maps of 64, value rows of 128 and 64); a loop of three
   passes over the last two layers; windows longer than a page.
D: maps of 128 and value rows of 256; ten heads on one key/value head; a map without rotation;
   sizes that are rounded up inside the tensor-core kernels; a single pass "loop".
"""
import json
import os

import numpy as np


def _rot(dims, base, factor=0.0, original=64, fast=8.0, slow=1.0):
    rot = {"dims": dims, "base": base}
    if factor:
        rot["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return rot


def _att(heads, kv, dim, vdim, scale, diff, size=0, rot=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if size:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = rot
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=0):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared}
    return mlp


def _a():
    return {"architecture": "Lotirax", "vocab": 150, "width": 72, "norm": {"eps": 1e-5},
            "residual_mult": 0.55, "loop": {"start": 0, "stop": 2, "times": 2},
            "layers": [
                _att(4, 2, 18, 10, 0.4, 0.3, 21, _rot(12, 500.0, 3.0), _moe(5, 2, 26, 34)),
                _att(6, 3, 10, 14, 0.5, 0.8, 33, _rot(10, 90.0, 2.0, 30), _dense(90)),
                _att(2, 1, 22, 30, 0.3, 0.5, 21, _rot(12, 500.0, 3.0), _moe(7, 3, 18))]}


def _b():
    return {"architecture": "Lotirax", "vocab": 97, "width": 40, "norm": {"eps": 1e-6},
            "layers": [
                _att(1, 1, 20, 24, 0.35, 0.2, 0, _rot(20, 100.0), _moe(3, 1, 14, 10)),
                _att(2, 2, 12, 12, 0.5, 0.7, 9, _rot(8, 50.0)),
                _att(3, 1, 14, 16, 0.4, 0.45, 17, _rot(14, 700.0, 4.0, 40, 6.0, 0.5), _dense(44))]}


def _c():
    return {"architecture": "Lotirax", "vocab": 320, "width": 128, "norm": {"eps": 1e-6},
            "residual_mult": 0.8, "loop": {"start": 1, "stop": 3, "times": 3},
            "layers": [
                _att(4, 2, 64, 128, 0.2, 0.4, 70, _rot(64, 1e4, 8.0, 128), _dense(192)),
                _att(3, 1, 64, 64, 0.2, 0.6, 129, _rot(32, 1e4, 2.0, 100), _moe(6, 2, 96, 64)),
                _att(2, 2, 64, 128, 0.15, 0.55, 64, _rot(64, 1e5, 4.0, 200), _moe(9, 1, 64, 160))]}


def _d():
    return {"architecture": "Lotirax", "vocab": 200, "width": 192, "norm": {"eps": 1e-6},
            "residual_mult": 0.6, "loop": {"start": 0, "stop": 3, "times": 1},
            "layers": [
                _att(3, 1, 128, 256, 0.12, 0.5, 100, _rot(128, 1e5, 4.0, 256), _dense(224)),
                _att(10, 1, 24, 40, 0.3, 0.35, 66, _rot(16, 300.0, 2.0, 50), _moe(8, 4, 64, 96)),
                _att(4, 4, 72, 136, 0.15, 0.65, 45, None, _dense(128))]}


SMALL = {"A": _a, "B": _b, "C": _c, "D": _d}

# name -> (seed, std of matrices, prompt lengths of the whole-prompt tests, decode steps)
HOW = {"A": (51, 0.12, [1, 9, 64, 150], 9), "B": (52, 0.16, [2, 63, 65, 131], 7),
       "C": (53, 0.09, [5, 128, 200], 6), "D": (54, 0.07, [3, 130], 5)}


def small_doc(name):
    return SMALL[name]()


class SmallModel:
    def __init__(self, name, folder):
        from mormot2_ai_b200 import DecoderModel, LotiraxConfig, write_safetensors
        from mormot2_ai_b200.weights import random_tensors
        from tests.plain import lotirax_plain as plain
        from tests.plain.qwen3_plain import read_safetensors
        self.name, self.doc = name, small_doc(name)
        self.seed, std, self.prompt_lens, self.decode_steps = HOW[name]
        self.config = LotiraxConfig.from_dict(self.doc)
        tensors = random_tensors(DecoderModel(self.config.to_model_spec()).tensors(), self.seed,
                                 std=std, norm_std=0.2)
        for n, t in tensors.items():
            # the vectors of the maps' weight so large that it is far from the constant alone,
            # and projections' biases that the norms see
            if n.rsplit(".", 1)[-1] in ("lq1", "lk1", "lq2", "lk2"):
                t.mul_(0.5 / (std * t.numel() ** 0.25))
            elif n.endswith(".b"):
                t.mul_(4.0)
            elif n == "embed":
                t.mul_(0.5 / std)
        self.folder = folder
        os.makedirs(folder, exist_ok=True)
        with open(os.path.join(folder, "config.json"), "w") as f:
            json.dump(self.doc, f)
        write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
        with open(os.path.join(folder, "config.json")) as f:
            self.plain_config = json.load(f)
        self.plain_config.setdefault("residual_mult", 1.0)
        self.weights = {k: v if v.dtype == np.int32 else np.asarray(v, dtype=np.float64)
                        for k, v in read_safetensors(os.path.join(folder, "model.safetensors")).items()}
        self.plain = plain
        self.runs = len(plain.layer_runs(self.plain_config))

    def tokens(self, n, seed=0):
        rng = np.random.default_rng(1000 * self.seed + seed)
        return rng.integers(0, self.doc["vocab"], n).tolist()

    def reference(self, ids, states=None):
        return self.plain.forward(self.plain_config, self.weights, ids, states=states)

    def rounded(self, ids, dtype="bfloat16"):
        """The plain logits with everything that a 16-bit run keeps in 16 bits rounded so (None
        for float32): how far rounding alone moves them."""
        if dtype != "bfloat16":
            return None
        return self.plain.forward(self.plain_config, self.weights, ids, rnd=self.plain.bfloat16)
