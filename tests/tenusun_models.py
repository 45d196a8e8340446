"""Small Tenusun configurations for the tests, their random model folders and the plain
implementation's view of them.

A: sizes that are no multiples of four; fewer rotating values than a head has; windows that
   decoding passes; three layers whose values are blended with a layer between them that is not;
   groups of experts of which one or two are kept; experts after latent attention too.
B: no embedding scale, no window, no blended values; a layer that rotates nothing; one head, as
   many key/value heads as heads; one expert a token without groups; a layer without feed-forward.
C: sizes that the tcgen05 prefills take (heads of 128, value rows of 64 and 128; latent attention
   with keys and values per head, and one that stays with the latents); windows longer than a page.
D: sizes that the warp-level kernels round up (heads of 40, 64 and 72, value rows of 24 and 136:
   the last one beyond them); twenty heads on one key/value head; a single latent layer last.
"""
import json
import os

import numpy as np


def _rot(dims, base, factor=0.0, original=64, fast=8.0, slow=1.0):
    rot = {"dims": dims, "base": base}
    if factor:
        rot["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return rot


def _att(heads, kv, dim, vdim, scale, rot=None, mix=False, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        m["rot"] = rot
    if mix:
        m["v_mix"] = True
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, size=0, base=100.0, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
         "kv_rank": kv_rank, "scale": scale, "rot": {"dims": rot_dim, "base": base}}
    if size:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff, groups=None):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def _a():
    return {"architecture": "Tenusun", "vocab": 150, "width": 70, "norm": {"eps": 1e-5},
            "embedding": {"scale": 3.5},
            "layers": [
                _lat(3, 18, 10, 14, 26, 30, 0.25, 21, 90.0, _moe(10, 3, 26, (5, 2))),
                _att(4, 2, 22, 10, 0.3, _rot(12, 500.0, 3.0), True, _dense(90, 0.8)),
                _att(3, 1, 14, 30, 0.35, _rot(14, 80.0), False, _moe(6, 2, 18, (2, 1))),
                _att(6, 2, 10, 10, 0.4, _rot(6, 300.0, 2.0, 30), True, _moe(9, 2, 22, (3, 2))),
                _lat(2, 10, 6, 22, 18, 42, 0.3, 33, 700.0, _dense(54, 1.5)),
                _att(2, 2, 18, 10, 0.3, _rot(12, 500.0, 3.0), True, _dense(34, 2.5))]}


def _b():
    return {"architecture": "Tenusun", "vocab": 97, "width": 36, "norm": {"eps": 1e-6},
            "layers": [
                _att(1, 1, 20, 24, 0.25, None, False, _moe(5, 1, 14)),
                _lat(1, 12, 4, 20, 10, 16, 0.35, 0, 50.0, None),
                _att(3, 3, 12, 12, 0.35, _rot(12, 100.0, 4.0, 40, 6.0, 0.5), False, _dense(44, 1.1))]}


def _c():
    return {"architecture": "Tenusun", "vocab": 320, "width": 128, "norm": {"eps": 1e-6},
            "embedding": {"scale": 11.0},
            "layers": [
                _att(4, 2, 128, 64, 0.06, _rot(96, 1e4, 8.0, 128), True, _moe(16, 4, 64, (4, 2))),
                _lat(4, 48, 32, 40, 72, 64, 0.12, 70, 1e4, _dense(192, 1.2)),
                _att(2, 1, 128, 128, 0.06, _rot(128, 1e5), False, _moe(8, 2, 96, (4, 3))),
                _att(6, 2, 128, 64, 0.07, _rot(32, 1e4, 2.0, 100), True, _dense(160, 0.9)),
                _lat(2, 64, 16, 128, 40, 128, 0.1, 129, 1e5, _moe(12, 3, 32, (6, 4)))]}


def _d():
    return {"architecture": "Tenusun", "vocab": 200, "width": 192, "norm": {"eps": 1e-6},
            "embedding": {"scale": 0.5},
            "layers": [
                _att(20, 1, 40, 24, 0.15, _rot(16, 300.0, 2.0, 50), True, _dense(224, 1.0)),
                _att(3, 1, 64, 24, 0.12, _rot(64, 1e4, 4.0, 256), True, _moe(32, 5, 64, (8, 3))),
                _att(4, 4, 72, 136, 0.12, _rot(48, 2e3), False, _dense(128, 3.0)),
                _lat(5, 24, 8, 16, 56, 48, 0.2, 45, 900.0, _moe(24, 6, 40, (3, 1)))]}


SMALL = {"A": _a, "B": _b, "C": _c, "D": _d}

# name -> (seed, std of matrices, prompt lengths of the whole-prompt tests, decode steps)
HOW = {"A": (61, 0.13, [1, 9, 64, 150], 9), "B": (62, 0.18, [2, 63, 65, 131], 7),
       "C": (63, 0.1, [5, 128, 200], 6), "D": (64, 0.09, [3, 130], 5)}


def small_doc(name):
    return SMALL[name]()


def sharpen(tensors, std):
    """Random weights in which a fault shows: corrections as large as the scores themselves (some
    choice scores are then negative), norms' biases that count, logits of the routers apart."""
    for n, t in tensors.items():
        if n.endswith(".correction"):
            t.mul_(0.6 / std)
        elif n.endswith(".router"):
            t.mul_(1.5)
        elif n.endswith(".b"):
            t.mul_(0.3 / std)
        elif n == "embed":
            t.mul_(0.5 / std)
    return tensors


class SmallModel:
    def __init__(self, name, folder):
        from mormot2_ai_b200 import DecoderModel, TenusunConfig, write_safetensors
        from mormot2_ai_b200.weights import random_tensors
        from tests.plain import tenusun_plain as plain
        from tests.plain.qwen3_plain import read_safetensors
        self.name, self.doc = name, small_doc(name)
        self.seed, std, self.prompt_lens, self.decode_steps = HOW[name]
        self.config = TenusunConfig.from_dict(self.doc)
        tensors = sharpen(random_tensors(DecoderModel(self.config.to_model_spec()).tensors(),
                                         self.seed, std=std, norm_std=0.2), std)
        self.folder = folder
        os.makedirs(folder, exist_ok=True)
        with open(os.path.join(folder, "config.json"), "w") as f:
            json.dump(self.doc, f)
        write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
        with open(os.path.join(folder, "config.json")) as f:
            self.plain_config = json.load(f)
        self.weights = {k: np.asarray(v, dtype=np.float64) for k, v in
                        read_safetensors(os.path.join(folder, "model.safetensors")).items()}
        self.plain = plain
        self.runs = len(self.doc["layers"])

    def tokens(self, n, seed=0):
        rng = np.random.default_rng(1000 * self.seed + seed)
        return rng.integers(0, self.doc["vocab"], n).tolist()

    def reference(self, ids, states=None, routing=None):
        return self.plain.forward(self.plain_config, self.weights, ids, states=states,
                                  routing=routing)

    def rounded(self, ids, dtype="bfloat16", forced=None, states=None):
        """The plain logits with everything that a 16-bit run keeps in 16 bits rounded so (None
        for float32): how far rounding alone moves them, with the experts that ``forced`` names."""
        if dtype != "bfloat16":
            return None
        return self.plain.forward(self.plain_config, self.weights, ids, rnd=self.plain.bfloat16,
                                  states=states,
                                  routing=self.plain.Routing(forced, strict=False))
