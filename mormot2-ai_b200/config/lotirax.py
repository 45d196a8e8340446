"""The typed configuration of the Lotirax decoder, read from its own config.json keys.

config.json: ``architecture`` = "Lotirax", ``vocab``, ``width``, ``norm.eps``,
``residual_mult`` (absent: 1), ``loop`` with ``start``, ``stop`` and ``times`` (absent: every
layer runs once) and ``layers``, a list whose entries have ``type`` ("attention"), the mixer's
sizes in ``mixer`` and the feed-forward in ``mlp`` (``kind`` "dense" with ``ff``; ``kind``
"moe" with ``expert.ff``, ``router.experts``, ``router.top`` and ``shared.ff``; or null).
Tensor names: ``embed``, ``loop.in``, ``loop.step``, ``l<i>.norm1``, ``l<i>.ls1``,
``l<i>.ls2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``. The head is the embedding.

A layer has one norm (RMS, its weight stored around zero) that both sublayers read:
x += residual_mult * (ls1 * mixer(h) + ls2 * ff(h)). The layers ``start`` .. ``stop`` - 1 run
``times`` times in a row with the same weights, every pass with cache lines of its own; a pass
starts with x = W_in [x ; x0] + step[t], x0 the embedding's output.

The mixer is differential attention: ``heads`` query heads and ``kv_heads`` key heads of two
maps of ``dim`` values each, ``kv_heads`` value heads of ``vdim``; ``scale``, the constant
``diff``, a window ``mask.size``, a rotation ``rot`` (``base``, ``dims``, ``scaling`` with
``factor``, ``original``, ``fast`` and ``slow``).

The feed-forward of experts names a token's experts in a table over the vocabulary; an expert
is W_down relu(W_up h)^2.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from ..errors import ConfigError
from .busavik import MAX_POSITIONS, _dict, _int, _num
from .spec import LayerSpec, ModelSpec, PartSpec, Run


@dataclass(frozen=True)
class LotiraxConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    loop: Optional[Tuple[int, int, int]]          # (start, stop, times) or None
    layers: Tuple[Dict[str, Any], ...]            # as in config.json, checked
    extra: Dict[str, Any] = field(default_factory=dict, compare=False)

    ARCHITECTURE = "Lotirax"
    MODEL_TYPE = "lotirax"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def max_position_embeddings(self) -> int:
        return MAX_POSITIONS

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, doc: Dict[str, Any], source: str = "config") -> "LotiraxConfig":
        if not isinstance(doc, dict):
            raise ConfigError(f"{source} is no JSON object")
        if doc.get("architecture") != cls.ARCHITECTURE:
            raise ConfigError(f"{source}: architecture \"{doc.get('architecture')}\" is not "
                              f"{cls.ARCHITECTURE}")
        layers = doc.get("layers")
        if not isinstance(layers, list) or not 0 < len(layers) <= 1024:
            raise ConfigError(f"{source}: \"layers\" is missing, empty or too long")
        for i, layer in enumerate(layers):
            cls._check_layer(layer, f"{source}: layer {i}")
        norm = _dict(doc, "norm", source)
        loop = None
        if doc.get("loop") is not None:
            lp = _dict(doc, "loop", source)
            start = _int(lp, "start", source + " loop", lo=0, hi=len(layers) - 1)
            stop = _int(lp, "stop", source + " loop", lo=start + 1, hi=len(layers))
            loop = (start, stop, _int(lp, "times", source + " loop", hi=1024))
        return cls(vocab=_int(doc, "vocab", source, hi=1 << 22),
                   width=_int(doc, "width", source, hi=1 << 16),
                   norm_eps=_num(norm, "eps", source + " norm"),
                   residual_mult=(_num(doc, "residual_mult", source)
                                  if doc.get("residual_mult") is not None else 1.0),
                   loop=loop, layers=tuple(layers))

    @classmethod
    def _check_layer(cls, layer: Any, source: str) -> None:
        if not isinstance(layer, dict):
            raise ConfigError(f"{source} is no object")
        if layer.get("type") != "attention":
            raise ConfigError(f"{source}: mixer type \"{layer.get('type')}\" is not known "
                              "(known: attention)")
        m, ms = _dict(layer, "mixer", source), source + " mixer"
        heads = _int(m, "heads", ms, hi=1 << 12)
        kv = _int(m, "kv_heads", ms, hi=1 << 12) if m.get("kv_heads") is not None else heads
        if heads % kv:
            raise ConfigError(f"{ms}: {heads} heads on {kv} key/value heads")
        dim = _int(m, "dim", ms, hi=1 << 12)
        if m.get("vdim") is not None:
            _int(m, "vdim", ms, hi=1 << 12)
        _num(m, "scale", ms)
        _num(m, "diff", ms)
        if m.get("mask") is not None:
            mask = _dict(m, "mask", ms)
            if mask.get("size") is not None:
                _int(mask, "size", ms + " mask", hi=1 << 24)
        if m.get("rot") is not None:
            rot, rs = _dict(m, "rot", ms), ms + " rot"
            dims = _int(rot, "dims", rs, lo=0, hi=1 << 12)
            if dims % 2 or dims > dim:
                raise ConfigError(f"{source}: {dims} rotating values of {dim}")
            if dims and _num(rot, "base", rs) <= 0:
                raise ConfigError(f"{source}: a rotary base of {rot['base']}")
            if rot.get("scaling") is not None:
                sc = _dict(rot, "scaling", rs)
                for key in ("factor", "original", "fast", "slow"):
                    if _num(sc, key, rs + " scaling") <= 0:
                        raise ConfigError(f"{rs} scaling: {key} = {sc[key]}")
        mlp = layer.get("mlp")
        if mlp is None:
            return
        kind = mlp.get("kind", "dense") if isinstance(mlp, dict) else mlp
        if kind == "dense":
            _int(mlp, "ff", source + " mlp", hi=1 << 22)
        elif kind == "moe":
            _int(_dict(mlp, "expert", source + " mlp"), "ff", source + " mlp expert", hi=1 << 22)
            router = _dict(mlp, "router", source + " mlp")
            experts = _int(router, "experts", source + " mlp router", hi=4096)
            _int(router, "top", source + " mlp router", hi=min(experts, 32))
            if mlp.get("shared") is not None:
                _int(_dict(mlp, "shared", source + " mlp"), "ff", source + " mlp shared",
                     hi=1 << 22)
        else:
            raise ConfigError(f"{source}: feed-forward kind \"{kind}\" is not known "
                              "(known: dense, moe)")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> Dict[str, Any]:
        doc: Dict[str, Any] = {"architecture": self.ARCHITECTURE, "vocab": self.vocab,
                               "width": self.width, "norm": {"eps": self.norm_eps},
                               "residual_mult": self.residual_mult, "layers": list(self.layers)}
        if self.loop is not None:
            doc["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return doc

    # ------------------------------------------------------------------ the model as data
    def order(self) -> List[Tuple[int, int]]:
        """The order of layer runs as (layer, pass): ``pass`` is the number of the pass
        through the looped layers that this run opens, -1 for every other run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, -1) for i in range(n)]
        a, b, times = self.loop
        runs = [(i, -1) for i in range(a)]
        for t in range(times):
            runs += [(i, t if i == a else -1) for i in range(a, b)]
        return runs + [(i, -1) for i in range(b, n)]

    @staticmethod
    def _position(rot: Dict[str, Any], positions: Dict[str, PartSpec]) -> str:
        """The name of the position encoding that ``rot`` describes (added if it is new)."""
        if not int(rot.get("dims") or 0):
            return ""
        params = {"theta": float(rot["base"]), "rot_dim": int(rot["dims"])}
        scaling = rot.get("scaling")
        if scaling:
            params.update({k: float(scaling[k]) for k in ("factor", "original", "fast", "slow")})
            spec = PartSpec("rope_yarn", params)
        else:
            spec = PartSpec("rope_half", {**params, "rounding": "once"})
        name = next((n for n, have in positions.items() if have == spec), "")
        if not name:
            name = f"rot{len(positions)}"
            positions[name] = spec
        return name

    def _mixer(self, m: Dict[str, Any], positions: Dict[str, PartSpec]) -> PartSpec:
        heads = int(m["heads"])
        names = {k: "mix." + v for k, v in {
            "q": "q", "k": "k", "v": "v", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b",
            "q_norm": "q.norm", "k_norm": "k.norm", "lq1": "lq1", "lk1": "lk1", "lq2": "lq2",
            "lk2": "lk2", "o": "o"}.items()}
        return PartSpec("differential_attention", {
            "hidden_size": self.width, "heads": heads,
            "kv_heads": int(m.get("kv_heads") or heads), "dim": int(m["dim"]),
            "vdim": int(m.get("vdim") or m["dim"]), "scale": float(m["scale"]),
            "diff": float(m["diff"]), "eps": self.norm_eps,
            "window": int((m.get("mask") or {}).get("size") or 0),
            "position": self._position(m.get("rot") or {}, positions), "names": names})

    def _feed_forward(self, mlp: Optional[Dict[str, Any]]) -> PartSpec:
        if mlp is None:
            return PartSpec("none")
        if mlp.get("kind", "dense") == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width,
                                       "intermediate_size": int(mlp["ff"]),
                                       "names": {"gate": "mlp.gate", "up": "mlp.up",
                                                 "down": "mlp.down"}})
        shared = mlp.get("shared") or {}
        return PartSpec("table_experts", {
            "hidden_size": self.width, "vocab_size": self.vocab,
            "experts": int(mlp["router"]["experts"]), "top": int(mlp["router"]["top"]),
            "intermediate_size": int(mlp["expert"]["ff"]),
            "shared_size": int(shared.get("ff") or 0), "activation": "relu_squared",
            "names": {"table": "mlp.table", "expert": "mlp.e{}.", "shared": "mlp.shared.",
                      "up": "up", "down": "down"}})

    def to_model_spec(self) -> ModelSpec:
        c = self
        positions: Dict[str, PartSpec] = {}
        norm = lambda name: PartSpec("rmsnorm", {"name": name, "size": c.width,
                                                 "eps": c.norm_eps, "one_plus": True})
        layers: List[LayerSpec] = []
        for i, layer in enumerate(c.layers):
            mlp = layer.get("mlp")
            scales = {"mixer": "ls1"}
            if mlp is not None:
                scales["feed_forward"] = "ls2"
            layers.append(LayerSpec(
                block=PartSpec("parallel_residual", {"hidden_size": c.width,
                                                     "factor": c.residual_mult,
                                                     "scales": scales,
                                                     # a layer without a feed-forward may still
                                                     # store its scale: tolerated, unused
                                                     "spare": [] if mlp is not None else ["ls2"]}),
                mixer=c._mixer(layer["mixer"], positions), feed_forward=c._feed_forward(mlp),
                norms={"input": norm("norm1")}, prefix=f"l{i}."))
        schedule = []
        for n, (l, t) in enumerate(c.order()):
            before = None
            if t >= 0:
                before = PartSpec("pass_projection", {
                    "names": {"in": "loop.in", "step": "loop.step"}, "rows": c.loop[2], "row": t,
                    "size": c.width})
            schedule.append(Run(layer=l, cache_line=n, writes_cache=True, before=before))
        return ModelSpec(
            architecture=c.ARCHITECTURE, vocab_size=c.vocab, hidden_size=c.width,
            max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"name": "embed", "vocab_size": c.vocab,
                                                   "hidden_size": c.width}),
            positions=positions, layers=tuple(layers), schedule=tuple(schedule),
            final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"name": "head", "tied": True, "tied_to": "embed",
                                      "vocab_size": c.vocab, "hidden_size": c.width}),
            tolerated=() if c.loop is not None else (("loop.in", (c.width, 2 * c.width)),
                                                     ("loop.step", (-1, c.width))))
