"""The typed configuration of the Tenusun decoder, read from its own config.json keys.

config.json: ``architecture`` = "Tenusun", ``vocab``, ``width``, ``norm.eps``,
``embedding.scale`` (absent: 1) and ``layers``, a list whose entries have ``type``
("latent_attention" or "attention"), the mixer's sizes in ``mixer`` and the feed-forward in
``mlp`` (``kind`` "dense" with ``ff`` and ``limit``; ``kind`` "moe" with ``expert.ff`` and
``router``: ``experts``, ``top`` and optionally ``groups`` with ``count`` and ``keep``; or null).
Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b`` and
``final.norm`` (each with its bias ``.b``), ``l<i>.mix.*``, ``l<i>.mlp.*``. The head is the
embedding's table without its scale.

All norms of the residual are layer norms with a bias, one before and one after every sublayer:
x += norm1b(mixer(norm1(x))), x += norm2b(ff(norm2(x))).

Mixer ``latent_attention``: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``q_rank``, ``kv_rank``,
``scale``, ``rot``, a window ``mask.size``. Mixer ``attention``: ``heads``, ``kv_heads``, ``dim``,
``vdim``, ``scale``, ``rot`` (``base``, ``dims``, ``scaling`` with ``factor``, ``original``,
``fast`` and ``slow``), ``v_mix``: its values are blended with those of the first layer that has
it, a constant sink of score 0 and a gate for every value of the heads.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from ..errors import ConfigError
from .busavik import MAX_POSITIONS, _dict, _int, _num
from .spec import LayerSpec, ModelSpec, PartSpec, Run

LATENT_SIZES = ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")


@dataclass(frozen=True)
class TenusunConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[Dict[str, Any], ...]            # as in config.json, checked
    extra: Dict[str, Any] = field(default_factory=dict, compare=False)

    ARCHITECTURE = "Tenusun"
    MODEL_TYPE = "tenusun"

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
    def from_dict(cls, doc: Dict[str, Any], source: str = "config") -> "TenusunConfig":
        if not isinstance(doc, dict):
            raise ConfigError(f"{source} is no JSON object")
        if doc.get("architecture") != cls.ARCHITECTURE:
            raise ConfigError(f"{source}: architecture \"{doc.get('architecture')}\" is not "
                              f"{cls.ARCHITECTURE}")
        layers = doc.get("layers")
        if not isinstance(layers, list) or not 0 < len(layers) <= 1024:
            raise ConfigError(f"{source}: \"layers\" is missing, empty or too long")
        blended = None      # the value sizes of the layers whose values are blended
        for i, layer in enumerate(layers):
            where = f"{source}: layer {i}"
            cls._check_layer(layer, where)
            m = layer["mixer"]
            if layer["type"] == "attention" and m.get("v_mix"):
                sizes = (int(m.get("kv_heads") or m["heads"]), int(m.get("vdim") or m["dim"]))
                if blended not in (None, sizes):
                    raise ConfigError(f"{where}: values of {sizes[0]} x {sizes[1]} are blended "
                                      f"with those of {blended[0]} x {blended[1]}")
                blended = sizes
        scale = 1.0
        if doc.get("embedding") is not None:
            emb = _dict(doc, "embedding", source)
            if emb.get("scale") is not None:
                scale = _num(emb, "scale", source + " embedding")
        return cls(vocab=_int(doc, "vocab", source, hi=1 << 22),
                   width=_int(doc, "width", source, hi=1 << 16),
                   norm_eps=_num(_dict(doc, "norm", source), "eps", source + " norm"),
                   embedding_scale=scale, layers=tuple(layers))

    @staticmethod
    def _check_rotation(m: Dict[str, Any], most: int, source: str) -> None:
        if m.get("rot") is None:
            return
        rot, rs = _dict(m, "rot", source), source + " rot"
        dims = _int(rot, "dims", rs, lo=0, hi=1 << 12)
        if dims % 2 or dims > most:
            raise ConfigError(f"{source}: {dims} rotating values of {most}")
        if dims and _num(rot, "base", rs) <= 0:
            raise ConfigError(f"{source}: a rotary base of {rot['base']}")
        if rot.get("scaling") is not None:
            sc = _dict(rot, "scaling", rs)
            for key in ("factor", "original", "fast", "slow"):
                if _num(sc, key, rs + " scaling") <= 0:
                    raise ConfigError(f"{rs} scaling: {key} = {sc[key]}")

    @classmethod
    def _check_layer(cls, layer: Any, source: str) -> None:
        if not isinstance(layer, dict):
            raise ConfigError(f"{source} is no object")
        m, ms = _dict(layer, "mixer", source), source + " mixer"
        _num(m, "scale", ms)
        if layer.get("type") == "latent_attention":
            for key in LATENT_SIZES:
                _int(m, key, ms, lo=0 if key == "rot_dim" else 1, hi=1 << 14)
            cls._check_rotation(m, int(m["rot_dim"]), ms)
        elif layer.get("type") == "attention":
            heads = _int(m, "heads", ms, hi=1 << 12)
            kv = _int(m, "kv_heads", ms, hi=1 << 12) if m.get("kv_heads") is not None else heads
            if heads % kv:
                raise ConfigError(f"{ms}: {heads} heads on {kv} key/value heads")
            dim = _int(m, "dim", ms, hi=1 << 12)
            if m.get("vdim") is not None:
                _int(m, "vdim", ms, hi=1 << 12)
            cls._check_rotation(m, dim, ms)
        else:
            raise ConfigError(f"{source}: mixer type \"{layer.get('type')}\" is not known "
                              "(known: attention, latent_attention)")
        if m.get("mask") is not None:
            mask = _dict(m, "mask", ms)
            if mask.get("size") is not None:
                _int(mask, "size", ms + " mask", hi=1 << 24)
        mlp = layer.get("mlp")
        if mlp is None:
            return
        kind = mlp.get("kind", "dense") if isinstance(mlp, dict) else mlp
        if kind == "dense":
            _int(mlp, "ff", source + " mlp", hi=1 << 22)
            _num(mlp, "limit", source + " mlp")
        elif kind == "moe":
            _int(_dict(mlp, "expert", source + " mlp"), "ff", source + " mlp expert", hi=1 << 22)
            router, rs = _dict(mlp, "router", source + " mlp"), source + " mlp router"
            experts = _int(router, "experts", rs, hi=256)
            top = _int(router, "top", rs, hi=min(experts, 32))
            if router.get("groups") is not None:
                groups = _dict(router, "groups", rs)
                count = _int(groups, "count", rs + " groups", hi=min(experts, 32))
                keep = _int(groups, "keep", rs + " groups", hi=count)
                if experts % count:
                    raise ConfigError(f"{rs}: {experts} experts in {count} groups")
                if top > keep * (experts // count):
                    raise ConfigError(f"{rs}: {top} experts from {keep} groups of "
                                      f"{experts // count}")
        else:
            raise ConfigError(f"{source}: feed-forward kind \"{kind}\" is not known "
                              "(known: dense, moe)")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
                "layers": list(self.layers)}

    # ------------------------------------------------------------------ the model as data
    @staticmethod
    def _position(rot: Optional[Dict[str, Any]], positions: Dict[str, PartSpec]) -> str:
        """The name of the position encoding that ``rot`` describes (added if it is new)."""
        if not rot or not int(rot.get("dims") or 0):
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

    def _mixer(self, layer: Dict[str, Any], positions: Dict[str, PartSpec],
               first: bool) -> PartSpec:
        """``first``: this is the first layer whose values others are blended with."""
        m = layer["mixer"]
        common = {"hidden_size": self.width, "heads": int(m["heads"]), "scale": float(m["scale"]),
                  "window": int((m.get("mask") or {}).get("size") or 0),
                  "position": self._position(m.get("rot"), positions)}
        if layer["type"] == "latent_attention":
            return PartSpec("latent_attention", {
                **common, **{k: int(m[k]) for k in LATENT_SIZES}, "latent_norm_eps": self.norm_eps,
                "names": {"dq": "mix.dq", "dq_norm": "mix.dq.norm", "uq": "mix.uq",
                          "dkv": "mix.dkv", "dkv_norm": "mix.dkv.norm", "uk": "mix.uk",
                          "uv": "mix.uv", "o": "mix.o"}})
        names = {k: "mix." + k for k in ("q", "k", "v", "g", "o")}
        if m.get("v_mix"):
            names["vmix"] = "mix.vmix"
        return PartSpec("gqa_attention", {
            **common, "kv_heads": int(m.get("kv_heads") or m["heads"]), "head_dim": int(m["dim"]),
            "v_dim": int(m.get("vdim") or m["dim"]), "sink_value": 0.0, "gate": "value",
            "value_mix": ("first" if first else "blend") if m.get("v_mix") else None,
            "names": names})

    def _feed_forward(self, mlp: Optional[Dict[str, Any]]) -> PartSpec:
        if mlp is None:
            return PartSpec("none")
        if mlp.get("kind", "dense") == "dense":
            return PartSpec("gated_mlp", {
                "hidden_size": self.width, "intermediate_size": int(mlp["ff"]),
                "activation": "clamped_swish", "limit": float(mlp["limit"]),
                "names": {"gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"}})
        router = mlp["router"]
        groups = router.get("groups") or {"count": 1, "keep": 1}
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "experts": int(router["experts"]),
            "top": int(router["top"]), "intermediate_size": int(mlp["expert"]["ff"]),
            "activation": "silu", "weights": "sigmoid", "groups": int(groups["count"]),
            "keep_groups": int(groups["keep"]), "shared_gate": False,
            "names": {"router": "mlp.router", "correction": "mlp.correction",
                      "expert": "mlp.e{}.", "shared": "mlp.shared.", "gate": "gate", "up": "up",
                      "down": "down"}})

    def to_model_spec(self) -> ModelSpec:
        c = self
        positions: Dict[str, PartSpec] = {}

        def norm(name, optional=False):
            return PartSpec("layernorm", {"name": name, "size": c.width, "eps": c.norm_eps,
                                          "bias": True, "optional": optional})

        layers: List[LayerSpec] = []
        first = True
        for i, layer in enumerate(c.layers):
            mlp = layer.get("mlp")
            # a layer without a feed-forward may still store its norms: tolerated, unused
            norms = {"mixer": norm("norm1"), "mixer_out": norm("norm1b"),
                     "feed_forward": norm("norm2", mlp is None),
                     "feed_forward_out": norm("norm2b", mlp is None)}
            layers.append(LayerSpec(
                block=PartSpec("sandwich_residual", {"feed_forward": mlp is not None}),
                mixer=c._mixer(layer, positions, first), feed_forward=c._feed_forward(mlp),
                norms=norms, prefix=f"l{i}."))
            if layer["type"] == "attention" and layer["mixer"].get("v_mix"):
                first = False
        schedule = tuple(Run(layer=i, cache_line=i, writes_cache=True) for i in range(len(layers)))
        return ModelSpec(
            architecture=c.ARCHITECTURE, vocab_size=c.vocab, hidden_size=c.width,
            max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"name": "embed", "vocab_size": c.vocab,
                                                   "hidden_size": c.width,
                                                   "scale": c.embedding_scale}),
            positions=positions, layers=tuple(layers), schedule=schedule,
            final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"name": "head", "tied": True, "tied_to": "embed",
                                      "vocab_size": c.vocab, "hidden_size": c.width}))
