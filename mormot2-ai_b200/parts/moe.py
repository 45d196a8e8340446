"""A feed-forward of routed experts, entirely on the device (``csrc/moe.cu``).

    z = W_router h (float32)          the ``top`` largest logits choose a token's experts
    w = softmax over the chosen logits only
    x += sum_k w_k · expert_k(h) + sigmoid(w_sg · h) · shared(h)
    expert(h) = W_d (act(W_g h) * (W_u h)), no biases; the shared expert (optional) has the
    same form with a size of its own and runs for every token.

The router and the shared expert's gate are one product with float32 results. The (token, k)
assignments are listed expert by expert by a kernel, the experts' two products run over
those lists in tiles (rows gathered for the first, results scattered back to the
assignment's own row by the second), and one kernel adds everything into the residual in a
fixed order. Nothing is read back to the host, so a decode pass stays a CUDA graph.

Options that a design may name. ``weights = "softmax_of_all"``: s = softmax(z) over every
router output; the choice goes by s + ``correction`` (a stored vector), the weights are the
chosen s times ``route_scale``, not renormalized. ``weights = "sigmoid"``: the same with
s = sigmoid(z). ``groups`` with ``keep_groups`` (with either): the experts are that many equal
groups of neighbours, a group's score is the sum of its two largest s + ``correction``, and only
experts of the best ``keep_groups`` groups can be chosen. ``identity`` = n: the last n router outputs
are identity experts without tensors, whose output is the input h times the weight.
``activation = "clamped_swish"`` with ``limit``: g = min(W_g h, limit),
u = clamp(W_u h, −limit, limit), g · sigmoid(1.702 g) · (u + 1) (the shared expert has a
``shared_limit`` of its own). ``shared_gate = False``: the shared expert is added as it is.

``table_experts``: experts without a router. A table [vocab, top] names every token id's
experts, each with the weight 1 / top; an expert is W_d act(W_u h) without a gate, and so is the
shared one, which runs for every token. The lists of a step depend on its token ids only: they
are made once in a pass of the model, however often its layer runs.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .. import kernels as K
from ..errors import ConfigError, WeightsError
from .base import FEED_FORWARDS, Part, TensorNeed
from .linear import Linear, Pending


def _sums(result):
    """A product's float32 result [T, N], or its pending split sums as [parts, T, N]."""
    return result.partial if isinstance(result, Pending) else result


def tile_rows(rt, w_up, T: int, A: int, E: int, hidden: int, inter: int) -> int:
    """Rows per tile of an expert's list: 128 where the tcgen05 kernel runs (bfloat16; 8 for a
    decode step of at most 8 tokens, the form that reads weights into registers), else 64, or
    16 while an expert has few rows, so that few multiply-adds are wasted."""
    fast = rt.fast_kernels and w_up.dtype == torch.bfloat16 and hidden % 8 == 0 and inter % 8 == 0
    if fast and T <= 8 and hidden % 32 == 0 and inter % 32 == 0:
        return 8        # a decode step: no expert has more rows, its weights stream once
    return 128 if fast else (64 if A > 16 * E else 16)


def expert_products(rt, h, w_up, w_down, plan, bm: int, max_tiles: int, top: int, act: int,
                    gated: bool = True, limit: float = 0.0, weight=None):
    """Both products of the chosen experts over a step's lists: y [T * top, hidden] float32, the
    row of assignment t * top + k times ``weight`` (None: one)."""
    A, dev = h.shape[0] * top, h.device
    inter = w_down.shape[2]
    mid = torch.empty((A, inter), dtype=rt.dtype, device=dev)
    y = torch.empty((A, w_down.shape[1]), dtype=torch.float32, device=dev)
    if bm == 128:       # the tcgen05 kernel, whose tiles are rows that lie one after the other
        rows = torch.empty((A, h.shape[1]), dtype=h.dtype, device=dev)
        K.moe_gather(h, plan, A, w_up.shape[0], top, rows)
        K.moe_gemm_tc(rows, w_up, mid, plan, max_tiles, True, rt.sms, rt.error_word, act,
                      gated=gated, limit=limit)
        K.moe_gemm_tc(mid, w_down, y, plan, max_tiles, False, rt.sms, rt.error_word,
                      weight=weight)
    else:
        K.moe_gemm(h, w_up, mid, plan, A, max_tiles, bm, top, True, act, limit=limit, gated=gated)
        K.moe_gemm(mid, w_down, y, plan, A, max_tiles, bm, top, False, act, weight)
    return y


class RoutedExperts(Part):
    capturable = True

    def __init__(self, spec, prefix: str = ""):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.experts, self.top = int(p["experts"]), int(p["top"])
        self.inter = int(p["intermediate_size"])
        self.shared_size = int(p.get("shared_size", 0))
        if not 0 < self.top <= min(self.experts + int(p.get("identity", 0)), 32):
            raise ConfigError(f"{self.top} of {self.experts} experts per token")
        modes = {"softmax_of_chosen": K.ROUTE_SOFTMAX_OF_CHOSEN,
                 "softmax_of_all": K.ROUTE_SOFTMAX_OF_ALL, "sigmoid": K.ROUTE_SIGMOID}
        if p.get("weights", "softmax_of_chosen") not in modes:
            raise ConfigError(f"expert weights \"{p['weights']}\" are not known "
                              f"(known: {', '.join(sorted(modes))})")
        self.mode = modes[p.get("weights", "softmax_of_chosen")]
        self.identity = int(p.get("identity", 0))
        self.routed = self.experts + self.identity      # what the router chooses among
        self.route_scale = float(p.get("route_scale", 1.0))
        self.limit = float(p.get("limit", 0.0))
        self.shared_limit = float(p.get("shared_limit", self.limit))
        self.shared_gate = bool(p.get("shared_gate", True))
        scored = self.mode != K.ROUTE_SOFTMAX_OF_CHOSEN
        if scored and (self.routed > 256 or self.shared_gate and int(p.get("shared_size", 0))):
            raise ConfigError("scores over all router outputs: at most 256 outputs, and a "
                              "shared expert without a gate")
        self.groups = int(p.get("groups", 1))
        self.keep_groups = int(p.get("keep_groups", self.groups))
        if self.groups > 1 and (not scored or self.groups > 32 or self.routed % self.groups
                                or not 1 <= self.keep_groups <= self.groups
                                or self.top > self.keep_groups * (self.routed // self.groups)):
            raise ConfigError(f"{self.top} of {self.routed} experts from {self.keep_groups} of "
                              f"{self.groups} groups")
        if self.identity and not scored:
            raise ConfigError("identity experts come with scores over all router outputs")
        if self.top > self.routed:
            raise ConfigError(f"{self.top} of {self.routed} experts per token")
        if p.get("activation", "silu") not in K.ACTIVATIONS:
            raise ConfigError(f"activation \"{p['activation']}\" is not known")
        self.act = K.ACTIVATIONS[p.get("activation", "silu")]
        names = p["names"]
        self.n_router = prefix + names["router"]
        self.n_expert = [prefix + names["expert"].format(e) for e in range(self.experts)]
        self.n_shared = prefix + names["shared"]
        self.n_shared_gate = prefix + names.get("shared_gate", "")
        self.n_correction = prefix + names["correction"] if "correction" in names else None
        self.leaf = {k: names[k] for k in ("gate", "up", "down")}
        # for tests and debugging: called with (part, step, chosen experts [T, top] on the
        # device) in every forward; while it is set the part is not captured into graphs
        self.probe = None

    def libraries(self, rt) -> List[str]:
        return ["moe"] + (["moe_tc"] if rt.fast_kernels else [])

    can_store = True      # forward(..., store=True) writes its output into x instead of adding

    def tensors(self) -> List[TensorNeed]:
        l = self.leaf
        out = [TensorNeed(self.n_router, (self.routed, self.hidden))]
        if self.n_correction:
            out.append(TensorNeed(self.n_correction, (self.routed,), "bias"))
        for e in self.n_expert:
            out += [TensorNeed(e + l["gate"], (self.inter, self.hidden)),
                    TensorNeed(e + l["up"], (self.inter, self.hidden)),
                    TensorNeed(e + l["down"], (self.hidden, self.inter))]
        if self.shared_size:
            s = self.n_shared
            out += [TensorNeed(s + l["gate"], (self.shared_size, self.hidden)),
                    TensorNeed(s + l["up"], (self.shared_size, self.hidden)),
                    TensorNeed(s + l["down"], (self.hidden, self.shared_size))]
            if self.shared_gate:
                out.append(TensorNeed(self.n_shared_gate, (1, self.hidden)))
        return out

    def bind(self, weights: Dict[str, torch.Tensor], rt) -> None:
        self.rt = rt
        l = self.leaf
        consume = getattr(rt, "consume_weights", False)
        take = (lambda name: weights.pop(name)) if consume else (lambda name: weights[name])
        router = [take(self.n_router)]
        if self.shared_size and self.shared_gate:
            router.append(take(self.n_shared_gate))
        self.correction = (weights[self.n_correction].to(torch.float32).contiguous()
                           if self.n_correction else None)
        if len({w.dtype for w in router}) > 1:
            router = [w.float() for w in router]
        self.router = Linear(torch.cat(router, dim=0), rt)      # the gate's row behind the experts'
        ws = [take(e + l[k]) for e in self.n_expert for k in ("gate", "up", "down")]
        kind = ws[0].dtype if len({w.dtype for w in ws}) == 1 else torch.float32
        dev = ws[0].device
        # all experts' weights in two tensors: [E, 2 ff, hidden] (gate rows, then up rows) and
        # [E, hidden, ff]
        self.w_up = torch.empty((self.experts, 2 * self.inter, self.hidden), dtype=kind, device=dev)
        self.w_down = torch.empty((self.experts, self.hidden, self.inter), dtype=kind, device=dev)
        for e in range(self.experts):
            self.w_up[e, :self.inter].copy_(ws[3 * e])
            self.w_up[e, self.inter:].copy_(ws[3 * e + 1])
            self.w_down[e].copy_(ws[3 * e + 2])
            ws[3 * e] = ws[3 * e + 1] = ws[3 * e + 2] = None
        self.shared_up = self.shared_down = None
        if self.shared_size:
            g, u = take(self.n_shared + l["gate"]), take(self.n_shared + l["up"])
            if g.dtype != u.dtype:
                g, u = g.float(), u.float()
            # SiLU: gate and up rows alternate and the product's epilogue applies the activation
            # (as the SwiGLU feed-forward does); another activation: gate rows, then up rows,
            # and the activation kernel after the product
            self.shared_fused = self.act == K.ACT_SILU
            if self.shared_fused:
                both = torch.stack([g, u], dim=1).reshape(2 * self.shared_size, self.hidden)
            else:
                both = torch.cat([g, u], dim=0)
            self.shared_up = Linear(both, rt, swiglu=self.shared_fused)
            self.shared_down = Linear(weights[self.n_shared + l["down"]], rt)

    def forward_parts(self, h, step):
        """The output as the rows of a token's choices [top, T, hidden] float32, which the caller
        adds up in order; None for a part that has more to add (a shared expert, identity
        experts)."""
        if self.shared_size or self.identity:
            return None
        y, _, _ = self._chosen(h, step)
        return y.view(h.shape[0], self.top, self.hidden).transpose(0, 1)

    def _chosen(self, h, step, sg=None):
        """The chosen experts' rows y [T * top, hidden] (row t * top + k, weighted), their ids and
        weights [T, top]; ``sg`` [T] receives the shared expert's gate."""
        T, dev = h.shape[0], h.device
        E, top = self.experts, self.top
        A = T * top
        # [T, E (+ 1)] float32, or the split sums of the product, which the router adds up
        z = _sums(self.router(h, out_dtype=torch.float32, defer=True))
        ids = torch.empty((T, top), dtype=torch.int32, device=dev)
        w = torch.empty((T, top), dtype=torch.float32, device=dev)
        bm = tile_rows(self.rt, self.w_up, T, A, E, self.hidden, self.inter)
        max_tiles = (A + bm - 1) // bm + E
        plan = torch.empty((2 + E + A + 2 * max_tiles,), dtype=torch.int32, device=dev)
        R = self.routed
        if T <= 64:          # the router's choice and the lists in one kernel
            K.moe_route_plan(z, E, top, R, ids, w, sg, bm, max_tiles, plan, self.mode,
                             self.correction, self.route_scale, R, self.groups, self.keep_groups)
        else:
            K.moe_route(z, R, top, R, ids, w, sg, self.mode, self.correction, self.route_scale,
                        self.groups, self.keep_groups)
            K.moe_plan(ids, E, bm, max_tiles, plan)
        if self.probe is not None:
            self.probe(self, step, ids)
        y = expert_products(self.rt, h, self.w_up, self.w_down, plan, bm, max_tiles, top, self.act,
                            limit=self.limit, weight=w)
        return y, ids, w

    def forward(self, h, x, step, store: bool = False):
        T, dev, E, top = h.shape[0], h.device, self.experts, self.top
        sg = (torch.empty((T,), dtype=torch.float32, device=dev)
              if self.shared_size and self.shared_gate else None)
        y, ids, w = self._chosen(h, step, sg)
        shared = None
        if self.shared_size:
            if self.shared_fused:
                sa = self.shared_up(h)
            else:
                gu = self.shared_up(h)
                sa = torch.empty((T, self.shared_size), dtype=self.rt.dtype, device=dev)
                K.gated_act(gu, sa, self.act, limit=self.shared_limit)
            shared = _sums(self.shared_down(sa, out_dtype=torch.float32, defer=True))
        if self.identity:
            K.moe_combine(x, y, top, shared, sg, ids, w, E, h, store=store)
        else:
            K.moe_combine(x, y, top, shared, sg, store=store)
        return None


class TableExperts(Part):
    capturable = True

    def __init__(self, spec, prefix: str = ""):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden, self.vocab = int(p["hidden_size"]), int(p["vocab_size"])
        self.experts, self.top = int(p["experts"]), int(p["top"])
        self.inter, self.shared_size = int(p["intermediate_size"]), int(p.get("shared_size", 0))
        if not 0 < self.top <= self.experts:
            raise ConfigError(f"{self.top} of {self.experts} experts per token")
        if p["activation"] not in K.UNARY_ACTIVATIONS:
            raise ConfigError(f"activation \"{p['activation']}\" is not known "
                              f"(known: {', '.join(sorted(K.UNARY_ACTIVATIONS))})")
        self.act = K.UNARY_ACTIVATIONS[p["activation"]]
        names = p["names"]
        self.n_table = prefix + names["table"]
        self.n_expert = [prefix + names["expert"].format(e) for e in range(self.experts)]
        self.n_shared = prefix + names["shared"]
        self.up, self.down = names["up"], names["down"]
        # for measurements: as ``RoutedExperts.probe``, once for all runs of the layer in a pass
        self.probe = None

    def libraries(self, rt) -> List[str]:
        return ["moe"] + (["moe_tc"] if rt.fast_kernels else [])

    def tensors(self) -> List[TensorNeed]:
        out = [TensorNeed(self.n_table, (self.vocab, self.top), "choices", choices=self.experts)]
        pairs = [(e, self.inter) for e in self.n_expert]
        if self.shared_size:
            pairs.append((self.n_shared, self.shared_size))
        for name, size in pairs:
            out += [TensorNeed(name + self.up, (size, self.hidden)),
                    TensorNeed(name + self.down, (self.hidden, size))]
        return out

    def bind(self, weights: Dict[str, torch.Tensor], rt) -> None:
        self.rt = rt
        consume = getattr(rt, "consume_weights", False)
        take = (lambda name: weights.pop(name)) if consume else (lambda name: weights[name])
        self.table = weights[self.n_table].contiguous()
        if self.table.dtype != torch.int32:
            raise WeightsError(f"{self.n_table} holds {self.table.dtype}, not integers")
        lo, hi = int(self.table.min()), int(self.table.max())
        if lo < 0 or hi >= self.experts:
            raise WeightsError(f"{self.n_table} names experts {lo} to {hi} of {self.experts}")
        ws = [take(e + k) for e in self.n_expert for k in (self.up, self.down)]
        kind = ws[0].dtype if len({w.dtype for w in ws}) == 1 else torch.float32
        # all experts' weights in two tensors: [E, ff, hidden] and [E, hidden, ff]
        self.w_up = torch.empty((self.experts, self.inter, self.hidden), dtype=kind,
                                device=ws[0].device)
        self.w_down = torch.empty((self.experts, self.hidden, self.inter), dtype=kind,
                                  device=ws[0].device)
        for e in range(self.experts):
            self.w_up[e].copy_(ws[2 * e])
            self.w_down[e].copy_(ws[2 * e + 1])
            ws[2 * e] = ws[2 * e + 1] = None
        self.shared_up = self.shared_down = None
        if self.shared_size:
            self.shared_up = Linear(weights[self.n_shared + self.up], rt, unary=self.act)
            self.shared_down = Linear(weights[self.n_shared + self.down], rt)

    def plan(self, step, T: int):
        """(rows per tile, most tiles, the device's lists), made at the layer's first run in a
        pass of the model."""
        have = step.memo.get(id(self))
        if have is None:
            A = T * self.top
            bm = tile_rows(self.rt, self.w_up, T, A, self.experts, self.hidden, self.inter)
            max_tiles = (A + bm - 1) // bm + self.experts
            plan = torch.empty((2 + self.experts + A + 2 * max_tiles,), dtype=torch.int32,
                               device=self.table.device)
            if self.probe is not None:
                self.probe(self, step, self.table[step.tok_ids.long()])
            K.moe_table_plan(self.table, step.tok_ids, self.experts, bm, max_tiles, plan)
            have = step.memo[id(self)] = (bm, max_tiles, plan)
        return have

    def forward_terms(self, h, step):
        """The output as terms [(y, factor)]: the experts' rows as one part per choice, and the
        shared expert's product."""
        T = h.shape[0]
        bm, max_tiles, plan = self.plan(step, T)
        y = expert_products(self.rt, h, self.w_up, self.w_down, plan, bm, max_tiles, self.top,
                            self.act, gated=False)
        # row t * top + k is token t's k-th choice
        terms = [(y.view(T, self.top, self.hidden).transpose(0, 1), 1.0 / self.top)]
        if self.shared_size:
            sa = self.shared_up(h)
            terms.append((_sums(self.shared_down(sa, out_dtype=torch.float32, defer="any")), 1.0))
        return terms

    def forward(self, h, x, step):
        K.branch_norm(x, [(y, f, None) for y, f in self.forward_terms(h, step)])
        return None


FEED_FORWARDS.register("routed_experts", RoutedExperts)
FEED_FORWARDS.register("table_experts", TableExperts)
