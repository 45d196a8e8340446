"""Token embedding (rows of the table into the float32 residual, times ``scale`` where a
design names one; the reference scales nothing: ``decoder.pas:3292-3309``) and the head (logits = h · Headᵀ in float32, the
head being the embedding when tied: ``model.qwen3.pas:555-579``; a head with ``scale``
multiplies its float32 logits by that constant; one with ``softcap`` c turns them into
c tanh(logits / c))."""
from __future__ import annotations

from typing import Dict, List

import torch

from .. import kernels as K
from .base import EMBEDDINGS, ENTRIES, HEADS, Part, TensorNeed
from .linear import Linear, Pending


class TokenEmbedding(Part):
    capturable = True

    def __init__(self, spec, prefix: str = ""):
        super().__init__(spec, prefix)
        self.name = spec.params["name"]
        self.vocab, self.hidden = int(spec.params["vocab_size"]), int(spec.params["hidden_size"])
        self.scale = float(spec.params.get("scale", 1.0))

    def tensors(self) -> List[TensorNeed]:
        return [TensorNeed(self.name, (self.vocab, self.hidden), "table")]

    def bind(self, weights: Dict[str, torch.Tensor], rt) -> None:
        self.table = weights[self.name]

    def forward(self, ids: torch.Tensor, x: torch.Tensor) -> None:
        """x [T, hidden], or [streams, T, hidden]: every stream starts as the same rows."""
        K.embed(self.table, ids, x, self.scale)


class LmHead(Part):
    capturable = True

    def __init__(self, spec, prefix: str = ""):
        super().__init__(spec, prefix)
        p = spec.params
        self.tied = bool(p["tied"])
        self.name = p["tied_to"] if self.tied else p["name"]
        self.stored_name = p["name"]
        self.vocab, self.hidden = int(p["vocab_size"]), int(p["hidden_size"])
        self.scale = float(p.get("scale", 1.0))
        self.softcap = float(p.get("softcap") or 0.0)    # logits <- c tanh(logits / c)

    def tensors(self) -> List[TensorNeed]:
        if self.tied:
            # a stored copy of a tied head is tolerated when it equals the embedding
            return [TensorNeed(self.stored_name, (self.vocab, self.hidden), "table", optional=True,
                               must_equal=self.name)]
        return [TensorNeed(self.name, (self.vocab, self.hidden), "matrix")]

    def bind(self, weights: Dict[str, torch.Tensor], rt) -> None:
        self.linear = Linear(weights[self.name], rt)

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        logits = self.linear(h, out_dtype=torch.float32)
        if self.scale != 1.0:
            K.scale_rows(logits, self.scale)
        if self.softcap > 0:
            K.softcap_rows(logits, self.softcap)
        return logits


class PassInput(Part):
    """What a pass through looped layers adds to the residual before its first layer: row
    ``row`` of the table ``name`` [rows, size] and, with ``add_embedding``, the embedding's
    output once more (the model keeps a copy of it for the runs that ask)."""
    capturable = True

    def __init__(self, spec, prefix: str = ""):
        super().__init__(spec, prefix)
        p = spec.params
        self.name = prefix + p["name"]
        self.rows, self.row, self.size = int(p["rows"]), int(p["row"]), int(p["size"])
        self.add_embedding = bool(p.get("add_embedding", False))

    def tensors(self) -> List[TensorNeed]:
        return [TensorNeed(self.name, (self.rows, self.size), "bias")]

    def bind(self, weights: Dict[str, torch.Tensor], rt) -> None:
        self.vector = weights[self.name][self.row].contiguous()

    def forward(self, x: torch.Tensor, x0) -> None:
        K.pass_input(x, self.vector, x0 if self.add_embedding else None)


class PassProjection(Part):
    """What a pass through looped layers starts from: x = W_in [x ; x0] + step[row], x0 the
    embedding's output (``names``: ``in`` [size, 2 size], x's columns first, and ``step`` [rows,
    size]). One kernel adds what is still pending into x, writes [x ; x0] in the activation type
    (x0 from the embedding's table) and puts step[row] in x's place; the product is added onto
    that."""
    capturable = True
    accepts_pending = True      # forward(..., pending=) -> what is pending afterwards

    def __init__(self, spec, prefix: str = ""):
        super().__init__(spec, prefix)
        p = spec.params
        self.names = {k: prefix + v for k, v in p["names"].items()}
        self.rows, self.row, self.size = int(p["rows"]), int(p["row"]), int(p["size"])

    def tensors(self) -> List[TensorNeed]:
        return [TensorNeed(self.names["in"], (self.size, 2 * self.size)),
                TensorNeed(self.names["step"], (self.rows, self.size), "bias")]

    def bind(self, weights: Dict[str, torch.Tensor], rt) -> None:
        self.rt = rt
        self.linear = Linear(weights[self.names["in"]], rt)
        self.vector = weights[self.names["step"]][self.row].to(torch.float32).contiguous()

    def forward(self, x: torch.Tensor, step, embedding, pending=None):
        from .block import BranchSums, settle
        if pending is not None and not isinstance(pending, BranchSums):
            settle(x, pending)
            pending = None
        both = torch.empty((x.shape[0], 2 * self.size), dtype=self.rt.dtype, device=x.device)
        K.pass_concat(x, pending.terms if pending is not None else [], embedding.table,
                      step.tok_ids, embedding.scale, self.vector, both)
        y = self.linear(both, out_dtype=torch.float32, defer="any")
        return BranchSums([(y.partial if isinstance(y, Pending) else y, 1.0, None)])


EMBEDDINGS.register("token_embedding", TokenEmbedding)
ENTRIES.register("pass_input", PassInput)
ENTRIES.register("pass_projection", PassProjection)
HEADS.register("lm_head", LmHead)
