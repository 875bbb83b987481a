"""The front end of a model: token ids to rows of the 32-bit residual stream.

``x[t] = table[tok[t]]``, the row as stored, without the scaling by the square root of the width that some
architectures apply (``kindi/nbq.cu:472-487``; ``kindi/nanbeige.py:577,681``); an architecture that does scale gives
``scale``. With ``sinusoid`` (``{"base": 10000.0}``) a position vector is added to the scaled row: column 2i gets
``sin(p * base^(-2i / width))`` and column 2i + 1 the cosine of the same angle, p the row's position in its sequence
(angles and functions in 64-bit). With ``positions`` (``{"name", "count"}``) row p of a learned table is added; with
``pairs`` (``{"name", "buckets", "mul_prev", "mul_cur"}``) a row of a table over pairs of neighbouring tokens: row
``(previous token * mul_prev + token * mul_cur) mod buckets``, and row ``buckets``, the table's last, for a sequence's first
token. The previous token is a sequence's state: the part then owns a cache entry of its own (``cache_need``), one number per
slot. Tensors' full names, the vocabulary size and the constants are parameters of the part. An architecture whose front end
is something else registers its own part of the category "embedding" with the same ``forward``.
"""
from __future__ import annotations

from typing import Dict, Tuple

import torch

from ..config.registry import register_part
from ..config.spec import PartSpec
from ..kernels import lib as K
from .base import Embedding, StateNeed, StepContext, WeightView


class TokenEmbedding(Embedding):
    @classmethod
    def tensor_shapes(cls, spec: PartSpec, width: int) -> Dict[str, Tuple[int, ...]]:
        out = {spec["name"]: (int(spec["vocab"]), width)}
        if spec.get("pairs"):
            out[spec["pairs"]["name"]] = (int(spec["pairs"]["buckets"]) + 1, width)
        if spec.get("positions"):
            out[spec["positions"]["name"]] = (int(spec["positions"]["count"]), width)
        return out

    @classmethod
    def cache_need(cls, spec: PartSpec, width: int):
        return StateNeed((1,)) if spec.get("pairs") else None

    def __init__(self, spec, width, weights: WeightView, *, dtype, device):
        super().__init__(spec, width, weights, dtype=dtype, device=device)
        self.table = weights(spec["name"])
        self.scale = float(spec.get("scale") or 1.0)
        self.freq = None
        sin = spec.get("sinusoid")
        if sin:
            base = float(sin.get("base", 10000.0))
            self.freq = torch.tensor([base ** (-2.0 * i / width) for i in range((width + 1) // 2)],
                                     dtype=torch.float64, device=device)
        pairs, positions = spec.get("pairs"), spec.get("positions")
        self.pairs = weights(pairs["name"]) if pairs else None
        self.muls = (int(pairs["mul_prev"]), int(pairs["mul_cur"])) if pairs else (0, 0)
        self.positions = weights(positions["name"]) if positions else None
        if pairs and self.table.shape[0] > 1 << 24:
            raise ValueError("a table over token pairs keeps the newest token as a 32-bit float: vocabularies up to 2^24")
        if any(w is not None and w.dtype != self.table.dtype for w in (self.pairs, self.positions)):
            raise ValueError("the embedding's tables are stored in different dtypes")

    def forward(self, ctx: StepContext) -> torch.Tensor:
        x = torch.empty((ctx.T, self.width), dtype=torch.float32, device=self.table.device)
        if self.pairs is None and self.positions is None:
            K.embed(self.table, ctx.tok, x, ctx.status, self.scale)
        else:
            last = ctx.cache.state_view(self.cache_entry) if self.pairs is not None else None
            K.embed_sum(self.table, self.pairs, self.positions, ctx, last, *self.muls, x, self.scale)
        if self.freq is not None:
            K.sinusoid_add(x, ctx.pos, self.freq)
        return x

    def bytes_read(self, n_rows: int = 0) -> int:
        tables = 1 + (self.pairs is not None) + (self.positions is not None)
        return tables * n_rows * self.width * self.table.element_size()


register_part("embedding", "table", TokenEmbedding)
