"""State-space duality (the Mamba-2 layer; Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms
Through Structured State Space Duality"): a recurrent mixer whose cache is a matrix per head and a convolution's last inputs.

One product gives ``[z (inner) | x (inner) | B (G N) | C (G N) | dt (H)]`` with ``inner = H * v_head_dim`` and N = ``state``.
x, B and C pass a causal convolution over time per channel (``conv`` taps and a bias, the last tap meets the current token,
zeros before the sequence's start) and silu. ``dt = softplus(dt + dt_bias)``. Head h uses group ``h // (H / G)``:

    S <- exp(-exp(A_log) dt) S + dt B x^T;   y = S^T C + D x

The concatenated heads are multiplied by ``silu(z)``, RMS-normed in ``norm_groups`` equal parts (each by its own root mean
square, ``eps``), multiplied by the gains ``norm`` and projected by ``W_o``.

Step sizes, decays, the recurrence and the norm are 32-bit. The cache entry holds two states per sequence, zero when it
starts: S (``[H, v_head_dim, N]``) and the last ``conv - 1`` inputs of the convolution. Prompts of the serving path run in runs
of tokens side by side; single tokens, short steps and the true 32-bit path token by token. Sizes, ``eps`` and the tensors'
suffixes (``names``) are parameters of the part.
"""
from __future__ import annotations

from typing import Dict, Tuple

import torch

from ..config.registry import register_part
from ..config.spec import PartSpec
from ..kernels import lib as K
from ..kernels import linear as L
from .base import Branch, Mixer, StateNeed, StepContext, WeightView
from .gated_delta import pad_rows
from .mlstm import scan_in_runs

_DEFAULT_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D",
                  "norm": "norm", "o": "o"}


class StateSpaceDuality(Mixer):
    @classmethod
    def _names(cls, spec: PartSpec):
        n = dict(_DEFAULT_NAMES)
        n.update(spec.get("names") or {})
        return n

    @classmethod
    def _sizes(cls, spec: PartSpec):
        return int(spec["n_heads"]), int(spec.get("n_groups") or 1), int(spec["state"]), int(spec["v_head_dim"]), \
            int(spec["conv"])

    @classmethod
    def tensor_shapes(cls, spec: PartSpec, width: int) -> Dict[str, Tuple[int, ...]]:
        H, G, N, dv, taps = cls._sizes(spec)
        n = cls._names(spec)
        inner, C = H * dv, H * dv + 2 * G * N
        return {n["in"]: (inner + C + H, width), n["conv"]: (C, taps), n["conv_bias"]: (C,), n["dt_bias"]: (H,),
                n["A_log"]: (H,), n["D"]: (H,), n["norm"]: (inner,), n["o"]: (width, inner)}

    @classmethod
    def tensor_init(cls, spec: PartSpec, width: int) -> Dict[str, str]:
        n = cls._names(spec)
        return {n["norm"]: "gain", n["D"]: "gain"}

    @classmethod
    def cache_need(cls, spec: PartSpec, width: int):
        H, G, N, dv, taps = cls._sizes(spec)
        needs = [StateNeed((H, dv, N))]
        if taps > 1:
            needs.append(StateNeed((taps - 1, H * dv + 2 * G * N)))
        return tuple(needs)

    def __init__(self, spec, width, weights: WeightView, *, dtype, device):
        super().__init__(spec, width, weights, dtype=dtype, device=device)
        self.H, self.G, self.N, self.dv, self.taps = self._sizes(spec)
        if self.H % self.G:
            raise ValueError("n_heads %d is not a multiple of n_groups %d" % (self.H, self.G))
        if self.N > 512:
            raise ValueError("a state of up to 512 elements per value is supported, found %d" % self.N)
        if not (1 <= self.taps <= 8):
            raise ValueError("a short convolution has 1 to 8 taps, found %d" % self.taps)
        self.inner = self.H * self.dv
        self.parts = int(spec.get("norm_groups") or 1)
        if self.inner % self.parts:
            raise ValueError("%d elements cannot be normed in %d equal parts" % (self.inner, self.parts))
        self.C = self.inner + 2 * self.G * self.N
        self.eps = float(spec["eps"])
        n = self._names(spec)
        self.w_in = pad_rows(weights(n["in"]))
        self.w_conv = weights(n["conv"]).to(torch.float32).contiguous()
        self.b_conv = weights(n["conv_bias"]).to(torch.float32).contiguous()
        self.dt_bias, self.a_log, self.D, self.g_norm = (weights(n[k]).to(torch.float32).contiguous()
                                                         for k in ("dt_bias", "A_log", "D", "norm"))
        self.w_o = weights(n["o"])
        self._no_tails = torch.zeros((1, 1), dtype=torch.float32, device=device)

    def forward(self, ctx: StepContext, y: torch.Tensor) -> Branch:
        H, G, N, dv, C, inner = self.H, self.G, self.N, self.dv, self.C, self.inner
        a = L.rows_or_planes(ctx, y, self.w_in, self.dtype)
        entry = ctx.entry.cache
        state = ctx.cache.state_view(entry, self.state_base)
        tails = ctx.cache.state_view(entry, self.state_base + 1).view(-1, (self.taps - 1) * C) if self.taps > 1 \
            else self._no_tails
        # (padding rows of a recorded step are written by nobody)
        new = torch.zeros if ctx.graph and not ctx.decode else torch.empty
        c = new((ctx.T, C), dtype=a.dtype, device=y.device)
        K.short_conv(a, inner, C, None, self.w_conv, True, tails, ctx.pos, ctx.seq, ctx.slot, ctx.q_start, c,
                     out_bias=self.b_conv)
        o = new((ctx.T, inner), dtype=torch.float32, device=y.device)
        K.gated_scan("mamba2", c, inner + G * N, inner, 0, H // G, a, inner + C, 0, self.dt_bias, self.a_log, self.D, 0.0,
                     1.0, ctx.B, H, N, dv, ctx.q_start, ctx.slot, state, None, o, None, None,
                     chunked=scan_in_runs(ctx, c, N))
        yn = torch.empty((ctx.T, inner), dtype=self.dtype, device=y.device)
        K.scan_norm("mamba2", o, self.parts, self.g_norm, self.eps, a, 0, None, None, None, ctx.pos, ctx.seq, ctx.slot,
                    ctx.q_start, yn)
        return Branch(L.planes(ctx, yn, self.w_o))

    def bytes_read(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_o))


register_part("mixer", "mamba2", StateSpaceDuality)
