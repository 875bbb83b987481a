"""Matrix memory with exponential gates (the mLSTM of xLSTM; Beck et al., "xLSTM: Extended Long Short-Term Memory"): a
recurrent mixer whose cache is a matrix, a vector and one number per head.

``q = W_q y / sqrt(head_dim)``, ``k = W_k y`` (H heads of ``head_dim``), ``v = W_v y`` (H heads of ``v_head_dim``), no biases.
Per head a log input gate ``i = cap tanh((W_i y + b_i) / cap)`` and a log forget gate
``f = log sigmoid(cap tanh((W_f y + b_f) / cap))``. With a running maximum ``m`` (zero when a sequence starts):

    m_t = max(f + m_(t-1), i);   a = exp(f + m_(t-1) - m_t);   w = exp(i - m_t)
    S <- a S + w k v^T;   n <- a n + w k;   o = S^T q / (max(|n . q|, exp(-m_t)) + 1e-6)

Each head's o is divided by its root mean square over ``v_head_dim`` (``eps``); the concatenated heads are multiplied by the
gains ``norm`` (one per element of all heads) and by ``sigmoid(W_g y)``; then ``W_o``.

All six projections are one product; gates, maxima, the recurrence and the norm are 32-bit. The cache entry holds two states
per sequence, zero when it starts: S with n as one more row (``[H, v_head_dim + 1, head_dim]``) and m (``[H]``). Prompts of
the serving path run in runs of tokens side by side; single tokens, short steps and the true 32-bit path token by token.
Sizes, ``cap``, ``eps`` and the tensors' suffixes (``names``; ``bias``: how a gate's bias is named) are parameters of the part.
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

_DEFAULT_NAMES = {"q": "q", "k": "k", "v": "v", "i": "i", "f": "f", "bias": "%s.b", "norm": "norm", "gate": "g", "o": "o"}


def scan_in_runs(ctx: StepContext, rows: torch.Tensor, key_size: int) -> bool:
    """whether a step's recurrence runs in the form for long prompts: bf16 rows (a step of more rows than the products
    split into planes), a sequence of more than one run, keys that fit a run's tile"""
    return ctx.fast and not ctx.decode and rows.dim() == 2 and rows.dtype == torch.bfloat16 and key_size <= 256 \
        and ctx.max_q > K.scan_run()


class MatrixMemory(Mixer):
    @classmethod
    def _names(cls, spec: PartSpec):
        n = dict(_DEFAULT_NAMES)
        n.update(spec.get("names") or {})
        return n

    @classmethod
    def _sizes(cls, spec: PartSpec):
        return int(spec["n_heads"]), int(spec["head_dim"]), int(spec["v_head_dim"])

    @classmethod
    def tensor_shapes(cls, spec: PartSpec, width: int) -> Dict[str, Tuple[int, ...]]:
        H, d, dv = cls._sizes(spec)
        n = cls._names(spec)
        return {n["q"]: (H * d, width), n["k"]: (H * d, width), n["v"]: (H * dv, width), n["gate"]: (H * dv, width),
                n["o"]: (width, H * dv), n["norm"]: (H * dv,), n["i"]: (H, width), n["bias"] % n["i"]: (H,),
                n["f"]: (H, width), n["bias"] % n["f"]: (H,)}

    @classmethod
    def tensor_init(cls, spec: PartSpec, width: int) -> Dict[str, str]:
        return {cls._names(spec)["norm"]: "gain"}

    @classmethod
    def cache_need(cls, spec: PartSpec, width: int):
        H, d, dv = cls._sizes(spec)
        return (StateNeed((H, dv + 1, d)), StateNeed((H,)))

    def __init__(self, spec, width, weights: WeightView, *, dtype, device):
        super().__init__(spec, width, weights, dtype=dtype, device=device)
        self.H, self.d, self.dv = self._sizes(spec)
        if self.d > 512:
            raise ValueError("a matrix memory's keys have up to 512 elements, found %d" % self.d)
        self.cap = float(spec["cap"])
        if not (self.cap > 0):
            raise ValueError("the gates' cap must be positive, found %r" % self.cap)
        self.eps = float(spec["eps"])
        n = self._names(spec)
        ws = [weights(n[k]) for k in ("q", "k", "v", "gate", "i", "f")]
        if len({w.dtype for w in ws}) != 1:
            raise ValueError("the projections of %s are stored in different dtypes" % weights.prefix)
        self.w_in = pad_rows(torch.cat(ws, dim=0))              # [q | k | v | gate | i | f]
        self.b_i = weights(n["bias"] % n["i"]).to(torch.float32).contiguous()
        self.b_f = weights(n["bias"] % n["f"]).to(torch.float32).contiguous()
        self.g_norm = weights(n["norm"]).to(torch.float32).contiguous()
        self.w_o = weights(n["o"])

    def forward(self, ctx: StepContext, y: torch.Tensor) -> Branch:
        H, d, dv = self.H, self.d, self.dv
        a = L.rows_or_planes(ctx, y, self.w_in, self.dtype)
        entry = ctx.entry.cache
        state, m_state = (ctx.cache.state_view(entry, self.state_base + k) for k in (0, 1))
        # (padding rows of a recorded step are written by nobody)
        new = torch.zeros if ctx.graph and not ctx.decode else torch.empty
        buf = new((ctx.T * H * (dv + 2),), dtype=torch.float32, device=y.device)
        o = buf[:ctx.T * H * dv].view(ctx.T, H * dv)
        nq, m_rows = buf[ctx.T * H * dv:].view(2, ctx.T, H)
        gate = 2 * H * d + H * dv
        K.gated_scan("mlstm", a, 0, H * d, 2 * H * d, 1, a, gate + H * dv, gate + H * dv + H, self.b_i, self.b_f, None,
                     self.cap, float(d) ** -0.5, ctx.B, H, d, dv, ctx.q_start, ctx.slot, state, m_state, o, nq, m_rows,
                     chunked=scan_in_runs(ctx, a, d))
        yn = torch.empty((ctx.T, H * dv), dtype=self.dtype, device=y.device)
        K.scan_norm("mlstm", o, H, self.g_norm, self.eps, a, gate, nq, m_rows, m_state, ctx.pos, ctx.seq, ctx.slot,
                    ctx.q_start, yn)
        return Branch(L.planes(ctx, yn, self.w_o))

    def bytes_read(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_o))


register_part("mixer", "mlstm", MatrixMemory)
