"""Time mixing with a decay per key channel (the WKV recurrence of RWKV-6; Peng et al., "Eagle and Finch: RWKV with
Matrix-Valued States and Dynamic Recurrence"): a recurrent mixer whose cache is a matrix per head and the token before.

With ``y'`` the input of the token before (zeros for a sequence's first token), every stream s of r, k, v, g, w reads a mix
of its own, ``y_s = y + (y' - y) mu_s``. ``r = W_r y_r``, ``k = W_k y_k`` (H heads of ``head_dim``), ``v = W_v y_v`` (H heads
of ``head_dim``), no biases; the decay of every key channel is ``w = exp(-exp(W_2 tanh(W_1 y_w) + w0))``. Per head, with a
bonus ``u`` per key channel for the current token:

    o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t;   S_t = diag(w_t) S_(t-1) + k_t v_t^T

Each head's o is divided by its root mean square (``eps``); the concatenated heads are multiplied by the gains ``norm`` (one
per element of all heads) and by ``silu(W_g y_g)``; then ``W_o``.

The mixes of a step are one kernel, the five projections products of its parts; decays, the recurrence and the norm are
32-bit. The cache entry holds two states per sequence, zero when it starts: S (``[H, head_dim, head_dim]``, values first) and
y' (``[width]``). Sizes, ``eps`` and the tensors' suffixes (``names``; ``mu``: how a stream's mixing weights are named) are
parameters of the part; the rank of the decay's projection is the tensors' own (``rank``: the one random weights get).
"""
from __future__ import annotations

from typing import Dict, Tuple

import torch

from ..config.registry import register_part
from ..config.spec import PartSpec
from ..kernels import lib as K
from ..kernels import linear as L
from .base import Branch, Mixer, StateNeed, StepContext, WeightView

_DEFAULT_NAMES = {"r": "r", "k": "k", "v": "v", "g": "g", "w1": "w1", "w2": "w2", "w0": "w0", "u": "u", "norm": "norm", "o": "o",
                  "mu": "mu.%s"}
_STREAMS = ("r", "k", "v", "g", "w")


class TimeMix(Mixer):
    @classmethod
    def _names(cls, spec: PartSpec):
        n = dict(_DEFAULT_NAMES)
        n.update(spec.get("names") or {})
        return n

    @classmethod
    def _sizes(cls, spec: PartSpec):
        return int(spec["n_heads"]), int(spec["head_dim"])

    @classmethod
    def tensor_shapes(cls, spec: PartSpec, width: int) -> Dict[str, Tuple[int, ...]]:
        H, d = cls._sizes(spec)
        n = cls._names(spec)
        rank = -int(spec.get("rank") or max(16, width // 64 // 8 * 8))          # (negative: any positive size)
        out = {n["mu"] % s: (width,) for s in _STREAMS}
        out.update({n[s]: (H * d, width) for s in ("r", "k", "v", "g")})
        out.update({n["w1"]: (rank, width), n["w2"]: (H * d, rank), n["w0"]: (H * d,), n["u"]: (H, d), n["norm"]: (H * d,),
                    n["o"]: (width, H * d)})
        return out

    @classmethod
    def tensor_init(cls, spec: PartSpec, width: int) -> Dict[str, str]:
        return {cls._names(spec)["norm"]: "gain"}

    @classmethod
    def cache_need(cls, spec: PartSpec, width: int):
        H, d = cls._sizes(spec)
        return (StateNeed((H, d, d)), StateNeed((width,)))

    def __init__(self, spec, width, weights: WeightView, *, dtype, device):
        super().__init__(spec, width, weights, dtype=dtype, device=device)
        self.H, self.d = self._sizes(spec)
        if self.d > 256:
            raise ValueError("time mixing supports heads of up to 256 channels, found %d" % self.d)
        self.eps = float(spec["eps"])
        n = self._names(spec)

        def f32(suffix):
            return weights(suffix).to(torch.float32).contiguous()
        self.mu = torch.stack([f32(n["mu"] % s) for s in _STREAMS]).contiguous()
        ws = [weights(n[s]) for s in ("r", "k", "v", "g", "w1")]
        if len({w.dtype for w in ws}) != 1:
            raise ValueError("the projections of %s are stored in different dtypes" % weights.prefix)
        self.w_in = L.GroupedWeight(ws)
        self.w2 = weights(n["w2"]).contiguous()
        self.rank = ws[-1].shape[0]
        if self.w2.shape[1] != self.rank:
            raise ValueError("%s%s has %d rows and %s%s %d columns: the decay's projection has one rank"
                             % (weights.prefix, n["w1"], self.rank, weights.prefix, n["w2"], self.w2.shape[1]))
        self.w0, self.u, self.g_norm = f32(n["w0"]), f32(n["u"]).view(-1), f32(n["norm"])
        self.w_o = weights(n["o"])

    def forward(self, ctx: StepContext, y: torch.Tensor) -> Branch:
        H, d, T = self.H, self.d, ctx.T
        state, last = (ctx.cache.state_view(ctx.entry.cache, self.state_base + k) for k in (0, 1))
        mixed = torch.empty((T, len(_STREAMS) * self.width), dtype=self.dtype, device=y.device)
        K.token_mix(y, self.mu, last, ctx, mixed)
        r, k, v, g, low = L.grouped_rows_or_planes(ctx, mixed, self.w_in, self.dtype)
        z = None
        if r.dim() == 2:
            # finished rows: the decay's exponent is a product too (small steps leave it to the recurrence's kernel)
            th = torch.empty((T, self.rank), dtype=self.dtype, device=y.device)
            K.tanh_rows(low, th)
            z = L.linear(ctx, th, self.w2, torch.float32)
        # (padding rows of a recorded step are written by nobody)
        new = torch.zeros if ctx.graph and not ctx.decode else torch.empty
        o = new((T, H * d), dtype=torch.float32, device=y.device)
        K.wkv(r, k, v, z, low, self.w2, self.w0, self.u, ctx.B, H, d, d, ctx.q_start, ctx.slot, state, o,
              runs=self._in_runs(ctx, r))
        yn = torch.empty((T, H * d), dtype=self.dtype, device=y.device)
        K.head_norm_gate(o, H, d, self.g_norm, self.eps, g, 0, "silu", yn)
        return Branch(L.planes(ctx, yn, self.w_o))

    def _in_runs(self, ctx: StepContext, rows: torch.Tensor) -> bool:
        """whether a step's recurrence runs in the form for long prompts: bf16 rows (a step of more rows than the products
        split into planes), a sequence of more than one run, heads that fit a run's tiles"""
        return ctx.fast and not ctx.decode and rows.dim() == 2 and rows.dtype == torch.bfloat16 and self.d <= 128 \
            and ctx.max_q > K.wkv_run()

    def bytes_read(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in.joined, self.w2, self.w_o))


register_part("mixer", "wkv", TimeMix)
