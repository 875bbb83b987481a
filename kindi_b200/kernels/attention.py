"""Attention over the cache: the choice of kernel by dtype and by the step's shape."""
from __future__ import annotations

import ctypes
import math
from typing import Optional

from . import lib as K


def tanh_polynomial(bound: float, terms: int = 6):
    """coefficients c of ``tanh(u) ~ u (c0 + c1 u^2 + ... )`` for |u| <= bound, and the largest relative error: Chebyshev
    interpolation of tanh(sqrt(z)) / sqrt(z) on [0, bound^2], in 64-bit"""
    import numpy as np
    top = bound * bound

    def f(z):
        r = np.sqrt(np.maximum(z, 1e-300))
        return np.where(z > 1e-12, np.tanh(r) / r, 1.0 - z / 3.0)
    cheb = np.polynomial.chebyshev.Chebyshev.interpolate(f, terms - 1, domain=[0.0, top])
    c = cheb.convert(kind=np.polynomial.Polynomial, domain=[-1.0, 1.0], window=[-1.0, 1.0]).coef
    c = np.concatenate([c, np.zeros(terms - len(c))])
    z = np.linspace(0.0, top, 4001)
    err = np.abs(np.polynomial.polynomial.polyval(z, c) / f(z) - 1.0).max()
    return c, float(err)


class ScoreCap:
    """``s -> softcap tanh(s / softcap)`` on attention scores ``s = scale (q . k)``, in the form the kernels take it.
    ``bound``: the largest ``|q . k|`` there can be, where it is known (unit-norm queries and keys): the kernels then use a
    polynomial where one of degree 11 is exact to 32-bit rounding, and the exponentials need no running maximum where the
    capped scores stay near zero"""

    POLY_ERROR = 2.5e-7         # largest relative error at which the polynomial stands in for tanh
    SAFE_LOG2 = 80.0            # capped scores within 2^+-80: sums of them stay far inside the 32-bit range

    def __init__(self, softcap: float, scale: float, bound: Optional[float] = None):
        self.softcap = float(softcap)
        log2e = 1.0 / math.log(2.0)
        reach = self.softcap
        mode, k = 1, [0.0] * 6
        if bound is not None:
            # (queries and keys are rounded to the run dtype after their norm: each element may grow by 2^-8)
            bound = 1.01 * float(bound)
            reach = min(reach, bound * scale)
            u = bound * scale / self.softcap
            c, err = tanh_polynomial(u)
            k = [log2e * self.softcap * float(ci) * (scale / self.softcap) ** (2 * i + 1) for i, ci in enumerate(c)]
            if err <= self.POLY_ERROR and all(v == 0.0 or 1e-36 < abs(v) for v in k):
                mode = 2
        bounded = 1 if reach * log2e <= self.SAFE_LOG2 else 0
        self.host = (ctypes.c_float * 10)(float(mode), float(bounded), 2.0 * log2e * scale / self.softcap,
                                          log2e * self.softcap, *k)
        self.mode, self.bounded = mode, bool(bounded)


def attention(ctx, q, out, nh, nkv, hd, scale, window, pool, table, n_pages, keep_first: int = 0, sink=None,
              gate=None, chunk: int = 0, cap: Optional[ScoreCap] = None) -> bool:
    """``out`` = attention of the (already position-encoded) query rows ``q`` over their sequences' cached keys and
    values, which include this step's: all positions up to the row's, or with ``window`` the last ``window`` of them
    and the sequence's first ``keep_first``. ``sink`` (float32 ``[nh]``): ``exp(sink_h)`` joins head h's softmax
    denominator. ``gate`` (rows or 32-bit planes laid out like ``out``): an output gate ``out *= sigmoid(gate)``; the
    return value says whether the kernel applied it (False: the caller still has to). ``chunk`` > 0: a row sees the
    positions of its own chunk of that many (counted from the sequence's first position) only. ``cap``: scores are capped"""
    if ctx.fast:
        from . import fast
        done = fast.attention_bf16(ctx, q, out, nh, nkv, hd, scale, window, pool, table, n_pages, keep_first, sink,
                                   gate, chunk, cap)
        if done:
            return done == 2
    rows_gate = gate if gate is not None and gate.dim() == 2 and gate.dtype == q.dtype else None
    K.attn_generic(q, out, ctx.pos, ctx.seq, ctx.slot, nh, nkv, hd, scale, window, pool, table, n_pages, ctx.status,
                   keep_first, sink, rows_gate, chunk, cap.softcap if cap is not None else 0.0)
    return rows_gate is not None


def latent_full_pays(ctx, *shape) -> bool:
    """see ``fast.latent_full_pays``"""
    from . import fast
    return fast.latent_full_pays(ctx, *shape)


def latent_attention(ctx, q, out, nh: int, hd: int, v_dim: int, scale: float, pool, table, n_pages) -> None:
    """``out`` ``[T, nh v_dim]`` = causal attention of the query rows ``q`` ``[T, nh hd]`` over their sequences' cached vectors
    (``pool`` ``[pages, 1, 1, 64, hd]``, this step's included): one per position, the key of every head, whose first ``v_dim``
    elements are the value"""
    if ctx.fast:
        from . import fast
        if fast.latent_attention_bf16(ctx, q, out, nh, hd, v_dim, scale, pool, table, n_pages):
            return
    K.attn_generic(q, out, ctx.pos, ctx.seq, ctx.slot, nh, 1, hd, scale, 0, pool, table, n_pages, ctx.status, v_dim=v_dim)


def attention_from_planes(ctx, qkv, out, nh, nkv, hd, scale, window, rotation, pool, table, n_pages) -> bool:
    """a decode step of the serving kernels whose QKV product came as 32-bit planes: one kernel sums them, rotates
    queries and the newest key by ``rotation`` (``(inv_freq, rotary_dim)`` of the position encoding, None when it is
    no rotation), stores the newest key and value and attends. False: not taken (the caller encodes, stores and
    attends in separate steps)"""
    if not (ctx.fast and ctx.decode and qkv.dim() == 3 and rotation is not None):
        return False
    from . import fast
    inv_freq, rotary_dim = rotation
    return fast.attention_decode_rope(ctx, qkv, out, nh, nkv, hd, scale, window, inv_freq, rotary_dim, pool, True,
                                      table, n_pages)


def sigmoid_attention(ctx, q, out, nh, nkv, hd, scale, bias, pool, table, n_pages) -> None:
    """``out`` = causal attention whose weights are ``sigmoid(q . k * scale + bias[h][distance])``, not normalised
    over keys, of the query rows ``q`` over their sequences' cached keys and values (this step's included). ``bias``:
    float32 ``[nh, n]`` over the distance, the last entry standing for every larger one, or None"""
    if ctx.decode and (hd * pool.element_size()) % 16 == 0:
        # single tokens, in either dtype: every sequence's pages in splits side by side
        from . import fast
        K.sigattn_decode(q, out, ctx.slot, ctx.kv_len, ctx.B, nh, nkv, hd, scale, bias, pool, table, n_pages,
                         splits=fast.sigmoid_decode_splits(ctx, nkv, nh // nkv), status=ctx.status)
        return
    if ctx.fast:
        from . import fast
        if fast.sigmoid_attention_bf16(ctx, q, out, nh, nkv, hd, scale, bias, pool, table, n_pages):
            return
    K.sigmoid_attn(q, out, ctx.pos, ctx.seq, ctx.slot, nh, nkv, hd, scale, bias, pool, table, n_pages, ctx.status)
