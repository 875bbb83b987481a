"""Matrix products ``out = a @ w^T`` (weights stored ``[out, in]``, as the reference's row-major ``[out][in]``
matrices, ``kindi/nbq.cu:266-296``): the choice of kernel by dtype and shape.

float32 operands always run the fixed-order 32-bit kernel (no tensor cores: the true 32-bit path). bfloat16
operands run the tcgen05 kernel where its alignment rules hold, else the general kernel. Nothing here calls a
library product.
"""
from __future__ import annotations

import torch

from . import fast
from . import lib as K


def linear(ctx, a: torch.Tensor, w: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
    """a [M, K] @ w [N, K]^T -> [M, N] in out_dtype"""
    out = torch.empty((a.shape[0], w.shape[0]), dtype=out_dtype, device=a.device)
    if not (ctx.fast and fast.gemm_rows(a, w, out, ctx.status)):
        K.gemm_simt(a, w, out)
    return out


def planes(ctx, a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """a @ w^T as 32-bit partial sums [S, M, N]: their sum over S, taken in order, is the product. The consumers
    (the next norm for a branch, the rotary/store and SwiGLU kernels) add the planes themselves, so a product that
    is split over K for the sake of parallelism needs no pass of its own to be reduced"""
    if ctx.fast:
        p = fast.gemm_planes(a, w, ctx.status)
        if p is not None:
            return p
    out = torch.empty((1, a.shape[0], w.shape[0]), dtype=torch.float32, device=a.device)
    K.gemm_simt(a, w, out[0])
    return out


def rows_or_planes(ctx, a: torch.Tensor, w: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
    """the product for a consumer that takes either form: 32-bit planes when the step is small (so that K can be
    split), else rows in out_dtype"""
    if ctx.fast and fast.wants_planes(a, w):
        p = fast.gemm_planes(a, w, ctx.status)
        if p is not None:
            return p
    return linear(ctx, a, w, out_dtype)


def linear_bias_act(ctx, y: torch.Tensor, w: torch.Tensor, bias, act: str, out_dtype: torch.dtype) -> torch.Tensor:
    """``act(y @ w^T + bias)`` (``[M, N]`` in out_dtype; ``bias`` float32 ``[N]`` or None): in the product's epilogue where a
    tensor-core kernel takes the shape, else the product as rows or 32-bit planes followed by one kernel"""
    h = torch.empty((y.shape[0], w.shape[0]), dtype=out_dtype, device=y.device)
    if ctx.fast and fast.gemm_bias_act(y, w, bias, act, h, ctx.status):
        return h
    K.bias_act(rows_or_planes(ctx, y, w, out_dtype), bias, act, h)
    return h


# ----------------------------------------------------------------------------------------------- gate / up / SwiGLU
GATE_UP_GROUP = 16      # rows of a gate group: a 32-column piece of a prompt-sized product's accumulator, the two
                        # half-warps of an epilogue warp of a decode-sized one


def join_gate_up(gate: torch.Tensor, up: torch.Tensor):
    """(the joined ``[2F, K]`` matrix, its group size). Gate and up rows alternate in groups of ``GATE_UP_GROUP``: 16
    gate rows, then the 16 up rows of the same outputs, so that a tile of the product holds both halves of its outputs
    and SwiGLU is finished in the product's epilogue; the stand-alone SwiGLU kernel reads the same grouping. A size
    that is no multiple of the group: all gates, then all ups (group = F)."""
    f, width = gate.shape
    group = GATE_UP_GROUP if f % GATE_UP_GROUP == 0 else f
    n = f // group
    joined = torch.stack([gate.view(n, group, width), up.view(n, group, width)], dim=1).reshape(2 * f, width)
    return joined.contiguous(), group


def gate_up_swiglu(ctx, y: torch.Tensor, wgu: torch.Tensor, group: int, f: int, out_dtype: torch.dtype,
                   act: str = "silu") -> torch.Tensor:
    """``act(g) * u`` (``[M, F]`` in out_dtype; ``act`` silu or gelu_tanh) with ``[g | u] = y @ wgu^T``, ``wgu`` as
    ``join_gate_up`` made it: inside the product where a tensor-core kernel takes the shape, else the product followed
    by the SwiGLU kernel"""
    h = torch.empty((y.shape[0], f), dtype=out_dtype, device=y.device)
    if ctx.fast and group == GATE_UP_GROUP and (fast.gemm_swiglu_decode(y, wgu, h, ctx.status, act)
                                                or fast.gemm_swiglu_rows(y, wgu, h, ctx.status, act)):
        return h
    gu = rows_or_planes(ctx, y, wgu, out_dtype)
    K.swiglu(gu, h, group, act)
    return h


def gate_up_glu_clamp(ctx, y: torch.Tensor, wgu: torch.Tensor, group: int, f: int, out_dtype: torch.dtype,
                      limit: float, alpha: float) -> torch.Tensor:
    """``g' sigmoid(alpha g') (u' + 1)`` with ``g' = min(g, limit)``, ``u' = clamp(u, -limit, limit)`` and
    ``[g | u] = y @ wgu^T`` (``wgu`` as ``join_gate_up`` made it): inside the product where a tensor-core kernel takes
    the shape, else the product as rows or 32-bit planes followed by the kernel of the clamped unit"""
    h = torch.empty((y.shape[0], f), dtype=out_dtype, device=y.device)
    # (the decode form that finishes the unit itself gives a tile of 128 rows of the joined matrix to at most two CTAs:
    # a matrix of fewer tiles than half the SMs - a shared expert is small - is faster as split-K planes and the
    # unit's own kernel: 18 against 31 us at 2688 x 4096 and eight rows)
    if ctx.fast and group == GATE_UP_GROUP and (
            (wgu.shape[0] >= 128 * (fast.N_SM // 2)
             and fast.gemm_swiglu_decode(y, wgu, h, ctx.status, "glu_clamp", (limit, alpha)))
            or fast.gemm_swiglu_rows(y, wgu, h, ctx.status, "glu_clamp", (limit, alpha))):
        return h
    gu = rows_or_planes(ctx, y, wgu, out_dtype)
    K.glu_clamp(gu, h, group, limit, alpha)
    return h


# ----------------------------------------------------------------------------------------------- several inputs at once
class GroupedWeight:
    """matrices ``[n_i, K]`` of one dtype that each multiply an input of their own, kept one below the other (``joined``)"""

    def __init__(self, ws):
        self.sizes = tuple(int(w.shape[0]) for w in ws)
        self.k = int(ws[0].shape[1])
        self.joined = torch.cat(list(ws), dim=0).contiguous()
        # all but the last of one size, and the last no larger: the groups' rows start at multiples of that size
        self.even = len(set(self.sizes[:-1])) == 1 and self.sizes[-1] <= self.sizes[0]

    def parts(self):
        at = 0
        for n in self.sizes:
            yield self.joined[at:at + n]
            at += n


def grouped_rows_or_planes(ctx, a: torch.Tensor, gw: GroupedWeight, out_dtype: torch.dtype):
    """the products ``a_i @ w_i^T`` of the inputs ``a = [a_0 | a_1 | ...]`` (``[M, n K]``) with the matrices of ``gw``, as a list
    in the form of ``rows_or_planes``; results of matrices of one size are laid out alike. A decode-sized step takes one launch
    for all of them where the kernel takes the shape"""
    if ctx.fast and gw.even:
        out = fast.gemm_planes_grouped(a, gw.joined, gw.sizes[0], ctx.status)
        if out is not None:
            at = [sum(gw.sizes[:i]) for i in range(len(gw.sizes))]
            return [out[:, :, c:c + n] for c, n in zip(at, gw.sizes)]
    # (a matrix with fewer rows than the first is a low-rank projection beside the others)
    return [(narrow if w.shape[0] < gw.sizes[0] else rows_or_planes)(ctx, a[:, i * gw.k:(i + 1) * gw.k], w, out_dtype)
            for i, w in enumerate(gw.parts())]


def narrow(ctx, a: torch.Tensor, w: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
    """``rows_or_planes`` for a product of few columns (a low-rank projection): 32-bit planes also for long prompts, where the
    product's few tiles would leave most of the GPU idle"""
    if ctx.fast:
        p = fast.gemm_narrow_planes(a, w, ctx.status)
        if p is not None:
            return p
    return rows_or_planes(ctx, a, w, out_dtype)
