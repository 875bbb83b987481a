"""The Zebovik architecture on the GPU against the plain implementation (``plain_zebovik``): each mechanism's kernel alone,
then whole models of five small configurations through the engine's step function, its cache and its generation loop, in
true 32-bit and in bfloat16.

The models carry a planted token (``tiny_zebovik.plant``): a probe's output rests on one needle token in every mixer, so a
dropped key, a chunk that is one token off, a page of another sequence, a lost state or a slot's old content changes a probe's
logits by many times the tolerance. The 32-bit runs are the sharp ones for everything else.
"""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_zebovik as PZ
import tiny
import tiny_zebovik as TZ

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F64 = torch.float64
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
# relative to a request's largest logit; bfloat16 stores activations in 16 bits, and a layer adds a branch of unit size
# whatever the branch's own size was. What the planted token changes is more than 20 %.
TOL = {"float32": 5e-5, "bfloat16": 0.12}
TYPICAL = 0.03             # bfloat16: the median row of a request
ROWS_OVER = 0.01           # bfloat16: rows that may miss the tolerance (a norm on a nearly cancelled sum amplifies rounding)


@pytest.fixture(scope="module")
def K():
    from kindi_b200.kernels import lib
    lib.load()
    return lib


def _status():
    return torch.zeros(1, dtype=torch.int32, device="cuda")


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).abs().max() / (b.abs().max() + 1e-30))


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _ctx(T, tdt, fast, **kw):
    from kindi_b200.parts.base import StepContext
    base = dict(T=T, B=1, tok=None, pos=None, seq=None, slot=None, q_start=None, kv_len=None, h_slot=None,
                h_q_start=None, h_kv_len=None, decode=False, max_q=T, max_kv=T, dtype=tdt, device=torch.device("cuda"),
                status=_status(), fast=fast)
    base.update(kw)
    return StepContext(**base)


# ------------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("T,E,planes,ydtype,wdtype,biased,rows", [
    (1, 64, 1, "float32", "float32", False, None), (5, 200, 3, "float32", "bfloat16", True, None),
    (33, 72, 1, "bfloat16", "bfloat16", False, None), (3, 4100, 2, "float32", "float32", True, None),
    (70, 13, 2, "bfloat16", "bfloat16", True, None), (9, 8192, 4, "bfloat16", "float32", False, None),
    (4, 12000, 2, "bfloat16", "bfloat16", True, None), (20, 320, 2, "bfloat16", "bfloat16", True, [19, 0, 7]),
    (6, 50, 1, "float32", "float32", True, [5, 5])])
def test_norm_on_a_branch_add_and_next_norm(K, T, E, planes, ydtype, wdtype, biased, rows):
    g = torch.Generator().manual_seed(T * 1000 + E)
    x = torch.randn(T, E, generator=g) * 2
    d = torch.randn(planes, T, E, generator=g) * 3
    w1, w2 = ((torch.randn(E, generator=g) * 0.3 + 1).to(DT[wdtype]) for _ in range(2))
    bias = torch.randn(E, generator=g) if biased else None
    v = d.double().sum(0) + (bias.double() if biased else 0.0)
    xn = x.double() + PZ.rms(v, 1e-5) * w1.double()
    want = PZ.rms(xn, 3e-6) * w2.double()
    if rows is not None:
        want = want[rows]
    xd, st = x.cuda(), _status()
    y = torch.full(want.shape, float("nan"), dtype=DT[ydtype], device="cuda")
    K.norm_add_norm(xd, d.cuda(), bias.cuda() if biased else None, w1.cuda(), 1e-5, w2.cuda(), 3e-6, y,
                    None if rows is None else _i32(rows), rows is None, st)
    assert int(st.item()) == 0
    assert _rel(y, want) < (3e-6 if ydtype == "float32" else 6e-3)
    if rows is None:
        assert _rel(xd, xn) < 2e-6
    else:
        assert torch.equal(xd.cpu(), x)
        K.norm_add_norm(xd, d.cuda(), None, w1.cuda(), 1e-5, w2.cuda(), 3e-6, y, _i32([T] * len(rows)), False, st)
        assert int(st.item()) == K.ST_BAD_ROW


@pytest.mark.parametrize("act", ["relu2", "silu", "gelu_tanh", "none"])
@pytest.mark.parametrize("T,N,form", [(3, 40, "rows32"), (7, 13, "planes"), (130, 96, "rows16"), (9, 4100, "planes")])
def test_bias_and_activation(K, T, N, form, act):
    g = torch.Generator().manual_seed(N)
    a = torch.randn(3, T, N, generator=g) if form == "planes" else torch.randn(T, N, generator=g)
    b = torch.randn(N, generator=g)
    if form == "rows16":
        a = a.to(torch.bfloat16)
    z = (a.double().sum(0) if form == "planes" else a.double()) + b.double()
    want = {"relu2": torch.clamp(z, min=0) ** 2, "silu": PZ.silu(z), "none": z,
            "gelu_tanh": 0.5 * z * (1 + torch.tanh((2 / np.pi) ** 0.5 * (z + 0.044715 * z ** 3)))}[act]
    out = torch.empty((T, N), dtype=torch.float32 if form == "rows32" else torch.bfloat16, device="cuda")
    K.bias_act(a.cuda(), b.cuda(), act, out)
    assert _rel(out, want) < (2e-6 if form == "rows32" else 6e-3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M,N,Kd", [(1, 64, 64), (8, 4224, 1024), (40, 200, 136), (129, 96, 64), (300, 1000, 256),
                                    (700, 2048, 512), (5, 50, 72), (200, 36, 20)])
def test_product_with_bias_and_activation(K, M, N, Kd, dtype):
    """decode-sized and prompt-sized steps, sizes the tensor-core products take and sizes they do not"""
    from kindi_b200.kernels import linear as L
    g = torch.Generator().manual_seed(M + N)
    a = torch.randn(M, Kd, generator=g).to(DT[dtype])
    w = (torch.randn(N, Kd, generator=g) / Kd ** 0.5).to(DT[dtype])
    b = torch.randn(N, generator=g)
    ctx = _ctx(M, DT[dtype], dtype == "bfloat16")
    for act in ("relu2", "silu"):
        z = a.double() @ w.double().T + b.double()
        want = torch.clamp(z, min=0) ** 2 if act == "relu2" else PZ.silu(z)
        got = L.linear_bias_act(ctx, a.cuda(), w.cuda(), b.cuda(), act, DT[dtype])
        assert int(ctx.status.item()) == 0
        assert _rel(got, want) < (2e-5 if dtype == "float32" else 1.2e-2)


@pytest.mark.parametrize("taps", [1, 2, 4, 8])
@pytest.mark.parametrize("form", ["float32", "planes", "bfloat16"])
def test_convolution_with_a_bias_after_it(K, taps, form):
    """unequal sequences, cut at every kind of place, one after the other in the same slots"""
    g = torch.Generator().manual_seed(taps)
    C, lens = 40, [1, 3, 30, 170]
    w, b = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    tdt = torch.bfloat16 if form == "bfloat16" else torch.float32
    x = [torch.randn(n, C + 16, generator=g).to(tdt) for n in lens]
    want = [PZ.silu(PZ.causal_conv(v[:, 8:8 + C].double(), w.double(), b.double())) for v in x]
    tails = torch.zeros((6, max(taps - 1, 1) * C), device="cuda")
    slots = [4, 0, 5, 2]
    at = [0] * 4
    for cut in (1, 2, 5, 64, 1000):
        part = [(i, min(cut, lens[i] - at[i])) for i in range(4) if at[i] < lens[i]]
        if not part:
            break
        rows = torch.cat([x[i][at[i]:at[i] + n] for i, n in part]).cuda()
        T = rows.shape[0]
        q = [0]
        for _, n in part:
            q.append(q[-1] + n)
        pos = torch.cat([torch.arange(at[i], at[i] + n) for i, n in part]).int().cuda()
        seq = torch.cat([torch.full((n,), k) for k, (_, n) in enumerate(part)]).int().cuda()
        src = torch.stack([rows * 0.25, rows * 0.75]) if form == "planes" else rows
        out = torch.empty((T, C), dtype=tdt, device="cuda")
        K.short_conv(src, 8, C, None, w.cuda(), True, tails, pos, seq, _i32([slots[i] for i, _ in part]), _i32(q), out,
                     out_bias=b.cuda())
        for k, (i, n) in enumerate(part):
            assert _rel(out[q[k]:q[k + 1]], want[i][at[i]:at[i] + n]) < (2e-6 if form != "bfloat16" else 2e-2), (cut, i)
            at[i] += n


def _scan_case(kind, H, d, dv, G, lens, seed):
    """plain results and packed inputs of unequal sequences: (rows [T, C] float32, columns, parameters, wanted o, nq or None)"""
    g = torch.Generator().manual_seed(seed)
    T = sum(lens)
    q, k = torch.randn(T, G, d, generator=g), torch.randn(T, G, d, generator=g)
    v = torch.randn(T, H, dv, generator=g)
    q = (0.7 * k + 0.4 * q).to(torch.bfloat16).float()
    k, v = k.to(torch.bfloat16).float(), v.to(torch.bfloat16).float()
    z0, z1 = (torch.randn(T, H, generator=g).to(torch.bfloat16).float() for _ in range(2))
    p0 = torch.randn(H, generator=g)
    p1 = torch.randn(H, generator=g) + (3.0 if kind == "mlstm" else -2.0)
    p2 = torch.randn(H, generator=g)
    return q, k, v, z0, z1, p0, p1, p2


def _plain_scan(kind, H, G, q, k, v, z0, z1, p0, p1, p2, cap, qscale):
    """[n, H, dv] of one sequence; matrix memory: already divided"""
    out = torch.zeros(v.shape, dtype=F64)
    for h in range(H):
        a = h // (H // G)
        if kind == "mlstm":
            i, f, _ = PZ.mlstm_gates((z0[:, h] + p0[h]).tolist(), (z1[:, h] + p1[h]).tolist(), cap)
            out[:, h] = PZ.mlstm_head(q[:, a].double() * qscale, k[:, a].double(), v[:, h].double(), i, f)
        else:
            dt = [PZ.softplus(x) for x in (z0[:, h] + p0[h]).tolist()]
            out[:, h] = PZ.ssd_head(v[:, h].double(), k[:, a].double(), q[:, a].double(), dt, float(p1[h]), float(p2[h]))
    return out


@pytest.mark.parametrize("form", ["float32", "planes", "bfloat16", "runs"])
@pytest.mark.parametrize("kind,H,d,dv,G", [("mlstm", 2, 16, 24, 2), ("mlstm", 3, 64, 32, 3), ("mlstm", 1, 128, 80, 1),
                                           ("mlstm", 3, 10, 7, 3), ("mlstm", 2, 200, 72, 2), ("mamba2", 4, 24, 16, 1),
                                           ("mamba2", 8, 64, 16, 4), ("mamba2", 3, 128, 130, 3), ("mamba2", 2, 5, 9, 2),
                                           ("mamba2", 4, 48, 64, 2)])
def test_gated_recurrences(K, kind, H, d, dv, G, form):
    """the recurrence, its state and its norm: unequal sequences side by side, cut into steps of which the later ones start
    from the states the earlier ones left, in scattered slots; token by token and in runs"""
    lens = [1, 70, 200, 333] if form == "runs" else [1, 5, 40, 18]
    T0 = sum(lens)
    q, k, v, z0, z1, p0, p1, p2 = _scan_case(kind, H, d, dv, G, lens, seed=H * 100 + d)
    cap, qscale, eps = 6.0, (float(d) ** -0.5 if kind == "mlstm" else 1.0), 1e-5
    gen = torch.Generator().manual_seed(5)
    gate = torch.randn(T0, H * dv, generator=gen).to(torch.bfloat16).float()
    gain = torch.randn(H * dv, generator=gen) * 0.3 + 1
    parts = H if kind == "mlstm" else (G if (H * dv) % G == 0 else 1)
    b0 = [0]
    for n in lens:
        b0.append(b0[-1] + n)
    want = torch.cat([_plain_scan(kind, H, G, *(x[b0[i]:b0[i + 1]] for x in (q, k, v, z0, z1)), p0, p1, p2, cap, qscale)
                      for i in range(4)])
    if kind == "mlstm":
        yn = (PZ.rms(want, eps).reshape(T0, -1) * gain.double()) * PZ.sigmoid(gate.double())
    else:
        y = want.reshape(T0, -1) * PZ.silu(gate.double())
        yn = PZ.rms(y.view(T0, parts, -1), eps).reshape(T0, -1) * gain.double()
    rows = torch.cat([q.reshape(T0, -1), k.reshape(T0, -1), v.reshape(T0, -1), gate, z0, z1], dim=1)
    pad = -rows.shape[1] % 8
    rows = torch.cat([rows, torch.zeros(T0, pad)], dim=1)
    oq, ok, ov, og = 0, G * d, 2 * G * d, 2 * G * d + H * dv
    r = dv + (1 if kind == "mlstm" else 0)
    state, m_state = torch.zeros((7, H, r, d), device="cuda"), torch.zeros((7, H), device="cuda")
    slots = [5, 0, 6, 3]
    tdt = torch.bfloat16 if form in ("bfloat16", "runs") else torch.float32
    ydt = torch.float32 if form == "float32" else torch.bfloat16
    got, goty = torch.zeros(T0, H, dv), torch.zeros(T0, H * dv)
    at = [0] * 4
    cuts = (65, 130, 1000) if form == "runs" else (1, 2, 16, 1000)
    dev = [t.cuda() for t in (p0, p1, p2, gain)]
    for cut in cuts:
        part = [(i, min(cut, lens[i] - at[i])) for i in range(4) if at[i] < lens[i]]
        pick = torch.cat([torch.arange(b0[i] + at[i], b0[i] + at[i] + n) for i, n in part])
        T = len(pick)
        qs = [0]
        for _, n in part:
            qs.append(qs[-1] + n)
        a = rows[pick].to(tdt).cuda()
        if form == "planes":
            a = torch.stack([a * 0.5, a * 0.5])
        o = torch.full((T, H * dv), float("nan"), device="cuda")
        nq, mr = (torch.full((T, H), float("nan"), device="cuda") for _ in range(2))
        sl, qd = _i32([slots[i] for i, _ in part]), _i32(qs)
        pos = torch.cat([torch.arange(at[i], at[i] + n) for i, n in part]).int().cuda()
        seq = torch.cat([torch.full((n,), b) for b, (_, n) in enumerate(part)]).int().cuda()
        K.gated_scan(kind, a, oq, ok, ov, H // G, a, og + H * dv, og + H * dv + H, dev[0], dev[1], dev[2], cap, qscale,
                     len(part), H, d, dv, qd, sl, state, m_state if kind == "mlstm" else None, o,
                     nq if kind == "mlstm" else None, mr if kind == "mlstm" else None, chunked=form == "runs")
        y = torch.empty((T, H * dv), dtype=ydt, device="cuda")
        K.scan_norm(kind, o, parts, dev[3], eps, a, og, nq, mr, m_state, pos, seq, sl, qd, y)
        o = o.cpu().view(T, H, dv)
        if kind == "mlstm":
            den = torch.maximum(nq.abs(), torch.exp(-mr)).cpu() + 1e-6
            o = o / den[:, :, None]
        got[pick], goty[pick] = o, y.float().cpu()
        for i, n in part:
            at[i] += n
    assert at == lens
    assert _rel(got, want) < (2e-5 if form != "runs" else 5e-5), _rel(got, want)
    assert _rel(goty, yn) < (1e-4 if form == "float32" else 2e-2), _rel(goty, yn)
    assert float(state[[1, 2, 4]].abs().max()) == 0.0            # (slots of other sequences are not touched)


def _scatter_table(lengths, seed, extra=3):
    rng = random.Random(seed)
    n_blocks = [-(-n // 64) for n in lengths]
    n_pages = sum(n_blocks) + extra
    order = list(range(n_pages))
    rng.shuffle(order)
    table = torch.full((len(lengths), max(n_blocks) + 1), -1, dtype=torch.int32)
    at = 0
    for s, nb in enumerate(n_blocks):
        for b in range(nb):
            table[s, b] = order[at]
            at += 1
    return table, n_pages


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("step", ["decode", "prompt", "portion"])
@pytest.mark.parametrize("nh,nkv,hd,chunk,softcap,scale,unit", [
    (4, 2, 64, 40, 20.0, 0.19, True), (6, 1, 128, 150, 6.0, 0.1, True), (2, 2, 128, 64, 30.0, 0.09, False),
    (8, 2, 64, 1, 30.0, 0.2, True), (3, 3, 64, 1000, 200.0, 0.9, True), (5, 1, 24, 17, 9.0, 0.4, True),
    (4, 4, 128, 0, 15.0, 0.1, True), (4, 1, 64, 96, None, 0.125, True), (20, 1, 128, 100, 30.0, 0.1, True)])
def test_chunked_capped_attention(K, nh, nkv, hd, chunk, softcap, scale, unit, step, dtype):
    """keys just inside and just outside the chunk carry large values and, for some queries, the largest scores; scattered
    pages (everything outside the mapped ones is NaN); one in the denominator"""
    from kindi_b200.kernels import attention as A
    tdt = DT[dtype]
    g = torch.Generator().manual_seed(nh * 100 + chunk)
    lens = [1, 65, 200, 333]
    new = {"decode": [1, 1, 1, 1], "prompt": lens, "portion": [1, 3, 70, 130]}[step]
    table, n_pages = _scatter_table(lens, seed=hd)
    pool = torch.full((n_pages, 2, nkv, 64, hd), float("nan"), dtype=tdt)
    qs, want = [], []
    for s, L in enumerate(lens):
        k, v = torch.randn(L, nkv, hd, generator=g), torch.randn(L, nkv, hd, generator=g)
        q = torch.randn(L, nh, hd, generator=g)
        for i in range(0, L, 3):                                 # every third query rests on the key at its chunk's edge
            lo = PZ.chunk_start(i, chunk)
            for h in range(nh):
                q[i, h] = k[(lo, max(lo - 1, 0))[h % 2], h // (nh // nkv)] * 1.2
        if chunk:
            v[::chunk] += 3.0
            v[chunk - 1::chunk] -= 3.0
        if unit:
            q, k = PZ.rms(q, 1e-5), PZ.rms(k, 1e-5)
        q, k, v = q.to(tdt), k.to(tdt), v.to(tdt)
        for b in range(-(-L // 64)):
            n = min(64, L - b * 64)
            pool[table[s, b], 0, :, :n] = k[b * 64:b * 64 + n].transpose(0, 1)
            pool[table[s, b], 1, :, :n] = v[b * 64:b * 64 + n].transpose(0, 1)
            pool[table[s, b], :, :, n:] = 0.0                    # (a page's unused rows are finite, as in the cache)
        o = torch.stack([PZ.capped_attention(q[:, h].double(), k[:, h // (nh // nkv)].double(), v[:, h // (nh // nkv)].double(),
                                             scale, softcap, chunk) for h in range(nh)], dim=1)
        qs.append(q[L - new[s]:])
        want.append(o[L - new[s]:])
    q, want = torch.cat(qs).reshape(-1, nh * hd).cuda(), torch.cat(want).reshape(-1, nh * hd)
    T = q.shape[0]
    q_start = [0]
    for n in new:
        q_start.append(q_start[-1] + n)
    pos = torch.cat([torch.arange(L - n, L) for L, n in zip(lens, new)]).int().cuda()
    seq = torch.cat([torch.full((n,), b) for b, n in enumerate(new)]).int().cuda()
    ctx = _ctx(T, tdt, dtype == "bfloat16", B=4, pos=pos, seq=seq, slot=_i32([0, 1, 2, 3]), q_start=_i32(q_start),
               kv_len=_i32(lens), decode=step == "decode", max_q=max(new))
    cap = None if softcap is None else A.ScoreCap(softcap, scale, float(hd) if unit else None)
    sink = torch.zeros(nh, device="cuda")
    out = torch.full((T, nh * hd), float("nan"), dtype=tdt, device="cuda")
    A.attention(ctx, q, out, nh, nkv, hd, scale, 0, pool.cuda(), table.cuda(), n_pages, sink=sink, chunk=chunk, cap=cap)
    assert int(ctx.status.item()) == 0
    assert _rel(out, want) < (1e-5 if dtype == "float32" else 1e-2), _rel(out, want)
    if dtype == "bfloat16" and hd in (64, 128):
        # the two other tensor-core forms (mma.sync tiles for prompts) on the same step
        out2 = torch.full((T, nh * hd), float("nan"), dtype=tdt, device="cuda")
        K.attn_mma(q, out2, ctx.slot, ctx.q_start, ctx.kv_len, 4, nh, nkv, hd, scale, 0, pool.cuda(), table.cuda(), n_pages,
                   decode=False, grid_x=-(-max(new) * (nh // nkv) // 64), status=ctx.status, sink=sink, chunk=chunk,
                   cap=cap.host if cap else None)
        assert _rel(out2, want) < 1e-2


@pytest.mark.parametrize("dtype,planes", [("float32", 1), ("bfloat16", 1), ("bfloat16", 4)])
@pytest.mark.parametrize("nh,nkv,hd,dim,vdim,rot,shared", [(4, 2, 64, 16, 24, 8, False), (6, 2, 64, 64, 64, 64, False),
                                                           (4, 1, 128, 128, 64, 32, False), (3, 3, 64, 9, 24, 2, False),
                                                           (8, 2, 128, 80, 80, 0, True), (2, 2, 64, 64, 64, 64, True)])
def test_biases_rotation_and_unit_norm(K, dtype, planes, nh, nkv, hd, dim, vdim, rot, shared):
    """q and k: bias, rotation, unit norm over the head's own elements; v: bias; the widened elements stay zero; a layer
    without keys and values writes queries only"""
    g = torch.Generator().manual_seed(nh + hd + dim)
    tdt = DT[dtype]
    T, p0 = 70, 40
    own = 0 if shared else nkv
    sizes = [dim] * nh + [dim] * own + [vdim] * own
    a, b = torch.zeros(planes, T, len(sizes), hd), torch.zeros(len(sizes), hd)
    for h, n in enumerate(sizes):
        a[:, :, h, :n] = torch.randn(planes, T, n, generator=g)
        b[h, :n] = torch.randn(n, generator=g)
    if dtype == "bfloat16" and planes == 1:
        a = a.to(tdt)
    rows = a.double().sum(0) + b.double()
    pad = torch.zeros(p0, nh + own, dim, dtype=F64)
    qk = PZ.rotate_half(torch.cat([pad, rows[:, :nh + own, :dim]]), 10000.0, rot)[p0:]
    qk = PZ.rms(qk, 1e-5)
    f64 = 10000.0 ** (-2.0 * torch.arange(max(rot // 2, 1), dtype=F64) / max(rot, 1))
    xin = a.reshape(planes, T, -1).cuda()
    xin = xin if planes > 1 else xin[0]
    q = torch.full((T, nh * hd), float("nan"), dtype=tdt, device="cuda")
    pool = torch.zeros((4, 2, nkv, 64, hd), dtype=tdt, device="cuda")
    table = _i32([[2, 0, -1]])
    st = _status()
    K.headnorm_rope_store(xin, q, None, None, 1e-5, dim, "after", f64.float().cuda() if rot else None,
                          f64.cuda() if rot else None, rot, 0.0, 1, _i32(list(range(p0, p0 + T))), _i32([0] * T), _i32([0]),
                          nh, own, own, hd, pool if own else None, table, 4, st, bias=b.view(-1).cuda())
    assert int(st.item()) == 0
    tol = 3e-6 if dtype == "float32" else 6e-3
    q = q.view(T, nh, hd).cpu()
    assert _rel(q[..., :dim], qk[:, :nh]) < tol and float(q[..., dim:].abs().sum()) == 0.0
    flat = torch.cat([pool[2], pool[0]], dim=2).cpu()            # [k|v][kv head][position]
    if shared:
        assert float(flat.abs().sum()) == 0.0
        return
    kk, vv = flat[0][:, p0:p0 + T].transpose(0, 1), flat[1][:, p0:p0 + T].transpose(0, 1)
    assert _rel(kk[..., :dim], qk[:, nh:]) < tol and _rel(vv[..., :vdim], rows[:, nh + nkv:, :vdim]) < tol
    assert float(kk[..., dim:].abs().sum()) == 0.0 and float(vv[..., vdim:].abs().sum()) == 0.0
    assert float(flat[:, :, :p0].abs().sum()) == 0.0


# ------------------------------------------------------------------------------------------- whole models
def _plain(folder, reqs):
    cfg, w = PZ.load_model(folder)
    return {rid: PZ.logits(cfg, w, toks).numpy() for rid, toks in reqs.items()}


def _compare(got, reqs, want, tol, what):
    """every row within ``tol`` of the plain model's, relative to the request's largest logit; in bfloat16 one row in a
    hundred may miss it (and never by the size of what the planted token changes for all of its probes)"""
    sharp = tol < 1e-3
    errs = []
    for rid, toks in reqs.items():
        mine = np.stack([got[(rid, i)] for i in range(len(toks))])
        err = np.max(np.abs(mine - want[rid]), axis=1) / np.max(np.abs(want[rid]))
        row = int(np.argmax(err))
        if sharp:
            assert err[row] <= tol, "%s %s: %.3g at position %d of %d" % (what, rid, err[row], row, len(toks))
        else:
            assert np.median(err) <= TYPICAL, "%s %s: the median row is %.3g off" % (what, rid, np.median(err))
            probes = [i for i, t in enumerate(toks) if t == TZ.PROBE]
            assert not probes or np.median(err[probes]) <= 2 * TYPICAL, "%s %s: probes %.3g" % (what, rid,
                                                                                               np.median(err[probes]))
        errs.append((err, rid))
    if not sharp:
        over = [(rid, int(i), round(float(e[i]), 3)) for e, rid in errs for i in np.nonzero(e > tol)[0]]
        n = sum(len(e) for e, _ in errs)
        assert len(over) <= max(2, ROWS_OVER * n), "%s: %d of %d rows over: %s" % (what, len(over), n, over[:12])


def _edge_requests(raw, seed, L=200):
    """requests whose needle stands at the places that matter - the first positions, just inside and just outside chunks and
    pages, far back, right before the probes - with probes over the last positions and around every border; and the shortest
    sequences there are"""
    rng = random.Random(seed)
    vocab = raw["vocab"]
    edges = TZ.edge_places(raw, L)
    near = [p for p in edges if p >= L // 2][:4]
    reqs = {}
    for p in sorted({0, 1, 63, 64, L - 8} | set(near)):
        probes = set(range(L - 6, L)) | {e for e in edges if e > p} | {p + 1, p + 2, p + 5}
        reqs["n%d" % p] = TZ.needle_request(vocab, L, p, sorted(probes), rng)
    reqs["one"] = [rng.randrange(5, vocab)]
    reqs["two"] = [TZ.NEEDLE, TZ.PROBE]
    return reqs


def _engine(folder, steps, dtype, **kw):
    from kindi_b200.engine.engine import Engine
    return Engine(folder, ctx=tiny.max_live_tokens(steps) + 64, dtype=dtype,
                  max_batch=max(len(s["entries"]) for s in steps), **kw)


def _nothing_held(eng):
    eng.check_status()
    eng.cache.check()
    assert eng.cache.slots.n_held == 0 and all(g.pages.pool.n_held == 0 for g in eng.cache.groups)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TZ.TINY))
def test_whole_prompts_and_token_by_token(tmp_path, name, dtype):
    """every request whole in one step, then again with its last 60 tokens one by one (chunk and page borders pass under
    decoded tokens), in the same engine, slots and pages"""
    raw = TZ.TINY[name][0]
    folder = TZ.make_model(tmp_path, name, dtype)
    reqs = _edge_requests(raw, seed=3)
    want = _plain(folder, reqs)
    steps = tiny.trace_whole(reqs)
    later = tiny.trace_last_n(reqs, 60)
    for s in later:
        s["step"] += len(steps)
    eng = _engine(folder, steps + later, dtype)
    out = str(tmp_path / "out")
    tiny.run_replay(eng, steps, out)
    _compare(tiny.collect(out, steps, raw["vocab"]), reqs, want, TOL[dtype], "%s %s whole" % (name, dtype))
    tiny.run_replay(eng, later, out)
    _compare(tiny.collect(out, later, raw["vocab"]), reqs, want, TOL[dtype], "%s %s decoded" % (name, dtype))
    _nothing_held(eng)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_prompts_in_portions(tmp_path, name, dtype):
    """a prompt cut into portions of 2, 3, 31, 64, 65 and 140 tokens, and a step limit that cuts it inside the engine: the
    logits are those of the whole prompt"""
    from kindi_b200.engine.engine import Engine
    raw = TZ.TINY[name][0]
    folder = TZ.make_model(tmp_path, name, dtype)
    reqs = {k: v for k, v in _edge_requests(raw, seed=4).items() if k in ("n0", "n64", "two")}
    want = _plain(folder, reqs)
    for portion in (2, 3, 31, 64, 65, 140):
        steps = []
        for rid, toks in reqs.items():
            for a in range(0, len(toks), portion):
                part = toks[a:a + portion]
                steps.append({"step": len(steps), "entries": [{"id": rid, "tokens": part,
                                                               "want": list(range(len(part)))}],
                              "end": [rid] if a + portion >= len(toks) else []})
        eng = _engine(folder, steps, dtype)
        out = str(tmp_path / ("out%d" % portion))
        tiny.run_replay(eng, steps, out)
        _nothing_held(eng)
        _compare(tiny.collect(out, steps, raw["vocab"]), reqs, want, TOL[dtype], "%s %s by %d" % (name, dtype, portion))
    steps = tiny.trace_whole(reqs)
    eng = Engine(folder, ctx=tiny.max_live_tokens(steps) + 64, dtype=dtype, max_batch=2, max_step_tokens=64)
    out = str(tmp_path / "outcut")
    tiny.run_replay(eng, steps, out)
    _compare(tiny.collect(out, steps, raw["vocab"]), reqs, want, TOL[dtype], "%s %s cut inside" % (name, dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TZ.TINY))
def test_unequal_batches_and_reused_slots(tmp_path, name, dtype):
    """batches of unequal requests that start together and are decoded together, shorter ones ending earlier, a second batch
    in the slots and pages the first gave back: every row as if its request ran alone"""
    raw = TZ.TINY[name][0]
    folder = TZ.make_model(tmp_path, name, dtype)
    reqs = _edge_requests(raw, seed=6)
    ids = list(reqs)
    rng = random.Random(9)
    decode = {r: min(len(reqs[r]) - 1, rng.choice([0, 3, 9, 30])) for r in ids}
    half = len(ids) // 2
    steps = tiny.trace_group({r: reqs[r] for r in ids[:half]}, decode)
    steps += tiny.trace_group({r: reqs[r] for r in ids[half:]}, decode, first_step=len(steps))
    want = _plain(folder, reqs)
    eng = _engine(folder, steps, dtype)
    out = str(tmp_path / "out")
    tiny.run_replay(eng, steps, out)
    _nothing_held(eng)
    _compare(tiny.collect(out, steps, raw["vocab"]), reqs, want, TOL[dtype], "%s %s batches" % (name, dtype))


def test_a_row_is_the_same_bits_alone_and_in_a_batch(tmp_path):
    """true 32-bit: cut any way, in any company, in any slot, a row's logits are the same numbers bit for bit"""
    from kindi_b200.engine.batch import StepEntry
    raw = TZ.TINY["A"][0]
    folder = TZ.make_model(tmp_path, "A", "float32")
    from kindi_b200.engine.engine import Engine
    eng = Engine(folder, ctx=2048, dtype="float32", max_batch=8)
    reqs = list(tiny.random_requests(raw["vocab"], [90, 130, 61], seed=8).values())

    def run(entries_of):
        slots = [eng.alloc() for _ in reqs]
        at, rows = [0] * 3, [[] for _ in reqs]
        for ns in entries_of:
            live = [(i, n) for i, n in enumerate(ns) if n]
            lg = eng.step([StepEntry(slots[i], tuple(reqs[i][at[i]:at[i] + n]), tuple(range(n))) for i, n in live])
            k = 0
            for i, n in live:
                rows[i].append(lg[k:k + n].cpu())
                k += n
                at[i] += n
        for s in slots:
            eng.free(s)
        return [torch.cat(r) for r in rows]
    a = run([[90, 130, 61]])
    b = run([[0, 130, 0], [90, 0, 0], [0, 0, 61]])
    c = run([[50, 100, 2], [40, 30, 59]])
    for x, y, z in zip(a, b, c):
        assert torch.equal(x, y) and torch.equal(x, z)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_in_a_batch(tmp_path, dtype):
    """three requests decoded together for 200 steps (recorded decode steps) across chunk and page borders, probes all the way"""
    raw = TZ.TINY["B"][0]
    folder = TZ.make_model(tmp_path, "B", dtype)
    rng = random.Random(2)
    reqs = {"a": TZ.needle_request(raw["vocab"], 320, 2, list(range(60, 320, 3)), rng),
            "b": TZ.needle_request(raw["vocab"], 250, 69, list(range(100, 250, 2)), rng),
            "c": TZ.needle_request(raw["vocab"], 215, 10, list(range(20, 215, 5)), rng)}
    steps = tiny.trace_group(reqs, {"a": 200, "b": 200, "c": 200})
    want = _plain(folder, reqs)
    eng = _engine(folder, steps, dtype)
    out = str(tmp_path / "out")
    tiny.run_replay(eng, steps, out)
    assert eng.graph_replays > 150
    _nothing_held(eng)
    _compare(tiny.collect(out, steps, raw["vocab"]), reqs, want, TOL[dtype], "long %s" % dtype)


@pytest.mark.parametrize("dtype,tie", [("float32", 1e-5), ("bfloat16", 5e-2)])
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(tmp_path, name, dtype, tie):
    from kindi_b200 import Engine
    raw = TZ.TINY[name][0]
    folder = TZ.make_model(tmp_path, name, dtype)
    cfg, w = PZ.load_model(folder)
    eng = Engine(folder, ctx=2048, dtype=dtype, max_batch=3)
    prompts = list(tiny.random_requests(raw["vocab"], [5, 9, 2, 80, 13], seed=3).values())
    res = eng.generate_batch(prompts, temperature=0.0, max_tokens=10, stop_token_ids=())
    assert res.stats.batches == 2 and eng.cache.slots.n_held == 0
    for p, got in zip(prompts, res.tokens):
        assert len(got) == 10
        seq = list(p)
        for t in got:
            z = PZ.logits(cfg, w, seq)[-1].numpy()
            best = int(np.argmax(z))
            assert t == best or z[best] - z[t] <= tie * np.abs(z).max(), (len(seq), t, best)
            seq.append(t)
    eng.cache.check()


def test_trace_run_and_command_line_as_programs(tmp_path):
    folder = TZ.make_model(tmp_path, "A", "bfloat16")
    vocab = TZ.ZE_A["vocab"]
    reqs = tiny.random_requests(vocab, [5, 40], seed=2)
    steps = tiny.trace_batched(reqs, batch=2, decode=4)
    out = str(tmp_path / "out")
    env = dict(os.environ, PYTHONDONTWRITEBYTECODE="1")
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "bfloat16", "--out", out,
                        "--max-tokens", str(tiny.max_live_tokens(steps))],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, env=env,
                       timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    _compare(tiny.collect(out, steps, vocab), reqs, _plain(folder, reqs), TOL["bfloat16"], "trace_run")
    r = subprocess.run([sys.executable, "-m", "kindi_b200", "--model", folder, "--ctx", "512", "generate",
                        "--prompt-ids", "1,2,3", "--prompt-ids", "9 8", "--temperature", "0", "--max-tokens", "5"],
                       capture_output=True, text=True, cwd=ROOT, env=env, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(l) for l in r.stdout.strip().split("\n")]
    assert len(lines) == 2 and all(len(l["tokens"]) == 5 for l in lines)
    r = subprocess.run([sys.executable, "-m", "kindi_b200", "--model", folder, "info"], capture_output=True, text=True,
                       cwd=ROOT, env=env, timeout=600)
    assert r.returncode == 0 and "Zebovik" in r.stdout + r.stderr, r.stderr[-2000:]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_recorded_prompt_steps_and_their_padding_rows(tmp_path, dtype):
    """short prompt steps are padded to a multiple of 64 rows and replayed from a recording once their shape has come twice:
    the padding rows store nothing and change no other row; in 32-bit a recorded step gives the bits of an engine that
    records nothing"""
    from kindi_b200.engine.batch import StepEntry
    from kindi_b200.engine.engine import Engine
    raw = TZ.TINY["B"][0]
    folder = TZ.make_model(tmp_path, "B", dtype)
    cfg, w = PZ.load_model(folder)
    rng = random.Random(9)
    eng = Engine(folder, ctx=4096, dtype=dtype, max_batch=4)
    plain_eng = Engine(folder, ctx=4096, dtype=dtype, max_batch=4, cuda_graphs=False)

    def run(e, groups, follow=3):
        out = []
        for group in groups:
            slots = [e.alloc() for _ in group]
            k = [len(t) - follow for t in group]
            logits = e.step([StepEntry(s, tuple(t[:n]), (n - 1,)) for s, t, n in zip(slots, group, k)])
            rows = [[logits[i].cpu().numpy()] for i in range(len(group))]
            for j in range(follow):
                lg = e.step([StepEntry(s, (t[n + j],), (0,)) for s, t, n in zip(slots, group, k)])
                for i in range(len(group)):
                    rows[i].append(lg[i].cpu().numpy())
            e.check_status()
            for s in slots:
                e.free(s)
            out.append([np.stack(r) for r in rows])
        return out

    lengths = [[103], [93], [131], [68], [73], [40, 71], [64, 9], [8, 100], [200], [190], [185]]
    groups = [[TZ.needle_request(raw["vocab"], n, 1, list(range(n - 5, n)), rng) for n in g] for g in lengths]
    got = run(eng, groups)
    assert sum(1 for k in eng._graphs if k[0] == "prompt") >= 3 and eng.graph_replays >= 6
    same = run(plain_eng, groups)
    for g, mine, other in zip(groups, got, same):
        for toks, a, b in zip(g, mine, other):
            want = PZ.logits(cfg, w, toks).numpy()[len(toks) - 4:]
            assert tiny.rel_err(a, want) <= TOL[dtype], (len(toks), tiny.rel_err(a, want))
            if dtype == "float32":
                assert np.array_equal(a, b), len(toks)
    _nothing_held(eng)
