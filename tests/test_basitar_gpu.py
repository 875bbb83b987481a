"""The Basitar architecture on the GPU against the plain implementation (``plain_basitar``): each mechanism's kernel alone, then
whole models of five small configurations through the engine's step function, its cache and its generation loop, in true
32-bit and in bfloat16.

The models carry a planted token (``tiny_basitar.plant``): a probe's output rests on one needle token in every mixer, so a
dropped key, a page of another sequence, a lost state or a slot's old content changes a probe's logits by many times the
tolerance. The 32-bit runs are the sharp ones for everything else.
"""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_basitar as PB
import tiny
import tiny_basitar as TB

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F64 = torch.float64
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
# relative to a request's largest logit; bfloat16 stores activations in 16 bits, and a layer adds a branch of unit size
# whatever the branch's own size was. What the planted token changes is more than 20 %.
TOL = {"float32": 5e-5, "bfloat16": 0.12}
TYPICAL = 0.04             # bfloat16: the median row of a request
ROWS_OVER = 0.03           # bfloat16: rows that may miss the tolerance (a router's close call, a norm on a nearly cancelled sum)


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


class _Cut:
    """unequal sequences cut into steps: for every step the rows of the concatenated sequences that it brings, and its
    metadata as a context"""

    def __init__(self, lens, slots, cuts, tdt, fast=True):
        self.lens, self.slots, self.cuts, self.tdt, self.fast = lens, slots, cuts, tdt, fast
        self.b0 = [sum(lens[:i]) for i in range(len(lens))]

    def __iter__(self):
        at = [0] * len(self.lens)
        for cut in self.cuts:
            part = [(i, min(cut, n - at[i])) for i, n in enumerate(self.lens) if at[i] < n]
            if not part:
                return
            pick = torch.cat([torch.arange(self.b0[i] + at[i], self.b0[i] + at[i] + n) for i, n in part])
            q = [0]
            for _, n in part:
                q.append(q[-1] + n)
            pos = torch.cat([torch.arange(at[i], at[i] + n) for i, n in part]).int().cuda()
            seq = torch.cat([torch.full((n,), k) for k, (_, n) in enumerate(part)]).int().cuda()
            yield pick, _ctx(len(pick), self.tdt, self.fast, B=len(part), pos=pos, seq=seq,
                             slot=_i32([self.slots[i] for i, _ in part]), q_start=_i32(q),
                             kv_len=_i32([at[i] + n for i, n in part]), max_q=max(n for _, n in part))
            for i, n in part:
                at[i] += n
        assert at == list(self.lens)


# ------------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,buckets,mul_prev,mul_cur", [(64, 97, 31, 5), (33, 1, 3, 2), (300, 7, 0, -3), (8, 100003, 2 ** 40, 1)])
def test_embedding_with_pairs_and_positions(K, E, buckets, mul_prev, mul_cur, dtype):
    """sums of three tables; the token before a portion's first one is what the step before left in the slot, in company and
    alone, with single tokens between; slots of other sequences are not touched"""
    g = torch.Generator().manual_seed(E)
    vocab, lens = 50, [1, 3, 30, 70]
    toks = [torch.randint(0, vocab, (n,), generator=g).tolist() for n in lens]
    tabs = [torch.randn(n, E, generator=g).to(DT[dtype]) for n in (vocab, buckets + 1, 80)]
    want = []
    for t in toks:
        rows = PB.bigram_rows(t, buckets, mul_prev, mul_cur)
        want.append(tabs[0].double()[t] * 1.5 + tabs[1].double()[rows] + tabs[2].double()[:len(t)])
    want, flat = torch.cat(want), torch.tensor(sum(toks, []), dtype=torch.int32)
    last = torch.full((7, 1), 7.0, device="cuda")
    dev = [t.cuda() for t in tabs]
    for pick, ctx in _Cut(lens, [4, 0, 5, 2], (1, 2, 1, 5, 1000), DT[dtype]):
        ctx.tok = flat[pick].cuda()
        x = torch.empty((len(pick), E), device="cuda")
        K.embed_sum(dev[0], dev[1], dev[2], ctx, last, mul_prev, mul_cur, x, 1.5)
        assert int(ctx.status.item()) == 0
        assert _rel(x, want[pick]) < 1e-6
    assert last[[1, 3, 6]].eq(7.0).all() and last[[4, 0, 5, 2], 0].int().tolist() == [t[-1] for t in toks]
    ctx = _ctx(2, DT[dtype], True, tok=_i32([vocab, 1]), pos=_i32([0, 80]), seq=_i32([0, 0]), slot=_i32([0]), q_start=_i32([0, 2]))
    K.embed_sum(dev[0], dev[1], dev[2], ctx, last, mul_prev, mul_cur, torch.empty((2, E), device="cuda"), 1.0)
    assert int(ctx.status.item()) == K.ST_BAD_TOKEN                     # (a token and a position outside the tables)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,n", [(64, 5), (2056, 5), (37, 3), (4096, 1), (2100, 2)])
def test_token_mix(K, E, n, dtype):
    g = torch.Generator().manual_seed(E + n)
    lens = [1, 3, 30, 70]
    y = [torch.randn(m, E, generator=g).to(DT[dtype]) for m in lens]
    mu = torch.randn(n, E, generator=g)
    want = torch.cat([torch.cat([PB.token_mix(v.double(), mu[s].double()) for s in range(n)], dim=1) for v in y])
    rows = torch.cat(y)
    last = torch.zeros((7, E), device="cuda")
    for pick, ctx in _Cut(lens, [4, 0, 5, 2], (1, 2, 1, 5, 1000), DT[dtype]):
        out = torch.empty((len(pick), n * E), dtype=DT[dtype], device="cuda")
        K.token_mix(rows[pick].cuda(), mu.cuda(), last, ctx, out)
        assert _rel(out, want[pick]) < (1e-6 if dtype == "float32" else 6e-3)
    for v, s in zip(y, [4, 0, 5, 2]):
        assert torch.equal(last[s].cpu(), v[-1].float())
    assert float(last[[1, 3, 6]].abs().max()) == 0.0


@pytest.mark.parametrize("form", ["float32", "planes", "low", "bfloat16", "runs"])
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("H,d", [(2, 16), (3, 64), (1, 128), (3, 10), (2, 48), (1, 200), (5, 32), (2, 100)])
def test_recurrence_with_a_decay_per_channel(K, H, d, strong, form):
    """unequal sequences side by side, cut into steps of which the later ones start from the states the earlier ones left, in
    scattered slots; token by token (the decay's exponent given, or made from the low-rank projection) and in runs. ``strong``:
    channels that forget at once beside channels that keep, whose sums of logs differ by thousands"""
    if form == "runs" and d > 128:
        pytest.skip("heads of up to 128 channels")
    g = torch.Generator().manual_seed(H * 1000 + d)
    lens = [1, 70, 200, 150] if form == "runs" else [1, 5, 40, 18]
    T0, rank = sum(lens), 12
    r, k, v = (torch.randn(T0, H, d, generator=g).to(torch.bfloat16).float() for _ in range(3))
    low = torch.randn(T0, rank, generator=g)
    w2 = torch.randn(H * d, rank, generator=g) * (1.0 if strong else 0.4)
    w0 = torch.randn(H * d, generator=g) * (3.0 if strong else 0.5) - (0.0 if strong else 2.0)
    u = torch.randn(H * d, generator=g)
    z = torch.tanh(low.double()) @ w2.double().T
    w = torch.exp(-torch.exp(z + w0.double())).view(T0, H, d)
    b0 = [sum(lens[:i]) for i in range(5)]
    want = torch.cat([torch.stack([PB.wkv_head(*(x[b0[i]:b0[i + 1], h].double() for x in (r, k, v)), w[b0[i]:b0[i + 1], h],
                                               u.view(H, d)[h].double()) for h in range(H)], dim=1) for i in range(4)])
    tdt = torch.bfloat16 if form in ("bfloat16", "runs") else torch.float32
    state = torch.zeros((7, H, d, d), device="cuda")
    got = torch.zeros(T0, H, d)
    cuts = (65, 130, 1000) if form == "runs" else (1, 2, 16, 1000)
    for pick, ctx in _Cut(lens, [5, 0, 6, 3], cuts, tdt):
        T = len(pick)
        rows = torch.cat([x[pick].reshape(T, -1) for x in (r, k, v)], dim=1).to(tdt).cuda()
        if form == "planes":
            rows = torch.stack([rows * 0.25, rows * 0.75])
        rr, kk, vv = (rows[..., i * H * d:(i + 1) * H * d] for i in range(3))
        lo = (torch.stack([low[pick] * 0.5] * 2) if form == "planes" else low[pick]).cuda()
        use_low = form in ("planes", "low")
        o = torch.full((T, H * d), float("nan"), device="cuda")
        K.wkv(rr, kk, vv, None if use_low else z[pick].float().cuda(), lo if use_low else None, w2.cuda() if use_low else None,
              w0.cuda(), u.cuda(), ctx.B, H, d, d, ctx.q_start, ctx.slot, state, o, runs=form == "runs")
        got[pick] = o.cpu().view(T, H, d)
    assert _rel(got, want) < (1e-5 if form != "runs" else 2e-5), _rel(got, want)
    assert float(state[[1, 2, 4]].abs().max()) == 0.0            # (slots of other sequences are not touched)


@pytest.mark.parametrize("M,sizes,Kd", [(1, (128, 128, 128, 128, 16), 64), (8, (256, 256, 40), 192), (100, (128, 128, 128), 320),
                                        (40, (96, 96, 8), 128), (7, (128, 128, 12), 72), (300, (128, 128, 64), 256),
                                        (2048, (384, 384, 24), 512), (129, (64, 64, 64), 64)])
def test_products_of_several_inputs(K, M, sizes, Kd):
    """one launch for a decode-sized step where the kernel takes the shape, a product each otherwise; a narrow product of a long
    prompt comes in planes"""
    from kindi_b200.kernels import linear as L
    g = torch.Generator().manual_seed(M)
    ws = [(torch.randn(n, Kd, generator=g) / Kd ** 0.5).to(torch.bfloat16).cuda() for n in sizes]
    a = torch.randn(M, len(sizes) * Kd, generator=g).to(torch.bfloat16).cuda()
    ctx = _ctx(M, torch.bfloat16, True)
    n0 = K.launch_count()
    outs = L.grouped_rows_or_planes(ctx, a, L.GroupedWeight(ws), torch.bfloat16)
    if M <= 128 and sizes[0] % 128 == 0 and Kd % 64 == 0:
        assert K.launch_count() == n0 + 1
    for i, (o, w) in enumerate(zip(outs, ws)):
        got = o.double().sum(0) if o.dim() == 3 else o.double()
        assert _rel(got, a[:, i * Kd:(i + 1) * Kd].double() @ w.double().T) < (1e-5 if o.dim() == 3 else 6e-3), i
    assert int(ctx.status.item()) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("pairing", ["half", "interleaved"])
@pytest.mark.parametrize("q_rank,kv_rank,rot,D,scaling", [(24, 40, 8, 64, None), (13, 19, 2, 64, None), (96, 144, 32, 192, (8.0, 256.0, 16.0, 2.0)),
                                                          (300, 512, 64, 576, (4.0, 64.0, 32.0, 1.0))])
def test_latents_rotated_in_either_pairing(K, q_rank, kv_rank, rot, D, scaling, pairing, dtype):
    """both norms, the rotated parts of key and queries at positions that cross pages, one vector a position in the cache"""
    from kindi_b200.parts.rope import yarn_frequencies
    g = torch.Generator().manual_seed(D)
    tdt, T, p0, H, dim = DT[dtype], 70, 100, 3, 10
    row = torch.randn(T, q_rank + kv_rank + rot + 5, generator=g).to(tdt)
    wq, wkv = torch.rand(q_rank, generator=g).to(tdt) + 0.5, torch.rand(kv_rank, generator=g).to(tdt) + 0.5
    rspec = {"base": 10000.0, "dims": rot}
    if scaling:
        rspec["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    pad = torch.zeros(p0, 1, rot, dtype=F64)

    def turned(x):                                       # x [T, n, rot] at positions p0 ..
        return PB.rotate(torch.cat([pad.expand(-1, x.shape[1], -1), x]), rspec, pairing == "interleaved")[p0:]
    r64 = row.double()
    f, m = yarn_frequencies(10000.0, rot, rspec.get("scaling"))
    pool = torch.full((5, 1, 1, 64, D), float("nan"), dtype=tdt, device="cuda")
    table = _i32([[2, 4, 0, -1]])
    cq = torch.empty(T, q_rank, dtype=tdt, device="cuda")
    turn = dict(pairing=pairing, freq64=f.cuda() if dtype == "float32" else None)
    pos, zeros, st = _i32(list(range(p0, p0 + T))), _i32([0] * T), _status()
    K.latent_prep(row.cuda(), q_rank, kv_rank, rot, wq.cuda(), wkv.cuda(), 1e-5, f.float().cuda(), m, pos, zeros, zeros[:1], cq, D,
                  pool, table, 5, st, **turn)
    assert int(st.item()) == 0
    tol = 1e-5 if dtype == "float32" else 1.2e-2
    assert _rel(cq, PB.rms(r64[:, :q_rank], 1e-5) * wq.double()) < tol
    flat = pool[[2, 4, 0], 0, 0].reshape(192, D).cpu()
    kd = flat[p0:p0 + T]
    assert _rel(kd[:, :kv_rank], PB.rms(r64[:, q_rank:q_rank + kv_rank], 1e-5) * wkv.double()) < tol
    assert _rel(kd[:, kv_rank:kv_rank + rot], turned(r64[:, None, q_rank + kv_rank:q_rank + kv_rank + rot])[:, 0]) < tol
    assert float(kd[:, kv_rank + rot:].float().abs().sum()) == 0.0
    assert torch.isnan(flat[:p0].float()).all() and torch.isnan(flat[p0 + T:].float()).all()
    q = torch.randn(T, H * (dim + rot), generator=g).to(tdt)
    out = torch.full((T, H * D), float("nan"), dtype=tdt, device="cuda")
    K.latent_qrope(q.cuda(), dim, rot, f.float().cuda(), m, pos, out, kv_rank, D, H, **turn)
    got = out.view(T, H, D)
    assert _rel(got[..., kv_rank:kv_rank + rot], turned(q.double().view(T, H, dim + rot)[..., dim:])) < tol
    assert float(got[..., kv_rank + rot:].float().abs().sum()) == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("step", ["decode", "prompt", "portion"])
@pytest.mark.parametrize("nh,hd,v_dim", [(4, 64, 40), (6, 128, 96), (5, 192, 144), (20, 256, 200), (48, 320, 256), (4, 576, 512),
                                         (40, 576, 512), (3, 24, 16), (128, 128, 128), (1, 192, 160), (7, 64, 64)])
def test_attention_over_latents(K, nh, hd, v_dim, step, dtype):
    """keys far away, at page borders and the row's own carry the largest scores for some queries; scattered pages (everything
    outside the mapped ones is NaN); values are the keys' beginnings"""
    from kindi_b200.kernels import attention as A
    tdt = DT[dtype]
    g = torch.Generator().manual_seed(nh * 1000 + hd)
    lens = [1, 65, 130, 333] if nh * hd < 9000 else [1, 65, 100, 140]
    new = {"decode": [1, 1, 1, 1], "prompt": lens, "portion": [1, 3, 70, 100]}[step]
    rng = random.Random(hd)
    n_blocks = [-(-n // 64) for n in lens]
    order = list(range(sum(n_blocks) + 3))
    rng.shuffle(order)
    table = torch.full((4, max(n_blocks) + 1), -1, dtype=torch.int32)
    pool = torch.full((len(order), 1, 1, 64, hd), float("nan"), dtype=tdt)
    scale, at = 1.3 * hd ** -0.5, 0
    qs, want = [], []
    for s, L in enumerate(lens):
        k = torch.randn(L, hd, generator=g).to(tdt)
        q = torch.randn(L, nh, hd, generator=g)
        for i in range(0, L, 3):                                 # every third query rests on one key
            for h in range(nh):
                q[i, h] = k[max(0, (i, 0, i // 64 * 64, i // 64 * 64 - 1)[h % 4])].float() * 1.2
        q = q.to(tdt)
        for b in range(n_blocks[s]):
            table[s, b] = order[at]
            n = min(64, L - b * 64)
            pool[order[at], 0, 0, :n] = k[b * 64:b * 64 + n]
            pool[order[at], 0, 0, n:] = 0.0                      # (a page's unused rows are finite, as in the cache)
            at += 1
        rows = range(L - new[s], L)
        o = torch.zeros(len(rows), nh, v_dim, dtype=F64)
        for j, i in enumerate(rows):
            sc = (q[i].double() @ k[:i + 1].double().T) * scale
            o[j] = torch.softmax(sc, dim=1) @ k[:i + 1, :v_dim].double()
        qs.append(q[L - new[s]:])
        want.append(o)
    q, want = torch.cat(qs).reshape(-1, nh * hd).cuda(), torch.cat(want).reshape(-1, nh * v_dim)
    q_start = [0]
    for n in new:
        q_start.append(q_start[-1] + n)
    pos = torch.cat([torch.arange(L - n, L) for L, n in zip(lens, new)]).int().cuda()
    seq = torch.cat([torch.full((n,), b) for b, n in enumerate(new)]).int().cuda()
    ctx = _ctx(q.shape[0], tdt, dtype == "bfloat16", B=4, pos=pos, seq=seq, slot=_i32([0, 1, 2, 3]), q_start=_i32(q_start),
               kv_len=_i32(lens), decode=step == "decode", max_q=max(new))
    out = torch.full((q.shape[0], nh * v_dim), float("nan"), dtype=tdt, device="cuda")
    A.latent_attention(ctx, q, out, nh, hd, v_dim, scale, pool.cuda(), table.cuda(), len(order))
    assert int(ctx.status.item()) == 0
    assert _rel(out, want) < (1e-5 if dtype == "float32" else 1e-2), _rel(out, want)
    if step == "decode" and dtype == "bfloat16" and hd in K.LATENT_DIMS:
        for splits in (1, 2, 17):
            out.fill_(float("nan"))
            K.latent_attn_decode(q, out, ctx.slot, ctx.q_start, ctx.kv_len, 4, nh, hd, v_dim, scale, pool.cuda(), table.cuda(),
                                 len(order), splits=splits, status=ctx.status)
            assert _rel(out, want) < 1e-2, splits


@pytest.mark.parametrize("pairing", ["half", "interleaved"])
@pytest.mark.parametrize("nh,d,rot,dv,gated", [(3, 64, 32, 64, True), (5, 128, 64, 128, False), (2, 48, 16, 72, True), (4, 8, 16, 8, False),
                                               (1, 120, 48, 40, True), (6, 64, 16, 128, False)])
@pytest.mark.parametrize("new", [[1, 65, 130, 333], [1, 3, 70, 200]])
def test_attention_over_expanded_keys(K, nh, d, rot, dv, gated, new, pairing):
    """cached latents and rotated parts gathered from scattered pages; keys far away, at tile borders and the row's own carry the
    largest scores; queries rotated on the way in, heads gated on the way out"""
    from kindi_b200.parts.rope import yarn_frequencies
    g = torch.Generator().manual_seed(nh * 1000 + d + rot)
    lens, kr, hd = [1, 65, 130, 333], 40, 128
    rng, bf = random.Random(d), torch.bfloat16
    n_blocks = [-(-n // 64) for n in lens]
    order = list(range(sum(n_blocks) + 3))
    rng.shuffle(order)
    table = torch.full((6, max(n_blocks) + 1), -1, dtype=torch.int32)
    pool = torch.full((len(order), 1, 1, 64, hd), float("nan"), dtype=bf)
    slots, at, N = [4, 0, 5, 2], 0, sum(lens)
    cached = torch.randn(N, kr + rot, generator=g).to(bf)
    k0 = [sum(lens[:i]) for i in range(4)]
    for s, n in enumerate(lens):
        for b in range(n_blocks[s]):
            table[slots[s], b] = order[at]
            m = min(64, n - b * 64)
            pool[order[at], 0, 0, :m, :kr + rot] = cached[k0[s] + b * 64:k0[s] + b * 64 + m]
            at += 1
    lat, rotk = (torch.full((N, n), float("nan"), dtype=bf, device="cuda") for n in (kr, rot))
    st, kv_len = _status(), _i32(lens)
    K.latent_gather(pool.cuda(), kr, rot, _i32(slots), kv_len, 4, table.cuda(), len(order), lat, rotk, st)
    assert torch.equal(torch.cat([lat, rotk], dim=1).cpu(), cached)
    kv = torch.randn(N, nh * (d + dv), generator=g).to(bf)
    rspec = {"base": 100.0, "dims": rot, "scaling": {"factor": 4.0, "original": 64, "fast": 32.0, "slow": 1.0}}
    f, m = yarn_frequencies(100.0, rot, rspec["scaling"])
    scale, qs, want, pos = 1.2 * (d + rot) ** -0.5, [], [], []
    gates = torch.randn(sum(new), nh + 2, generator=g).to(bf)
    for s, n in enumerate(lens):
        k = kv[k0[s]:k0[s] + n, :nh * d].view(n, nh, d)
        v = kv[k0[s]:k0[s] + n, nh * d:].view(n, nh, dv).double()
        q = torch.randn(n, nh, d + rot, generator=g)
        for i in range(0, n, 3):
            for h in range(nh):
                q[i, h, :d] = k[max(0, (i, 0, i // 64 * 64, i // 64 * 64 - 1)[h % 4]), h].float() * 1.5
        q = q.to(bf)
        qr = torch.cat([q[:, :, :d].double(), PB.rotate(q[:, :, d:].double(), rspec, pairing == "interleaved")], dim=2)
        kr_ = cached[k0[s]:k0[s] + n, kr:].double()
        o = torch.zeros(new[s], nh, dv, dtype=F64)
        for j, i in enumerate(range(n - new[s], n)):
            for h in range(nh):
                sc = (k[:i + 1, h].double() @ qr[i, h, :d] + kr_[:i + 1] @ qr[i, h, d:]) * scale
                o[j, h] = torch.softmax(sc, dim=0) @ v[:i + 1, h]
        qs.append(q[n - new[s]:])
        want.append(o)
        pos += list(range(n - new[s], n))
    q, want = torch.cat(qs).reshape(-1, nh * (d + rot)).cuda(), torch.cat(want)
    if gated:
        want = want * torch.sigmoid(gates[:, 1:1 + nh].double())[:, :, None]
    q_start = [sum(new[:i]) for i in range(5)]
    angles = K.rope_table(_i32(pos), f.float().cuda(), rot)
    out = torch.full((len(pos), nh * dv), float("nan"), dtype=bf, device="cuda")
    K.latent_attn_full(q, nh, d, rot, dv, kv.cuda(), rotk, angles, m, pairing, gates.cuda()[:, 1:1 + nh] if gated else None, out,
                       _i32(q_start), kv_len, 4, scale, max_q=max(new), status=st)
    assert int(st.item()) == 0
    assert _rel(out, want.reshape(len(pos), -1)) < 1.2e-2, _rel(out, want.reshape(len(pos), -1))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M,H,N,Kd,planes", [(1, 2, 5, 7, 1), (70, 4, 20, 16, 2), (130, 8, 48, 32, 1), (9, 1, 100, 136, 2), (5, 3, 1, 8, 1)])
def test_products_per_head_with_a_gate_per_head(K, dtype, M, H, N, Kd, planes):
    g = torch.Generator().manual_seed(M + N)
    tdt = DT[dtype]
    a = torch.randn(M, H * Kd, generator=g).to(tdt)
    w = (torch.randn(H, N, Kd, generator=g) * 0.3).to(tdt)
    wide = torch.randn(planes, M, H + 3, generator=g)
    gate = (wide if planes > 1 else wide[0].to(tdt))
    z = (gate.double().sum(0) if planes > 1 else gate.double())[:, 1:1 + H]
    want = torch.einsum("thk,hnk->thn", a.double().view(M, H, Kd), w.double()) * torch.sigmoid(z)[:, :, None]
    for tc in (True, False):
        out = torch.zeros(M, H * N, dtype=tdt, device="cuda")
        K.head_gemm(a.cuda(), Kd, w.cuda(), out, N, gate=gate.cuda()[..., 1:1 + H], tensor_cores=tc)
        assert _rel(out.view(M, H, N), want) < (2e-5 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("per_head", [False, True])
@pytest.mark.parametrize("form", ["float32", "planes", "bfloat16"])
def test_norm_of_every_head_with_gains_of_its_own(K, form, per_head):
    g = torch.Generator().manual_seed(3)
    T, H, n = 37, 5, 20
    x = torch.randn(T, H * n, generator=g)
    w = torch.randn(H * n if per_head else n, generator=g)
    gate = torch.randn(2, T, H * n, generator=g) if form == "planes" else torch.randn(T, H * n, generator=g)
    if form == "bfloat16":
        gate = gate.to(torch.bfloat16)
    z = gate.double().sum(0) if form == "planes" else gate.double()
    gains = w.double().view(H, n) if per_head else w.double()
    want = (PB.rms(x.double().view(T, H, n), 1e-5) * gains).reshape(T, -1) * PB.silu(z)
    out = torch.empty((T, H * n), dtype=torch.float32 if form == "float32" else torch.bfloat16, device="cuda")
    K.head_norm_gate(x.cuda(), H, n, w.cuda(), 1e-5, gate.cuda(), 0, "silu", out)
    assert _rel(out, want) < (2e-6 if form == "float32" else 6e-3)


# ------------------------------------------------------------------------------------------- whole models
def _plain(folder, reqs):
    cfg, w = PB.load_model(folder)
    return {rid: PB.logits(cfg, w, toks).numpy() for rid, toks in reqs.items()}


def _compare(got, reqs, want, tol, what):
    """every row within ``tol`` of the plain model's, relative to the request's largest logit; in bfloat16 a few rows in a
    hundred may miss it"""
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
            probes = [i for i, t in enumerate(toks) if t == TB.PROBE]
            assert not probes or np.median(err[probes]) <= 2 * TYPICAL, "%s %s: probes %.3g" % (what, rid,
                                                                                               np.median(err[probes]))
        errs.append((err, rid))
    if not sharp:
        over = [(rid, int(i), round(float(e[i]), 3)) for e, rid in errs for i in np.nonzero(e > tol)[0]]
        n = sum(len(e) for e, _ in errs)
        assert len(over) <= max(2, ROWS_OVER * n), "%s: %d of %d rows over: %s" % (what, len(over), n, over[:12])


def _edge_requests(raw, seed, L=200):
    """requests whose needle stands at the places that matter - the first positions, at page and run borders, far back, right
    before the probes - with probes over the last positions and around every border; and the shortest sequences there are"""
    rng = random.Random(seed)
    vocab = raw["vocab"]
    edges = TB.edge_places(L)
    reqs = {}
    for p in (0, 1, 63, 64, 127, L - 8):
        probes = set(range(L - 6, L)) | {e for e in edges if e > p} | {p + 1, p + 2, p + 5}
        reqs["n%d" % p] = TB.needle_request(vocab, L, p, sorted(probes), rng)
    reqs["one"] = [rng.randrange(5, vocab)]
    reqs["two"] = [TB.NEEDLE, TB.PROBE]
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
@pytest.mark.parametrize("name", sorted(TB.TINY))
def test_whole_prompts_and_token_by_token(tmp_path, name, dtype):
    """every request whole in one step, then again with its last 60 tokens one by one (page borders pass under decoded tokens),
    in the same engine, slots and pages"""
    raw = TB.TINY[name][0]
    folder = TB.make_model(tmp_path, name, dtype)
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
    raw = TB.TINY[name][0]
    folder = TB.make_model(tmp_path, name, dtype)
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
@pytest.mark.parametrize("name", sorted(TB.TINY))
def test_unequal_batches_and_reused_slots(tmp_path, name, dtype):
    """batches of unequal requests that start together and are decoded together, shorter ones ending earlier, a second batch
    in the slots and pages the first gave back: every row as if its request ran alone"""
    raw = TB.TINY[name][0]
    folder = TB.make_model(tmp_path, name, dtype)
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
    raw = TB.TINY["A"][0]
    folder = TB.make_model(tmp_path, "A", "float32")
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
    """three requests decoded together for 200 steps (recorded decode steps) across page borders, probes all the way"""
    raw = TB.TINY["B"][0]
    folder = TB.make_model(tmp_path, "B", dtype)
    rng = random.Random(2)
    reqs = {"a": TB.needle_request(raw["vocab"], 320, 2, list(range(60, 320, 3)), rng),
            "b": TB.needle_request(raw["vocab"], 250, 69, list(range(100, 250, 2)), rng),
            "c": TB.needle_request(raw["vocab"], 215, 10, list(range(20, 215, 5)), rng)}
    steps = tiny.trace_group(reqs, {"a": 200, "b": 200, "c": 200})
    want = _plain(folder, reqs)
    eng = _engine(folder, steps, dtype)
    out = str(tmp_path / "out")
    tiny.run_replay(eng, steps, out)
    assert eng.graph_replays > 150
    _nothing_held(eng)
    _compare(tiny.collect(out, steps, raw["vocab"]), reqs, want, TOL[dtype], "long %s" % dtype)


def test_long_prompts_in_both_forms_of_latent_attention(tmp_path, monkeypatch):
    """a long prompt whole, in long portions and beside another: once with the keys expanded wherever the kernel takes the shape,
    once never; the expanded form does run"""
    from kindi_b200.kernels import fast
    from kindi_b200.kernels import lib
    raw = TB.TINY["B"][0]
    folder = TB.make_model(tmp_path, "B", "bfloat16")
    rng = random.Random(5)
    reqs = {"a": TB.needle_request(raw["vocab"], 620, 2, list(range(60, 620, 7)), rng),
            "b": TB.needle_request(raw["vocab"], 410, 300, list(range(301, 410, 3)), rng)}
    want = _plain(folder, reqs)
    whole = tiny.trace_whole(reqs)
    cut = [(0, 0), (300, 100), (330, 101), (620, 410)]
    steps = [{"step": len(whole) + i, "entries": [{"id": r, "tokens": reqs[r][u[k]:v[k]], "want": list(range(v[k] - u[k]))}
                                                  for k, r in enumerate("ab")], "end": ["a", "b"] if i == 2 else []}
             for i, (u, v) in enumerate(zip(cut, cut[1:]))]
    real, calls = fast.latent_full_pays, []
    count = lib.latent_attn_full
    monkeypatch.setattr(lib, "latent_attn_full", lambda *x, **kw: (calls.append(1), count(*x, **kw)))
    for rows in (1, 10 ** 9):
        monkeypatch.setattr(fast, "LATENT_FULL_MIN_ROWS", rows)
        monkeypatch.setattr(fast, "latent_full_pays", lambda ctx, *s: real(ctx, *s[:5], 10 ** 6, *s[6:]) if rows == 1 else False)
        eng = _engine(folder, whole + steps, "bfloat16", cuda_graphs=False)
        out = str(tmp_path / ("out%d" % rows))
        del calls[:]
        tiny.run_replay(eng, whole, out)
        _compare(tiny.collect(out, whole, raw["vocab"]), reqs, want, TOL["bfloat16"], "rows from %d whole" % rows)
        tiny.run_replay(eng, steps, out)
        _compare(tiny.collect(out, steps, raw["vocab"]), reqs, want, TOL["bfloat16"], "rows from %d portions" % rows)
        _nothing_held(eng)
        assert bool(calls) == (rows == 1)


@pytest.mark.parametrize("dtype,tie", [("float32", 1e-5), ("bfloat16", 8e-2)])
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(tmp_path, name, dtype, tie):
    from kindi_b200 import Engine
    raw = TB.TINY[name][0]
    folder = TB.make_model(tmp_path, name, dtype)
    cfg, w = PB.load_model(folder)
    eng = Engine(folder, ctx=2048, dtype=dtype, max_batch=3)
    prompts = list(tiny.random_requests(raw["vocab"], [5, 9, 2, 80, 13], seed=3).values())
    res = eng.generate_batch(prompts, temperature=0.0, max_tokens=10, stop_token_ids=())
    assert res.stats.batches == 2 and eng.cache.slots.n_held == 0
    for p, got in zip(prompts, res.tokens):
        assert len(got) == 10
        seq = list(p)
        for t in got:
            z = PB.logits(cfg, w, seq)[-1].numpy()
            best = int(np.argmax(z))
            assert t == best or z[best] - z[t] <= tie * np.abs(z).max(), (len(seq), t, best)
            seq.append(t)
    eng.cache.check()


def test_a_sequence_ends_at_the_last_learned_position(tmp_path):
    """generation stops where the position table does, and a step beyond it is refused"""
    from kindi_b200 import Engine
    from kindi_b200.engine.batch import StepEntry
    from kindi_b200.engine.engine import EngineError
    TB.TINY["short"] = (dict(TB.BA_A, max_positions=20), 60)
    try:
        folder = TB.make_model(tmp_path, "short", "bfloat16")
    finally:
        del TB.TINY["short"]
    eng = Engine(folder, ctx=512, dtype="bfloat16", max_batch=2)
    res = eng.generate_batch([[5, 6, 7, 8, 9], [9, 8]], temperature=0.0, max_tokens=50, stop_token_ids=())
    assert all(len(p) + len(t) in (20, 21) for p, t in zip(([5] * 5, [9] * 2), res.tokens)), [len(t) for t in res.tokens]
    s = eng.alloc()
    with pytest.raises(EngineError):
        eng.step([StepEntry(s, tuple(range(5, 26)), (0,))])
    eng.free(s)


def test_trace_run_and_command_line_as_programs(tmp_path):
    folder = TB.make_model(tmp_path, "A", "bfloat16")
    vocab = TB.BA_A["vocab"]
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
    assert r.returncode == 0 and "Basitar" in r.stdout + r.stderr, r.stderr[-2000:]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_recorded_prompt_steps_and_their_padding_rows(tmp_path, dtype):
    """short prompt steps are padded to a multiple of 64 rows and replayed from a recording once their shape has come twice:
    the padding rows store nothing and change no other row; in 32-bit a recorded step gives the bits of an engine that
    records nothing"""
    from kindi_b200.engine.batch import StepEntry
    from kindi_b200.engine.engine import Engine
    raw = TB.TINY["B"][0]
    folder = TB.make_model(tmp_path, "B", dtype)
    cfg, w = PB.load_model(folder)
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
    groups = [[TB.needle_request(raw["vocab"], n, 1, list(range(n - 5, n)), rng) for n in g] for g in lengths]
    got = run(eng, groups)
    assert sum(1 for k in eng._graphs if k[0] == "prompt") >= 3 and eng.graph_replays >= 6
    same = run(plain_eng, groups)
    for g, mine, other in zip(groups, got, same):
        for toks, a, b in zip(g, mine, other):
            want = PB.logits(cfg, w, toks).numpy()[len(toks) - 4:]
            assert tiny.rel_err(a, want) <= TOL[dtype], (len(toks), tiny.rel_err(a, want))
            if dtype == "float32":
                assert np.array_equal(a, b), len(toks)
    _nothing_held(eng)
