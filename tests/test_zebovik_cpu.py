"""The Zebovik architecture without a GPU: its configuration reader, names and shapes, cache needs and the pages a chunked
layer keeps, the plain implementation's own sanity (closed forms of each recurrence, the planted token), and the host-side
numbers of the score cap."""
import copy
import math
import random

import numpy as np
import pytest
import torch

import plain_zebovik as PZ
import tiny
import tiny_zebovik as TZ
from kindi_b200.cache.sequence_cache import SequenceCache
from kindi_b200.config import ConfigError
from kindi_b200.config.registry import model_from_config
from kindi_b200.kernels.attention import ScoreCap, tanh_polynomial
from kindi_b200.parts.base import KVNeed, StateNeed
from kindi_b200.parts.model import cache_needs, expected_tensors, tensor_inits

F64 = torch.float64


def test_config_reads_every_size_from_the_nested_keys():
    cfg, spec = model_from_config(TZ.ZE_A)
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.logit_softcap) == (211, 64, 1e-5, 15.0)
    assert [l.kind for l in cfg.layers] == ["attention", "attention", "mlstm", "mamba2"]
    m = cfg.layers[1].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.softcap, m.rot_base, m.rot_dims, m.chunk, m.kv_from) == \
        (8, 2, 16, 24, 0.6, 35.0, 10000.0, 8, 56, 0)
    m = cfg.layers[2].mixer
    assert (m.heads, m.dim, m.vdim, m.gate_cap) == (2, 16, 24, 8.0)
    m = cfg.layers[3].mixer
    assert (m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups) == (4, 16, 24, 1, 4, 2)
    assert [l.ff for l in cfg.layers] == [48, None, 40, 56]
    for name in TZ.TINY:
        assert model_from_config(TZ.TINY[name][0])[0].to_dict() == TZ.TINY[name][0]
    names = expected_tensors(spec)
    assert names["embed"] == (211, 64) and names["head"] == (211, 64) and names["final.norm"] == (64,)
    assert names["l0.mix.q"] == (64, 64) and names["l0.mix.k.b"] == (32,) and names["l0.mix.v"] == (48, 64)
    assert names["l0.mix.o"] == (64, 96) and names["l0.norm1b"] == (64,) and names["l0.norm2b"] == (64,)
    assert names["l1.mix.q"] == (128, 64) and names["l1.mix.q.b"] == (128,) and names["l1.mix.o"] == (64, 192)
    assert not any(n.startswith(("l1.mix.k", "l1.mix.v", "l1.norm2", "l1.mlp")) for n in names)
    assert names["l2.mix.i"] == (2, 64) and names["l2.mix.f.b"] == (2,) and names["l2.mix.norm"] == (48,)
    assert names["l3.mix.in"] == (64 + 64 + 48 + 4, 64) and names["l3.mix.conv"] == (112, 4)
    assert names["l3.mix.conv.b"] == (112,) and names["l3.mix.D"] == (4,) and names["l3.mix.norm"] == (64,)
    assert names["l3.mlp.up"] == (56, 64) and names["l3.mlp.down.b"] == (64,)
    inits = tensor_inits(spec)
    assert inits["l0.norm1b"] == "gain" and inits["l2.mix.norm"] == "gain" and inits["l3.norm2b"] == "gain"


@pytest.mark.parametrize("change,word", [
    (lambda c: c.update(bogus=1), "bogus"),
    (lambda c: c["layers"][0]["mixer"].update(window=3), "window"),
    (lambda c: c["layers"][0].update(type="delta"), "delta"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "moe"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep=1), "keep"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=-1), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=8), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][3]["mixer"].update(groups=3), "groups"),
    (lambda c: c["layers"][3]["mixer"].update(norm_groups=5), "equal parts"),
    (lambda c: c["layers"][3]["mixer"].update(conv=9), "conv"),
    (lambda c: c["layers"][3]["mixer"].pop("state"), "state"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_config_errors_name_the_key(change, word):
    c = copy.deepcopy(TZ.ZE_A)
    change(c)
    with pytest.raises(ConfigError) as e:
        model_from_config(c)
    assert word in str(e.value)


@pytest.mark.parametrize("name", sorted(TZ.TINY))
def test_cache_needs_follow_the_mixers(name):
    raw = TZ.TINY[name][0]
    _, spec = model_from_config(raw)
    needs = cache_needs(spec)
    for i, (layer, need, entry) in enumerate(zip(raw["layers"], needs, spec.schedule)):
        m = layer["mixer"]
        if layer["type"] == "mlstm":
            assert need == (StateNeed((m["heads"], m["vdim"] + 1, m["dim"])), StateNeed((m["heads"],)))
        elif layer["type"] == "mamba2":
            rows = m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
            assert need[0] == StateNeed((m["heads"], m["vdim"], m["state"]))
            assert list(need[1:]) == ([StateNeed((m["conv"] - 1, rows))] if m["conv"] > 1 else [])
        elif m.get("kv_from") is not None:
            assert need is None and entry.reads_cache_of == m["kv_from"]
        else:
            # the cache keeps what the widest reader sees
            sizes = [l["mixer"]["mask"] for n, l in enumerate(raw["layers"]) if l["type"] == "attention"
                     and (n == i or l["mixer"].get("kv_from") == i)]
            want = None if any(s is None for s in sizes) else max(s["size"] for s in sizes)
            assert isinstance(need, KVNeed) and need.window == want and need.n_kv_heads == m["kv_heads"]
            assert need.head_dim >= max(m["dim"], m["vdim"]) and (need.head_dim in (64, 128) or need.head_dim > 128)


@pytest.mark.parametrize("chunk", [1, 17, 64, 100, 128, 150])
def test_a_chunked_layer_keeps_every_page_its_next_position_can_read(chunk):
    """a sequence that grows token by token (and by portions): the pages of the next position's chunk are always mapped,
    and older ones do come back"""
    cache = SequenceCache([KVNeed(1, 4, chunk)], max_tokens=640, n_slots=2, dtype=torch.float32, device="cpu",
                          max_step_tokens=64)
    for portion in (1, 7, 64):
        s = cache.alloc_slot()
        n = 0
        most = 0
        while n < 500:
            step = min(portion, 500 - n)
            cache.reserve(s, n + step)
            rows = cache.groups[0].pages.rows[s]
            for p in range(n, n + step):
                lo = PZ.chunk_start(p, chunk)
                assert all(b in rows for b in range(lo // 64, p // 64 + 1)), (portion, p)
            n += step
            cache.commit(s, n)
            most = max(most, len(rows))
        assert most <= -(-(chunk + portion) // 64) + 2
        cache.free_slot(s)
        cache.check()


# ------------------------------------------------------------------------------------------- the plain implementation
def test_the_plain_matrix_memory_is_the_sum_it_stands_for():
    """without the running maximum: S_t = sum_s exp(F_t - F_s + i_s) k_s v_s^T, and m only enters through the floor of the
    denominator"""
    g = torch.Generator().manual_seed(1)
    T, d, dv = 12, 5, 3
    q, k, v = (torch.randn(T, n, generator=g, dtype=F64) for n in (d, d, dv))
    i, f, m = PZ.mlstm_gates([3.0 * x for x in torch.randn(T, generator=g).tolist()], torch.randn(T, generator=g).tolist(), 4.0)
    assert all(abs(x) < 4.0 for x in i) and all(x < 0.0 for x in f) and m[0] == max(f[0], i[0])
    got = PZ.mlstm_head(q, k, v, i, f)
    for t in range(T):
        w = [math.exp(sum(f[s + 1:t + 1]) + i[s]) for s in range(t + 1)]
        num = sum(w[s] * float(k[s] @ q[t]) * v[s] for s in range(t + 1))
        den = sum(w[s] * float(k[s] @ q[t]) for s in range(t + 1))
        assert torch.allclose(got[t], num / (max(abs(den), 1.0) + 1e-6 * math.exp(m[t])), atol=1e-12)


def test_the_plain_state_space_head_is_the_sum_it_stands_for():
    g = torch.Generator().manual_seed(2)
    T, N, dv = 9, 4, 3
    x, B, C = torch.randn(T, dv, generator=g, dtype=F64), torch.randn(T, N, generator=g, dtype=F64), \
        torch.randn(T, N, generator=g, dtype=F64)
    dt = [PZ.softplus(u) for u in torch.randn(T, generator=g).tolist()]
    got = PZ.ssd_head(x, B, C, dt, -0.7, 1.3)
    for t in range(T):
        want = 1.3 * x[t]
        for s in range(t + 1):
            want = want + math.exp(-math.exp(-0.7) * sum(dt[s + 1:t + 1])) * dt[s] * float(B[s] @ C[t]) * x[s]
        assert torch.allclose(got[t], want, atol=1e-12)


def test_the_plain_attention_sees_its_chunk_and_one_in_the_denominator():
    T, d = 11, 4
    g = torch.Generator().manual_seed(3)
    q, k, v = (torch.randn(T, d, generator=g, dtype=F64) for _ in range(3))
    got = PZ.capped_attention(q, k, v, 0.5, 2.0, 4)
    for i in range(T):
        lo = i - i % 4
        s = 2.0 * torch.tanh((k[lo:i + 1] @ q[i]) * 0.5 / 2.0)
        want = (torch.exp(s)[:, None] * v[lo:i + 1]).sum(0) / (1.0 + torch.exp(s).sum())
        assert torch.allclose(got[i], want, atol=1e-12)
    x = torch.randn(3, 1, 6, generator=g, dtype=F64)
    assert torch.equal(PZ.rotate_half(x, 100.0, 4)[..., 4:], x[..., 4:])
    assert torch.allclose(PZ.rotate_half(x, 100.0, 4).norm(dim=-1), x.norm(dim=-1))


def test_the_planted_token_matters(tmp_path):
    """on the plain model: with the needle gone the last probe's logits move by far more than any tolerance of the GPU tests
    - in every configuration, and in one with each mixer alone"""
    alone = {"att": TZ._config(97, 64, 1e-5, None, [TZ._att(4, 2, 16, 16, None, 30.0, 10000.0, 8)]),
             "mem": TZ._config(97, 64, 1e-5, None, [TZ._mem(2, 16, 16, 8.0)]),
             "ssd": TZ._config(97, 64, 1e-5, None, [TZ._ssd(2, 16, 16, 1, 4, 1)])}
    try:
        for k, (n, c) in enumerate(alone.items()):
            TZ.TINY[n] = (c, 60 + k)
        for name in sorted(TZ.TINY):
            raw = TZ.TINY[name][0]
            folder = TZ.make_model(tmp_path, name, "float32")
            cfg, w = PZ.load_model(folder)
            toks = TZ.needle_request(raw["vocab"], 16, 2, [14, 15], random.Random(1))
            other = list(toks)
            other[2] = 7
            a, b = PZ.logits(cfg, w, toks).numpy(), PZ.logits(cfg, w, other).numpy()
            assert tiny.rel_err(a[14:], b[14:]) > 0.2, (name, tiny.rel_err(a[14:], b[14:]))
    finally:
        for n in alone:
            TZ.TINY.pop(n, None)


# ------------------------------------------------------------------------------------------- the score cap's numbers
@pytest.mark.parametrize("cap,scale,bound,mode", [(30.0, 0.1, 96.0, 2), (20.0, 0.08, 128.0, 2), (6.0, 0.1, 128.0, 1),
                                                  (30.0, 0.1, None, 1), (50.0, 1e-4, 64.0, None), (1000.0, 4.0, 64.0, None)])
def test_the_score_cap(cap, scale, bound, mode):
    c = ScoreCap(cap, scale, bound)
    assert mode is None or c.mode == mode
    h = list(c.host)
    log2e = 1.0 / math.log(2.0)
    x = np.linspace(-(bound or 500.0), bound or 500.0, 2001)
    want = log2e * cap * np.tanh(scale * x / cap)
    if c.mode == 2:
        r = x * x
        p = np.zeros_like(x)
        for k in reversed(h[4:]):
            p = p * r + k
        got = p * x
    else:
        with np.errstate(over="ignore"):
            got = h[3] * (1.0 - 2.0 / (1.0 + np.exp2(h[2] * x)))
    assert np.abs(got - want).max() <= 3e-6 * np.abs(want).max() + 1e-9
    assert c.bounded == (np.abs(want).max() <= 79.0) or abs(np.abs(want).max() - 80.0) < 2.0


def test_the_polynomial_knows_its_error():
    for bound in (0.1, 0.4, 0.9, 2.0):
        c, err = tanh_polynomial(bound)
        u = np.linspace(1e-3, bound, 999)
        got = u * np.polynomial.polynomial.polyval(u * u, c)
        assert np.abs(got / np.tanh(u) - 1.0).max() <= err * 1.01 + 1e-15
    assert tanh_polynomial(0.4)[1] < 1e-10 and tanh_polynomial(2.0)[1] > 1e-6


# ------------------------------------------------------------------------------------------- the tests' own sharpness
def _shifted_chunk(by):
    return lambda i, size: 0 if not size else max(0, min(i, (i + by) // size * size - by))


MISTAKES = {
    "chunk one token early": ("chunk_start", _shifted_chunk(1)),
    "chunk one token late": ("chunk_start", _shifted_chunk(-1)),
    "no chunk": ("chunk_start", lambda i, size: 0),
    "no cap": ("softcap", lambda x, cap: x),
    "no rotation": ("rotate_half", lambda x, base, dims: x),
    "relu instead of its square": ("feed_forward", lambda t, p, h: torch.clamp(
        h @ t[p + "up"].double().T + t[p + "up.b"].double(), min=0.0) @ t[p + "down"].double().T + t[p + "down.b"].double()),
    "bias in front of the convolution": ("causal_conv", lambda x, w, b: _ORIGINAL["causal_conv"](x + b, w, torch.zeros_like(b))),
    "no norm on the heads": ("rms", lambda x, eps: x if x.shape[-1] == 64 and x.dim() == 3 else _ORIGINAL["rms"](x, eps)),
}
_ORIGINAL = {n: getattr(PZ, n) for n in ("causal_conv", "rms")}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_a_mistake_shows_in_the_test_models(tmp_path, monkeypatch, mistake):
    """a mistake planted in the plain implementation moves the logits of a test model's requests far beyond the 32-bit
    tolerance of the GPU tests, most of them beyond the one of bfloat16"""
    model = "C" if mistake == "no cap" else "B"              # (C has caps that bend the scores)
    raw = TZ.TINY[model][0]
    folder = TZ.make_model(tmp_path, model, "float32")
    cfg, w = PZ.load_model(folder)
    toks = TZ.needle_request(raw["vocab"], 160, 95, [96, 97, 120, 149, 150, 151], random.Random(4))
    good = PZ.logits(cfg, w, toks).numpy()
    name, wrong = MISTAKES[mistake]
    monkeypatch.setattr(PZ, name, wrong)
    bad = PZ.logits(cfg, w, toks).numpy()
    assert np.max(np.abs(good - bad)) / np.max(np.abs(good)) > 0.02, mistake
