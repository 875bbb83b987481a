"""The Basitar architecture without a GPU: its configuration reader, names and shapes, cache needs, the schedule of layers that
run another layer's weights, the plain implementation's own sanity (closed forms of each mechanism, the planted token), and
the tests' sharpness against planted mistakes."""
import copy
import math
import random

import numpy as np
import pytest
import torch

import plain_basitar as PB
import tiny
import tiny_basitar as TB
from kindi_b200.cache.sequence_cache import SequenceCache
from kindi_b200.config import ConfigError
from kindi_b200.config.registry import model_from_config
from kindi_b200.parts.base import KVNeed, StateNeed
from kindi_b200.parts.model import cache_needs, expected_tensors, tensor_inits

F64 = torch.float64


def test_config_reads_every_size_from_the_nested_keys():
    cfg, spec = model_from_config(TB.BA_A)
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.max_positions) == (211, 64, 1e-5, 700) and spec.max_positions == 700
    assert (cfg.buckets, cfg.mul_prev, cfg.mul_cur) == (97, 31, 5)
    assert [l.kind for l in cfg.layers] == ["latent_attention", "wkv", "latent_attention_2", "wkv", "latent_attention"]
    assert [l.weights_of for l in cfg.layers] == [None, None, None, 1, 0]
    m = cfg.layers[2].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.rot_base, m.scaling) == \
        (3, 12, 4, 20, 16, 24, 16 ** -0.5, 500000.0, (4.0, 64.0, 32.0, 1.0))
    assert (cfg.layers[1].mixer.heads, cfg.layers[1].mixer.dim) == (2, 16)
    assert cfg.layers[0].ff == 48 and cfg.layers[2].ff is None
    assert (cfg.layers[1].ff.experts, cfg.layers[1].ff.top, cfg.layers[1].ff.ff) == (5, 2, 24)
    for name in TB.TINY:
        assert model_from_config(TB.TINY[name][0])[0].to_dict() == TB.TINY[name][0]
    assert [(e.layer, e.cache) for e in spec.schedule] == [(0, 0), (1, 1), (2, 2), (1, 3), (0, 4)] and len(spec.layers) == 3
    names = expected_tensors(spec)
    assert names["embed"] == (211, 64) and names["bigram"] == (98, 64) and names["pos"] == (700, 64) and "head" not in names
    assert names["l0.mix.dq"] == (24, 64) and names["l0.mix.uq"] == (96, 24) and names["l0.mix.dkv"] == (48, 64)
    assert names["l0.mix.uk"] == (64, 40) and names["l0.mix.uv"] == (96, 40) and names["l0.mix.o"] == (64, 96)
    assert "l0.mix.g" not in names and names["l2.mix.g"] == (3, 64)
    assert names["l1.mix.r"] == (32, 64) and names["l1.mix.mu.w"] == (64,) and names["l1.mix.u"] == (2, 16)
    assert names["l1.mix.w1"][0] < 0 and names["l1.mix.w2"] == (32, names["l1.mix.w1"][0])       # (any rank)
    assert names["l1.mlp.router"] == (5, 64) and names["l1.mlp.e4.down"] == (64, 24) and names["l0.mlp.gate"] == (48, 64)
    assert not any(n.startswith(("l2.norm2", "l2.mlp", "l3.", "l4.")) for n in names)
    inits = tensor_inits(spec)
    assert inits["l1.mix.norm"] == "gain" and inits["l0.mix.dq.norm"] == "gain" and "l0.norm1" not in inits


@pytest.mark.parametrize("change,word", [
    (lambda c: c.update(bogus=1), "bogus"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c["embedding"]["bigram"].pop("mul_prev"), "mul_prev"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda c: c["embedding"].update(scale=2.0), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(window=3), "window"),
    (lambda c: c["layers"][0].update(type="delta"), "delta"),
    (lambda c: c["layers"][0].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "glu"),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=7), "rot_dim"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6), "dims"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"].update(scale=0.0), "scale"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][1]["mlp"].update(shared={"ff": 3}), "shared"),
    (lambda c: c["layers"][3].update(weights_of=9), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=3), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=2), "weights_of"),
    (lambda c: c["layers"][3]["mixer"].update(heads=4), "weights_of"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_config_errors_name_the_key(change, word):
    c = copy.deepcopy(TB.BA_A)
    change(c)
    with pytest.raises(ConfigError) as e:
        model_from_config(c)
    assert word in str(e.value)


def test_weights_of_may_lead_on():
    c = copy.deepcopy(TB.BA_A)
    c["layers"].append(dict(copy.deepcopy(c["layers"][3]), weights_of=3))
    _, spec = model_from_config(c)
    assert spec.schedule[5].layer == spec.schedule[1].layer and spec.schedule[5].cache == 5


@pytest.mark.parametrize("name", sorted(TB.TINY))
def test_cache_needs_follow_the_mixers(name):
    raw = TB.TINY[name][0]
    _, spec = model_from_config(raw)
    needs = cache_needs(spec)
    assert len(needs) == len(raw["layers"]) + 1 and needs[-1] == StateNeed((1,))       # (the token before)
    for layer, need in zip(raw["layers"], needs):
        m = layer["mixer"]
        if layer["type"] == "wkv":
            assert need == (StateNeed((m["heads"], m["dim"], m["dim"])), StateNeed((raw["width"],)))
        else:
            n = m["kv_rank"] + m["rot_dim"]
            assert isinstance(need, KVNeed) and need.values_in_keys and need.planes == 1 and need.window is None
            assert need.n_kv_heads == 1 and n <= need.head_dim < n + 256 and need.head_dim % 64 == 0


def test_a_cache_of_one_plane():
    needs = [KVNeed(1, 64, values_in_keys=True), KVNeed(1, 64), KVNeed(1, 64, values_in_keys=True)]
    c = SequenceCache(needs, max_tokens=256, n_slots=2, dtype=torch.float32, device="cpu")
    assert len(c.groups) == 2 and c.kv_view(0)[0].shape == (4, 1, 1, 64, 64) and c.kv_view(1)[0].shape == (4, 2, 1, 64, 64)
    assert c.kv_bytes_per_token() == (1 + 2 + 1) * 64 * 4
    one = SequenceCache.bytes_needed(needs[:1], 256, 2, torch.float32)
    two = SequenceCache.bytes_needed(needs[1:2], 256, 2, torch.float32)
    assert two - one == 4 * 64 * 64 * 4


# ------------------------------------------------------------------------------------------- the plain implementation
def test_the_plain_recurrence_is_the_sum_it_stands_for():
    g = torch.Generator().manual_seed(1)
    T, d, dv = 9, 4, 3
    r, k = torch.randn(T, d, generator=g, dtype=F64), torch.randn(T, d, generator=g, dtype=F64)
    v, u = torch.randn(T, dv, generator=g, dtype=F64), torch.randn(d, generator=g, dtype=F64)
    w = torch.rand(T, d, generator=g, dtype=F64)
    got = PB.wkv_head(r, k, v, w, u)
    for t in range(T):
        want = float((r[t] * u * k[t]).sum()) * v[t]
        for s in range(t):
            want = want + float((r[t] * k[s] * w[s + 1:t].prod(dim=0)).sum()) * v[s]
        assert torch.allclose(got[t], want, atol=1e-12)


def test_the_plain_token_mix_and_pair_rows():
    h = torch.arange(12, dtype=F64).view(4, 3)
    mu = torch.tensor([0.0, 1.0, 0.5], dtype=F64)
    m = PB.token_mix(h, mu)
    assert torch.equal(m[0], h[0] * (1 - mu)) and torch.equal(m[2, 1], h[1, 1]) and torch.equal(m[:, 0], h[:, 0])
    assert PB.bigram_rows([4, 9, 9], 10, 3, 2) == [10, (4 * 3 + 18) % 10, (27 + 18) % 10]
    assert PB.bigram_rows([1], 1, 5, 5) == [1]


@pytest.mark.parametrize("interleaved", [False, True])
def test_the_plain_rotation_turns_pairs_and_scores_depend_on_the_distance(interleaved):
    g = torch.Generator().manual_seed(2)
    rot = {"base": 100.0, "dims": 6}
    x = torch.randn(1, 1, 6, generator=g, dtype=F64).expand(9, 1, 6).contiguous()
    y = PB.rotate(x, rot, interleaved)[:, 0]
    a, b = (0, 1) if interleaved else (0, 3)
    assert torch.equal(y[0], x[0, 0]) and abs(float(y[1, a]) - float(x[0, 0, a] * math.cos(1.0) - x[0, 0, b] * math.sin(1.0))) < 1e-12
    assert torch.allclose(y.norm(dim=1), x[:, 0].norm(dim=1))
    for n in (1, 3):
        assert torch.allclose((y[n:] * y[:-n]).sum(1), (y[n] * y[0]).sum().expand(9 - n))
    f, mult = PB.frequencies(dict(rot, scaling={"factor": 4.0, "original": 64, "fast": 32.0, "slow": 1.0}))
    plain, one = PB.frequencies(rot)
    assert one == 1.0 and abs(mult - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    assert all(p / 4.0 - 1e-15 <= q <= p + 1e-15 for p, q in zip(plain, f))


def test_absorbed_latent_attention_is_the_same_function():
    """what the kernels compute: scores of W_uk^T q against the latent itself, W_uv after the weighted sum of latents"""
    g = torch.Generator().manual_seed(3)
    c = TB.BA_A["layers"][2]["mixer"]
    H, d, r, dv, qr, kr, W, T = 3, 12, 4, 20, 16, 24, 64, 7
    shapes = {"dq": (qr, W), "dq.norm": (qr,), "uq": (H * (d + r), qr), "dkv": (kr + r, W), "dkv.norm": (kr,), "uk": (H * d, kr),
              "uv": (H * dv, kr)}
    t = {"m." + n: torch.randn(*s, generator=g, dtype=F64) for n, s in shapes.items()}
    h = torch.randn(T, W, generator=g, dtype=F64)
    want = PB.latent_attention(t, "m.", c, h, 1e-5, True)
    lat = PB.rms((h @ t["m.dkv"].T)[:, :kr], 1e-5) * t["m.dkv.norm"]
    k_rot = PB.rotate((h @ t["m.dkv"].T)[:, None, kr:], c["rot"], True)[:, 0]
    q = ((PB.rms(h @ t["m.dq"].T, 1e-5) * t["m.dq.norm"]) @ t["m.uq"].T).view(T, H, d + r)
    q_rot = PB.rotate(q[:, :, d:], c["rot"], True)
    for a in range(H):
        qa = torch.cat([q[:, a, :d] @ t["m.uk"].view(H, d, kr)[a], q_rot[:, a]], dim=1)
        o = PB.causal_attention(qa, torch.cat([lat, k_rot], dim=1), lat, c["scale"])
        assert torch.allclose(o @ t["m.uv"].view(H, dv, kr)[a].T, want[:, a], atol=1e-10)


def test_the_plain_router_weighs_its_picks_alone():
    idx, w = PB.route(torch.tensor([0.0, 3.0, -1.0, 2.0], dtype=F64), 2)
    assert idx == [1, 3] and abs(sum(w) - 1.0) < 1e-12 and abs(w[0] / w[1] - math.e) < 1e-12


def test_the_planted_token_matters(tmp_path):
    """on the plain model: with the needle gone the last probe's logits move by far more than any tolerance of the GPU tests
    - in every configuration, and in one with each mixer alone"""
    alone = {"lat1": TB._config(97, 64, 1e-5, (11, 3, 5), [TB._lat(1, 4, 16, 8, 16, 24, 32)]),
             "lat2": TB._config(97, 64, 1e-5, (11, 3, 5), [TB._lat(2, 1, 16, 8, 16, 24, 32)]),
             "wkv": TB._config(97, 64, 1e-5, (11, 3, 5), [TB._wkv(2, 16)])}
    try:
        for k, (n, c) in enumerate(alone.items()):
            TB.TINY[n] = (c, 70 + k)
        for name in sorted(TB.TINY):
            raw = TB.TINY[name][0]
            folder = TB.make_model(tmp_path, name, "float32")
            cfg, w = PB.load_model(folder)
            toks = TB.needle_request(raw["vocab"], 16, 2, [14, 15], random.Random(1))
            other = list(toks)
            other[2] = 7
            a, b = PB.logits(cfg, w, toks).numpy(), PB.logits(cfg, w, other).numpy()
            assert tiny.rel_err(a[14:], b[14:]) > 0.2, (name, tiny.rel_err(a[14:], b[14:]))
    finally:
        for n in alone:
            TB.TINY.pop(n, None)


# ------------------------------------------------------------------------------------------- the tests' own sharpness
_ORIGINAL = {n: getattr(PB, n) for n in ("bigram_rows", "wkv_head", "rotate", "route", "norm", "rms", "frequencies", "decay")}
MISTAKES = {
    "first token's row of the pair table": ("bigram_rows", lambda t, b, p, c: [0] + _ORIGINAL["bigram_rows"](t, b, p, c)[1:]),
    "multipliers swapped": ("bigram_rows", lambda t, b, p, c: _ORIGINAL["bigram_rows"](t, b, c, p)),
    "no row before": ("shifted", lambda h: torch.zeros_like(h)),
    "no bonus": ("wkv_head", lambda r, k, v, w, u: _ORIGINAL["wkv_head"](r, k, v, w, torch.ones_like(u))),
    "decay of the token before": ("wkv_head", lambda r, k, v, w, u: _ORIGINAL["wkv_head"](
        r, k, v, torch.cat([torch.ones_like(w[:1]), w[:-1]]), u)),
    "decay without its projection": ("decay", lambda t, p, m: torch.exp(-torch.exp(
        t[p + "w0"].double())).expand(m.shape[0], -1)),
    "the other pairing": ("rotate", lambda x, rot, il: _ORIGINAL["rotate"](x, rot, not il)),
    "frequencies not stretched": ("frequencies", lambda rot: _ORIGINAL["frequencies"](
        {k: v for k, v in rot.items() if k != "scaling"})),
    "no gate on the heads": ("head_gate", lambda t, p, h, o: o),
    "picks weighted alike": ("route", lambda z, top: (_ORIGINAL["route"](z, top)[0], [1.0 / top] * top)),
    "gains without one": ("norm", lambda x, w, eps: PB.rms(x, eps) * w),
    "a page of keys lost": ("causal_attention", None),
}


def _lossy_attention(q, k, v, scale):
    """the keys of positions 64 to 127 are not there for later pages' queries"""
    T = q.shape[0]
    out = torch.zeros((T, v.shape[1]), dtype=F64)
    for i in range(T):
        keep = [j for j in range(i + 1) if not (64 <= j < 128 and i >= 128)]
        s = (k[keep] @ q[i]) * scale
        out[i] = torch.softmax(s, dim=0) @ v[keep]
    return out


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_a_mistake_shows_in_the_test_models(tmp_path, monkeypatch, mistake):
    """a mistake planted in the plain implementation moves the logits of a test model's requests far beyond the 32-bit
    tolerance of the GPU tests"""
    raw = TB.TINY["B"][0]
    folder = TB.make_model(tmp_path, "B", "float32")
    cfg, w = PB.load_model(folder)
    toks = TB.needle_request(raw["vocab"], 160, 95, [96, 97, 120, 149, 150, 151], random.Random(4))
    good = PB.logits(cfg, w, toks).numpy()
    name, wrong = MISTAKES[mistake]
    monkeypatch.setattr(PB, name, wrong or _lossy_attention)
    bad = PB.logits(cfg, w, toks).numpy()
    moved = np.max(np.abs(good - bad)) / np.max(np.abs(good))
    assert moved > 0.02, (mistake, moved)
