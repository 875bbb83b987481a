"""Small Basitar configurations with seeded random weights for the tests, with one token that stands out.

The configurations differ in every size and option: the order of the mixers, head counts (one to more than a tile of the
attention kernels), latents whose cached vector fills each of the sizes the tensor-core kernels take and sizes nothing takes,
values wider and narrower than keys, both pairings with and without stretched frequencies, recurrences with heads from ten to
128 channels, layers that run another layer's weights, dense feed-forwards, experts (one pick and several) and none, pair
tables of one bucket and of many, with multipliers of zero and below.
"""
from __future__ import annotations

import json
import os
import random
from typing import List

NEEDLE, PROBE = 3, 4            # token ids: the needle stands out for every probe
CODE = 3.0                      # the size of the planted embedding features, far above the random ones
KEPT = 2                        # the stream's first columns keep the token's own features through all layers


def _ff(ff):
    """None, the inner size of a dense feed-forward, or (experts, top, inner size)"""
    if ff is None:
        return None
    if isinstance(ff, int):
        return {"kind": "dense", "ff": ff}
    return {"kind": "moe", "expert": {"ff": ff[2]}, "router": {"experts": ff[0], "top": ff[1]}}


def _lat(kind, heads, dim, rot, vdim, q_rank, kv_rank, ff=None, base=10000.0, scaling=None, scale=None):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention" if kind == 1 else "latent_attention_2",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale if scale is not None else (dim + rot) ** -0.5, "rot": r}, "mlp": _ff(ff)}


def _wkv(heads, dim, ff=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": _ff(ff)}


def _again(layers, j):
    layers.append(dict(json.loads(json.dumps(layers[j])), weights_of=j))
    return layers


def _config(vocab, width, eps, bigram, layers, max_positions=700):
    return {"architecture": "Basitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "max_positions": max_positions,
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers}


# A: small everything; both attentions, a recurrence, two layers with another's weights, a layer without a feed-forward
BA_A = _config(211, 64, 1e-5, (97, 31, 5), _again(_again([
    _lat(1, 4, 16, 8, 24, 24, 40, 48), _wkv(2, 16, (5, 2, 24)),
    _lat(2, 3, 12, 4, 20, 16, 24, None, 500000.0, (4.0, 64, 32.0, 1.0))], 1), 0))
# B: cached vectors of 176 (kept as 192) and of 128 exactly; a decode step's grouped product (heads x dim = 128); frequencies
#    stretched in both kinds
BA_B = _config(300, 128, 1e-6, (509, 131, 17), _again([
    _wkv(4, 32, (6, 3, 40)), _lat(2, 5, 48, 32, 64, 48, 144, (6, 3, 40), 30000.0, (8.0, 256, 16.0, 2.0)),
    _lat(1, 8, 32, 32, 24, 56, 96, 96, 100000.0, (2.0, 128, 32.0, 1.0))], 0))
# C: a cached vector of 224 (kept as 256) with values beyond 128, more heads than one tile of the decode kernel, a width that is
#    no multiple of 64, heads of 128 channels, the plain frequencies in the gated kind
BA_C = _config(257, 200, 2e-6, (1, 3, 2), [
    _lat(2, 20, 24, 24, 16, 40, 200, 72), _wkv(1, 128, (9, 4, 32)), _lat(1, 2, 40, 24, 80, 72, 30, (4, 4, 16))])
# D: sizes that no vector load or tensor-core tile takes; rotations of one pair; one pick of the router; multipliers of zero
#    and below
BA_D = _config(131, 72, 1e-5, (7, 0, -3), _again([
    _wkv(3, 10, 20), _lat(1, 3, 5, 2, 7, 13, 19, (3, 1, 12)), _lat(2, 5, 9, 2, 11, 9, 12, 36, 100.0)], 2))
# E: cached vectors of 304 (kept as 320) and of 576 exactly (values of 512 elements), 48 heads, heads of 64 channels
BA_E = _config(401, 160, 1e-5, (1009, 127, 3), [
    _lat(1, 48, 16, 48, 16, 64, 256, 64), _wkv(2, 64, (8, 2, 24)), _lat(2, 4, 32, 64, 40, 96, 512, (5, 3, 40), 500000.0)])
RANKS = {"B": 40, "C": 24, "D": 5}                    # the decay's projection (16 elsewhere): sizes that come from the tensors alone
TINY = {"A": (BA_A, 51), "B": (BA_B, 52), "C": (BA_C, 53), "D": (BA_D, 54), "E": (BA_E, 55)}


def plant(cfg: dict, t: dict, seed: int) -> None:
    """random weights made sharp, in place.

    The needle's embedding row has one large feature (column 0), a probe's another (column 1); the pair table, the positions and
    the branches leave those columns alone. Latent attention: the key/value latent's first element reads column 0, the query
    latent's first element column 1, and far above the random weights; even heads' plain keys and queries read those elements,
    odd heads' rotated parts read column 0 and the query latent's element into the pair that turns slowest. Values read the
    latent's first element. Time mixing: the first head's last key channel reads column 0, its r column 1, and that channel
    decays slowly; r is correlated with k, so that a token's own score is not a small difference of large numbers. Gains,
    mixing weights and biases are drawn large enough to matter, routers sharp enough that a pick is rarely a close call."""
    import torch
    g = torch.Generator().manual_seed(seed + 1)

    def randn(*shape):
        return torch.randn(*shape, generator=g)
    W = cfg["width"]
    for n in ("embed", "bigram", "pos"):
        t[n] = randn(*t[n].shape) * {"embed": 1.0, "bigram": 0.6, "pos": 0.3}[n]
        t[n][:, :KEPT] = 0.0
    t["embed"][NEEDLE, 0] = CODE * W ** 0.5 / 4
    t["embed"][PROBE, 1] = CODE * W ** 0.5 / 4
    for n in sorted(t):
        if n.endswith(("norm1", "norm2", "norm1b", "norm2b", "final.norm")):
            t[n] = 0.2 * randn(*t[n].shape)
        elif n.endswith("norm"):
            t[n] = 1.0 + 0.2 * randn(*t[n].shape)
        elif n.endswith("router"):
            t[n] = 2.5 * randn(*t[n].shape) / W ** 0.5
        elif n.endswith("router.b"):
            t[n] = randn(*t[n].shape)
        elif ".mu." in n:
            t[n] = 0.5 + 0.5 * randn(*t[n].shape)
            t[n][:KEPT] = 0.0
        elif t[n].dim() == 2 and n not in ("embed", "bigram", "pos"):
            t[n] = randn(*t[n].shape) / t[n].shape[1] ** 0.5
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, p = layer["mixer"], "l%d.mix." % i
        if layer["type"] == "wkv":
            d = m["dim"]
            t[p + "r"] = 0.8 * t[p + "k"] + 0.4 * t[p + "r"]
            for n, col in (("k", 0), ("r", 1)):
                t[p + n][d - 1, :] = 0.0
                t[p + n][d - 1, col] = 4.0
            t[p + "v"][:, 0] = torch.sign(t[p + "v"][:, 5])
            t[p + "w0"] = -2.5 + randn(*t[p + "w0"].shape)
            t[p + "w2"] *= 2.0
            t[p + "w0"][d - 1] = -6.5
            t[p + "w2"][d - 1] = 0.0
            t[p + "u"] = 0.7 * randn(*t[p + "u"].shape)
            continue
        H, d, r, qr, kr = m["heads"], m["dim"], m["rot_dim"], m["q_rank"], m["kv_rank"]
        slow = r // 2 - 1 if layer["type"] == "latent_attention" else r - 2
        t[p + "dq"][0] = 0.0
        t[p + "dq"][0, 1] = 6.0
        t[p + "dkv"][0] = 0.0
        t[p + "dkv"][0, 0] = 6.0
        t[p + "dkv"][kr + slow, 0] = 5.0 / W ** 0.5
        for h in range(H):
            q = t[p + "uq"].view(H, d + r, qr)[h]
            q[0] = 0.0
            if h % 2 == 0 or r == 2:                         # (a single pair turns too fast to rest a far key on)
                q[0, 0] = 3.5 * (qr * m["scale"]) ** -0.5
                t[p + "uk"].view(H, d, kr)[h, 0] = 0.0
                t[p + "uk"].view(H, d, kr)[h, 0, 0] = 4.0 * (kr * m["scale"]) ** -0.5
            else:
                q[d + slow] = 0.0
                q[d + slow, 0] = 5.0 / (m["scale"] * qr ** 0.5)
        t[p + "uv"][:, 0] = torch.sign(t[p + "uv"][:, 1])
    for n in list(t):
        if n.endswith((".mix.o", ".down")):
            t[n][:KEPT] = 0.0


def make_model(tmp_path, name: str, dtype: str = "bfloat16") -> str:
    """a model folder with the configuration's planted random weights (``plant``)"""
    import torch
    from kindi_b200.config.registry import model_from_config
    from kindi_b200.parts.model import expected_tensors, tensor_inits
    from kindi_b200.weights.random_init import random_tensors
    from kindi_b200.weights.safetensors_io import write_file
    cfg, seed = TINY[name]
    cfg = json.loads(json.dumps(cfg))
    d = os.path.join(str(tmp_path), "ba_%s_%s" % (name, dtype))
    if os.path.isfile(os.path.join(d, "model.safetensors")):
        return d
    os.makedirs(d, exist_ok=True)
    _, spec = model_from_config(cfg)
    shapes = expected_tensors(spec)
    for n, s in shapes.items():
        if n.endswith(".mix.w1") and name in RANKS:
            shapes[n] = (RANKS[name], s[1])
        elif n.endswith(".mix.w2") and name in RANKS:
            shapes[n] = (s[0], RANKS[name])
    t = random_tensors(shapes, seed, dtype=torch.float32, inits=tensor_inits(spec))
    plant(cfg, t, seed)
    tdt = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype]
    t = {n: v.to(tdt).contiguous() for n, v in t.items()}
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_file(os.path.join(d, "model.safetensors"), t, metadata={"format": "pt"})
    return d


def needle_request(vocab: int, length: int, needle_at: int, probes: List[int], rng: random.Random) -> List[int]:
    """random tokens (neither needle nor probe) with the needle at `needle_at` and probes at the listed places"""
    toks = []
    for i in range(length):
        t = rng.randrange(vocab)
        while t in (NEEDLE, PROBE):
            t = rng.randrange(vocab)
        toks.append(NEEDLE if i == needle_at else PROBE if i in probes else t)
    return toks


def edge_places(length: int) -> List[int]:
    """positions around the borders of the cache's pages (and the recurrence's runs) and of the pieces a run is cut into"""
    out = set()
    for s in (16, 64):
        for c in range(s, length, s):
            out |= {c - 1, c, c + 1}
    return sorted(p for p in out if 0 < p < length)
