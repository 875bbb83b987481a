"""The Basitar decoder: its config.json keys, its typed configuration and its ``ModelSpec``.

What the architecture is. ``x = embed[token] + bigram[(previous token * mul_prev + token * mul_cur) mod buckets] + pos[p]``
(the pair table's last row for a sequence's first token); a list of layers, each with a norm before and after every
sub-layer, ``x += norm1b(mixer(norm1(x)))``, then ``x += norm2b(ff(norm2(x)))``, all RMS norms whose gain is one plus the
stored weight; a final norm of the same kind and a head tied to the embedding table. ``layers[i].type`` names the layer's mixer:

* ``wkv``: time mixing with a decay per key channel and a bonus for the current token.
* ``latent_attention``: low-rank query and key/value latents with one rotated key part shared by the heads, rotated in
  pairs (i, i + rot_dim / 2).
* ``latent_attention_2``: the same with interleaved pairs, frequencies that may be stretched (``rot.scaling``), and an output
  gate ``sigmoid(W_g h)``, one number per head.

``weights_of: j``: the layer runs layer j's tensors with a cache of its own.

The feed-forward is dense (``mlp.kind`` = ``dense``: ``W_down (silu(W_gate h) * (W_up h))``) or a mixture of experts of that
form (``moe``: the router's ``top`` largest of ``experts`` logits, weighted by the softmax over the chosen ones); a layer may
have none (``mlp``: null).

config.json is nested: ``embedding.bigram.{buckets, mul_prev, mul_cur}``, ``layers[i] = {"type", "mixer": {...}, "mlp":
{...} | null, "weights_of"}``, ``norm.eps``, ``max_positions``, ``vocab``, ``width``. Tensors: ``embed``, ``bigram``, ``pos``,
``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``. Every size and
constant comes from the configuration; nothing here knows a particular model.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..config.model_config import ConfigError, ConfigReader
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


@dataclass(frozen=True)
class BasitarLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    scaling: Optional[Tuple[float, float, float, float]]        # factor, original, fast, slow


@dataclass(frozen=True)
class BasitarTimeMix:
    heads: int
    dim: int


@dataclass(frozen=True)
class BasitarExperts:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class BasitarLayer:
    kind: str                   # "wkv" | "latent_attention" | "latent_attention_2"
    mixer: Any
    ff: Any                     # None, an int (the dense feed-forward's inner size) or BasitarExperts
    weights_of: Optional[int] = None


@dataclass(frozen=True)
class BasitarConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    max_positions: int
    buckets: int
    mul_prev: int
    mul_cur: int
    layers: Tuple[BasitarLayer, ...]

    def to_dict(self) -> dict:
        """the config.json that reads back as this configuration"""
        layers = []
        for l in self.layers:
            m = l.mixer
            if l.kind == "wkv":
                mixer = {"heads": m.heads, "dim": m.dim}
            else:
                rot = {"base": m.rot_base, "dims": m.rot_dim}
                if m.scaling is not None:
                    rot["scaling"] = dict(zip(_SCALING, m.scaling))
                mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank,
                         "kv_rank": m.kv_rank, "scale": m.scale, "rot": rot}
            if l.ff is None:
                mlp = None
            elif isinstance(l.ff, int):
                mlp = {"kind": "dense", "ff": l.ff}
            else:
                mlp = {"kind": "moe", "expert": {"ff": l.ff.ff}, "router": {"experts": l.ff.experts, "top": l.ff.top}}
            entry = {"type": l.kind, "mixer": mixer, "mlp": mlp}
            if l.weights_of is not None:
                entry["weights_of"] = l.weights_of
            layers.append(entry)
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "max_positions": self.max_positions, "layers": layers,
                "embedding": {"bigram": {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}}}


_SCALING = ("factor", "original", "fast", "slow")


def _count(r: ConfigReader, key: str, where: str, *default) -> int:
    return int(_positive("%s.%s" % (where, key), r.integer(key, *default)))


def _positive(what: str, v):
    if not (v > 0):
        raise ConfigError("%s must be positive, found %r" % (what, v))
    return v


def _read_wkv(raw: Mapping[str, Any], where: str) -> BasitarTimeMix:
    r = ConfigReader(raw, where)
    m = BasitarTimeMix(_count(r, "heads", where), _count(r, "dim", where))
    r.finish(())
    return m


def _read_latent(raw: Mapping[str, Any], where: str) -> BasitarLatent:
    r = ConfigReader(raw, where)
    heads, dim = _count(r, "heads", where), _count(r, "dim", where)
    rot_dim = _count(r, "rot_dim", where)
    if rot_dim % 2:
        raise ConfigError("%s.rot_dim must be even, found %d" % (where, rot_dim))
    vdim, q_rank, kv_rank = _count(r, "vdim", where, dim), _count(r, "q_rank", where), _count(r, "kv_rank", where)
    scale = float(_positive(where + ".scale", r.number("scale", (dim + rot_dim) ** -0.5)))
    rr = ConfigReader(r.any("rot") or {}, where + ".rot")
    base = float(_positive(where + ".rot.base", rr.number("base", 10000.0)))
    dims = rr.integer("dims", rot_dim)
    if dims != rot_dim:
        raise ConfigError("%s.rot.dims is %d, the mixer's rotated part has rot_dim = %d" % (where, dims, rot_dim))
    scaling = None
    sraw = rr.any("scaling")
    if sraw is not None:
        s = ConfigReader(sraw, where + ".rot.scaling")
        scaling = tuple(float(_positive("%s.rot.scaling.%s" % (where, k), s.number(k))) for k in _SCALING)
        s.finish(())
    rr.finish(())
    r.finish(())
    return BasitarLatent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, scaling)


_MIXERS = {"wkv": _read_wkv, "latent_attention": _read_latent, "latent_attention_2": _read_latent}


def _read_mlp(raw: Optional[Mapping[str, Any]], where: str):
    if raw is None:
        return None
    fr = ConfigReader(raw, where)
    kind = fr.string("kind", "dense")
    if kind == "dense":
        ff = _count(fr, "ff", where)
        fr.finish(())
        return ff
    if kind != "moe":
        raise ConfigError("%s: kind %r is not a feed-forward of this architecture (dense, moe)" % (where, kind))
    er = ConfigReader(fr.any("expert") or {}, where + ".expert")
    ff = _count(er, "ff", where + ".expert")
    er.finish(())
    rr = ConfigReader(fr.any("router") or {}, where + ".router")
    experts, top = _count(rr, "experts", where + ".router"), _count(rr, "top", where + ".router")
    rr.finish(())
    fr.finish(())
    if top > experts:
        raise ConfigError("%s.router.top = %d exceeds the %d experts" % (where, top, experts))
    return BasitarExperts(experts, top, ff)


def read_config(raw: Mapping[str, Any]) -> BasitarConfig:
    r = ConfigReader(raw)
    where = "config.json"
    arch = r.string("architecture")
    vocab, width = _count(r, "vocab", where), _count(r, "width", where)
    max_positions = _count(r, "max_positions", where)
    norm = ConfigReader(r.any("norm") or {}, "config.json: norm")
    eps = float(_positive("config.json: norm.eps", norm.number("eps")))
    norm.finish(())
    emb = ConfigReader(r.any("embedding") or {}, "config.json: embedding")
    big = ConfigReader(emb.any("bigram") or {}, "config.json: embedding.bigram")
    buckets = _count(big, "buckets", "config.json: embedding.bigram")
    mul_prev, mul_cur = big.integer("mul_prev"), big.integer("mul_cur")
    big.finish(())
    emb.finish(())
    lraw = r.any("layers")
    if not isinstance(lraw, (list, tuple)) or not lraw:
        raise ConfigError("config.json: layers must be a non-empty list")
    layers = []
    for i, l in enumerate(lraw):
        where = "config.json: layers[%d]" % i
        lr = ConfigReader(l, where)
        kind = lr.string("type")
        if kind not in _MIXERS:
            raise ConfigError("%s: type %r is not a mixer of this architecture (%s)" % (where, kind, ", ".join(_MIXERS)))
        mixer = _MIXERS[kind](lr.any("mixer") or {}, where + ".mixer")
        ff = _read_mlp(lr.any("mlp"), where + ".mlp")
        layers.append(BasitarLayer(kind, mixer, ff, lr.integer("weights_of", None)))
        lr.finish(())
    r.finish()
    cfg = BasitarConfig(arch, vocab, width, eps, max_positions, buckets, mul_prev, mul_cur, tuple(layers))
    for i in range(len(layers)):
        owner(cfg, i)
    return cfg


def owner(cfg: BasitarConfig, i: int) -> int:
    """the layer whose tensors layer i runs; an error where that is no layer, or one of another shape"""
    j, seen = i, {i}
    while cfg.layers[j].weights_of is not None:
        j = cfg.layers[j].weights_of
        if not (0 <= j < len(cfg.layers)) or j in seen:
            raise ConfigError("config.json: layers[%d].weights_of does not lead to a layer with tensors of its own" % i)
        seen.add(j)
    a, b = cfg.layers[i], cfg.layers[j]
    if (a.kind, a.mixer, a.ff) != (b.kind, b.mixer, b.ff):
        raise ConfigError("config.json: layers[%d] has the weights_of layer %d, but another mixer or feed-forward" % (i, j))
    return j


EMBEDDING, PAIRS, POSITIONS, FINAL_NORM = "embed", "bigram", "pos", "final.norm"


def _mixer_part(l: BasitarLayer, eps: float) -> PartSpec:
    m = l.mixer
    if l.kind == "wkv":
        return PartSpec("wkv", {"n_heads": m.heads, "head_dim": m.dim, "eps": eps})
    gated = l.kind == "latent_attention_2"
    position = PartSpec("rotary", {"base": m.rot_base, "rotary_dim": m.rot_dim, "pairing": "interleaved" if gated else "half",
                                   "scaling": None if m.scaling is None else dict(zip(_SCALING, m.scaling))})
    return PartSpec("latent_attention", {
        "n_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_head_dim": m.vdim, "q_rank": m.q_rank,
        "kv_rank": m.kv_rank, "scale": m.scale, "eps": eps, "position": position, "head_gate": gated,
        "names": {"gate": "g" if gated else None}})


def _ff_part(l: BasitarLayer) -> Optional[PartSpec]:
    if l.ff is None:
        return None
    if isinstance(l.ff, int):
        return PartSpec("swiglu", {"intermediate": l.ff, "activation": "silu",
                                   "names": {"gate": "gate", "up": "up", "down": "down"}})
    return PartSpec("moe", {
        "n_experts": l.ff.experts, "top_k": l.ff.top, "intermediate": l.ff.ff, "gated": True, "activation": "silu",
        "score": "softmax", "router_bias": True,
        "names": {"router": "router", "router_bias": "router.b", "gate": "e%d.gate", "up": "e%d.up", "down": "e%d.down"}})


def build_spec(cfg: BasitarConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"eps": cfg.eps, "weight": "", "one_plus": True})
    layers, schedule, place = [], [], {}
    for i, l in enumerate(cfg.layers):
        if l.weights_of is None:
            place[i] = len(layers)
            layers.append(LayerSpec(PartSpec("sandwich", {
                "norm1": norm, "mixer": _mixer_part(l, cfg.eps), "norm1b": norm, "norm2": norm, "feed_forward": _ff_part(l),
                "norm2b": norm,
                "names": {"norm1": "norm1", "mixer": "mix.", "norm1b": "norm1b", "norm2": "norm2", "feed_forward": "mlp.",
                          "norm2b": "norm2b"}}), "l%d." % i))
    for i in range(len(cfg.layers)):
        schedule.append(ScheduleEntry(layer=place[owner(cfg, i)], cache=i))
    spec = ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, width=cfg.width, layers=tuple(layers),
        schedule=tuple(schedule), final_norm=norm, final_norm_prefix=FINAL_NORM,
        embedding=PartSpec("table", {
            "name": EMBEDDING, "vocab": cfg.vocab, "positions": {"name": POSITIONS, "count": cfg.max_positions},
            "pairs": {"name": PAIRS, "buckets": cfg.buckets, "mul_prev": cfg.mul_prev, "mul_cur": cfg.mul_cur}}),
        head=PartSpec("linear", {"tied_to": EMBEDDING, "vocab": cfg.vocab}), max_positions=cfg.max_positions,
        # a layer without a feed-forward has no use for its norms: a folder that stores them all the same is accepted
        may_ignore=tuple("l%d.%s" % (i, n) for i, l in enumerate(cfg.layers) if l.ff is None and l.weights_of is None
                         for n in ("norm2", "norm2b")))
    spec.validate()
    return spec


register_architecture("Basitar", build_spec, read_config)
