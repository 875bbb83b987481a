"""Random Zebovik configurations - widths, layer orders, head counts, groups and sizes (also sizes no vector load takes),
chunks of any size or none, shared keys and values, caps of any strength, taps, states and norm parts, feed-forwards or none -
each against the plain implementation: whole prompts, their last tokens one by one, and all requests as one unequal batch, in
both dtypes."""
import random

import pytest

import tiny
import tiny_zebovik as TZ
import test_zebovik_gpu as T

pytestmark = pytest.mark.gpu


def random_config(rng: random.Random) -> dict:
    width = rng.choice([48, 64, 72, 96, 128, 136, 256])
    layers, owners = [], []
    for n in range(rng.randint(2, 5)):
        ff = rng.choice([None, 20, 40, 96, 200])
        kind = rng.choice(["att", "att", "mem", "ssd"])
        if kind == "att":
            chunk = rng.choice([None, 3, 31, 64, 70, 128, 500])
            cap = rng.choice([None, 5.0, 15.0, 30.0, 80.0])
            if owners and rng.random() < 0.4:
                o = rng.choice(owners)
                m = layers[o]["mixer"]
                layers.append(TZ._att(m["kv_heads"] * rng.choice([1, 2, 5]), m["kv_heads"], m["dim"], m["vdim"], chunk, cap,
                                      m["rot"]["base"], m["rot"]["dims"], ff, kv_from=o, scale=rng.choice([6.0, 10.0]) / m["dim"]))
                continue
            kv = rng.choice([1, 2, 3])
            dim = rng.choice([8, 10, 20, 32, 48, 64, 96, 128])
            vdim = rng.choice([dim, 8, 12, 40, 64, 100, 128])
            owners.append(n)
            layers.append(TZ._att(kv * rng.choice([1, 2, 4]), kv, dim, vdim, chunk, cap, rng.choice([10000.0, 250000.0]),
                                  rng.choice([0, 2, dim // 2 - dim // 2 % 2, dim - dim % 2]), ff))
        elif kind == "mem":
            layers.append(TZ._mem(rng.choice([1, 2, 5]), rng.choice([8, 10, 32, 48, 64, 100, 128]),
                                  rng.choice([4, 12, 32, 64, 72, 130]), rng.choice([3.0, 9.0, 15.0]), ff))
        else:
            groups = rng.choice([1, 2, 3])
            heads, vdim = groups * rng.choice([1, 2, 4]), rng.choice([3, 8, 16, 64, 80])
            parts = rng.choice([p for p in (1, 2, 3, 4) if heads * vdim % p == 0])
            layers.append(TZ._ssd(heads, vdim, rng.choice([5, 16, 24, 64, 128]), groups, rng.choice([1, 2, 3, 4, 8]), parts, ff))
    return TZ._config(rng.choice([97, 211, 512]), width, rng.choice([1e-6, 1e-5]), rng.choice([None, 8.0, 30.0]), layers)


SEEDS = [100, 103, 106, 109, 112, 115, 118, 121, 124, 127]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("k", range(len(SEEDS)))
def test_random_configuration(tmp_path, k, dtype):
    rng = random.Random(SEEDS[k])
    cfg = random_config(rng)
    name = "R%d" % k
    TZ.TINY[name] = (cfg, 600 + k)
    try:
        folder = TZ.make_model(tmp_path, name, dtype)
    finally:
        del TZ.TINY[name]
    reqs = T._edge_requests(cfg, seed=3, L=160)
    reqs = dict(list(reqs.items())[:4] + list(reqs.items())[-3:])
    want = T._plain(folder, reqs)
    steps = tiny.trace_whole(reqs)
    later = tiny.trace_last_n(reqs, 24)
    for s in later:
        s["step"] += len(steps)
    eng = T._engine(folder, steps + later, dtype)
    out = str(tmp_path / "out")
    tiny.run_replay(eng, steps, out)
    T._compare(tiny.collect(out, steps, cfg["vocab"]), reqs, want, T.TOL[dtype], "%s %s whole" % (name, dtype))
    tiny.run_replay(eng, later, out)
    T._compare(tiny.collect(out, later, cfg["vocab"]), reqs, want, T.TOL[dtype], "%s %s decoded" % (name, dtype))
    decode = {r: min(len(reqs[r]) - 1, rng.choice([0, 3, 9])) for r in reqs}
    group = tiny.trace_group(reqs, decode)
    eng = T._engine(folder, group, dtype)
    out = str(tmp_path / "batch")
    tiny.run_replay(eng, group, out)
    T._nothing_held(eng)
    T._compare(tiny.collect(out, group, cfg["vocab"]), reqs, want, T.TOL[dtype], "%s %s batch" % (name, dtype))
