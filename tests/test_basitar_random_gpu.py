"""Random Basitar configurations - widths, layer orders, head counts and sizes (also sizes no vector load takes), latents of any
rank, both rotations, stretched or not, layers that run another's weights, experts, dense feed-forwards or none, pair tables of
any size - each against the plain implementation: whole prompts, their last tokens one by one, and all requests as one unequal
batch, in both dtypes."""
import random

import pytest

import tiny
import tiny_basitar as TB
import test_basitar_gpu as T

pytestmark = pytest.mark.gpu


def random_config(rng: random.Random) -> dict:
    width = rng.choice([48, 64, 72, 96, 128, 136, 256])
    layers = []
    for n in range(rng.randint(2, 5)):
        ff = rng.choice([None, 20, 40, 96, (4, 2, 24), (7, 3, 16), (3, 3, 40), (10, 4, 20)])
        kind = rng.choice(["lat1", "lat2", "wkv", "wkv", "again"])
        if kind == "again" and layers:
            j = rng.randrange(len(layers))
            TB._again(layers, layers[j].get("weights_of", j))
        elif kind == "wkv":
            layers.append(TB._wkv(rng.choice([1, 2, 4, 5]), rng.choice([8, 10, 32, 48, 64, 100, 128]), ff))
        else:
            rot = rng.choice([2, 6, 8, 16, 32])
            scaling = rng.choice([None, (2.0, 64, 32.0, 1.0), (8.0, 40, 4.0, 0.5)])
            dim = rng.choice([5, 8, 16, 24, 40])
            layers.append(TB._lat(1 if kind == "lat1" else 2, rng.choice([1, 2, 5, 9, 18]), dim, rot, rng.choice([dim, 7, 16, 50]),
                                  rng.choice([9, 16, 40, 72]), rng.choice([12, 19, 30, 56, 100, 128, 150, 230]), ff,
                                  rng.choice([10000.0, 250000.0]), scaling, rng.choice([0.7, 1.0, 1.5]) * (dim + rot) ** -0.5))
    bigram = (rng.choice([1, 13, 211, 4096]), rng.choice([1, 31, 1009]), rng.choice([0, 1, 7]))
    return TB._config(rng.choice([97, 211, 512]), width, rng.choice([1e-6, 1e-5]), bigram, layers, rng.choice([160, 200, 3000]))


SEEDS = [200, 203, 206, 209, 212, 215, 218, 221, 224, 227]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("k", range(len(SEEDS)))
def test_random_configuration(tmp_path, k, dtype):
    rng = random.Random(SEEDS[k])
    cfg = random_config(rng)
    name = "R%d" % k
    TB.TINY[name] = (cfg, 700 + k)
    try:
        folder = TB.make_model(tmp_path, name, dtype)
    finally:
        del TB.TINY[name]
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
