"""Lilulix models whose every size, option and order of layers is drawn at random, through the engine against the plain
implementation: in float32 in every schedule, in bfloat16 against the roundings the plain implementation makes itself."""
import random

import pytest
import torch

import lilulix_cases as LC
from helpers import random_tokens
from test_gpu_model import run_batches

pytestmark = pytest.mark.gpu


def random_config(rng):
    layers = []
    for _ in range(rng.randint(2, 5)):
        ff = rng.choice([None, 64, 100, 256, 47])
        if rng.random() < 0.5:
            dim, turned = rng.choice([16, 32, 48, 64, 10]), rng.choice([2, 8, 16, 32, 64, 6])
            layers.append(LC._lat(rng.choice([1, 2, 3, 4, 6, 17]), dim, turned, rng.choice([16, 32, 64, 24, 9]),
                                  rng.choice([16, 32, 64, 96, 120, 33, 200]), rng.choice([(dim + turned) ** -0.5, 0.1]),
                                  rng.choice([10000.0, 300000.0, 50.0]), ff))
        else:
            G = rng.choice([1, 2, 3])
            dim = rng.choice([16, 32, 64, 128, 48, 20, 7])
            layers.append(LC._att(G * rng.choice([1, 2, 3, 4, 8]), G, dim, rng.choice([dim ** -0.5, 0.1, 0.3]), ff))
    n = len(layers)
    start = rng.randrange(n)
    loop = rng.choice([None, (start, rng.randint(start + 1, n), rng.choice([1, 2, 3]))])
    return LC._model(rng.choice([300, 500, 257]), rng.choice([96, 128, 200, 100, 77]), rng.choice([1e-5, 1e-6]),
                     (rng.choice([1, 2, 101, 1024, 40009]), rng.choice([0, 1, 37, 1000003]), rng.choice([1, 19, 998244353])),
                     loop, layers)


@pytest.mark.parametrize("seed", list(range(12)))
def test_a_random_model_in_every_schedule_in_float32(seed):
    """Whole prompts, a prompt of 120 tokens then token by token, and two unequal batches in slots used again."""
    rng = random.Random(700 + seed)
    eng, cfg, w = LC.build(random_config(rng), seed, "float32")
    plain = LC.plain(cfg, w, "float32", wide=True)
    reqs = [random_tokens(n, cfg["vocab"], 900 + n + seed) for n in (1, 37, 150, 230)]
    want = [plain.forward(r) for r in reqs]

    def close(got, wl, what):
        err = LC.row_errors(got, wl)
        assert torch.isfinite(err).all() and err.max().item() < 2e-4 and err.median().item() < 2e-5, \
            f"{what}: row {int(err.argmax())} differs by {err.max().item():.3g}, median {err.median().item():.3g}"

    for r, wl in zip(reqs, want):
        s = eng.alloc_slot()
        got = eng.step([(s, r)], [list(range(len(r)))]).clone()
        eng.free_slot(s)
        close(got, wl, f"whole {len(r)}")
    r, wl = reqs[3], want[3]
    s = eng.alloc_slot()
    rows = [eng.step([(s, r[:120])], [list(range(120))]).clone()] + [eng.step([(s, [t])]).clone() for t in r[120:]]
    eng.free_slot(s)
    close(torch.cat(rows), wl, "decode")
    got = run_batches(eng, reqs, [[3, 0, 2], [1, 2, 3]], [1, 30, 100, 200])
    for i, wl in enumerate(want):
        close(got[i], wl, f"batched {i}")
    eng.cache.slots.check()


@pytest.mark.parametrize("seed", list(range(12)))
def test_a_random_model_in_bfloat16_errs_as_the_roundings_do(seed):
    """The distance from float64, row by row: half of the rows and nine in ten are no further than one and a half times the
    plain implementation's with the same roundings, in a prompt and in tokens decoded behind it."""
    rng = random.Random(700 + seed)
    eng, cfg, w = LC.build(random_config(rng), seed, "bfloat16")
    exact, rounded = LC.plain(cfg, w, "float32", wide=True), LC.plain(cfg, w, "bfloat16")
    r = random_tokens(180, cfg["vocab"], 77 + seed)
    ref = exact.forward(r)
    base = LC.row_errors(rounded.forward(r), ref)
    s = eng.alloc_slot()
    rows = [eng.step([(s, r[:110])], [list(range(110))]).clone()] + [eng.step([(s, [t])]).clone() for t in r[110:]]
    eng.free_slot(s)
    err = LC.row_errors(torch.cat(rows), ref)
    assert torch.isfinite(err).all()
    for part in (slice(0, 110), slice(110, 180)):
        for q in (0.5, 0.9):
            assert err[part].quantile(q) < 1.5 * base[part].quantile(q) + 2e-3, \
                f"{part}, quantile {q}: {err[part].quantile(q):.3g} against {base[part].quantile(q):.3g}"
