"""Tedulorn configurations drawn at random (sizes that are no multiples of anything in particular, layers in any
number and order whose sizes differ from one another, windows and kept starts in every relation to one another and
to the page), each replayed in a mixed trace, in portions and with a decoded tail against the plain implementation:
what a particular choice of sizes would hide, another one shows."""

import functools
import random

import pytest

from replay_util import collect, random_tokens, trace_mixed, trace_portions, trace_tail
from tedulorn_models import attention, dense, model, moe, retention, rot, without_choice, write_model
from test_tedulorn_gpu import DTYPES, assert_rows_match, replay

pytestmark = pytest.mark.gpu


def draw_config(seed: int) -> dict:
    rng = random.Random(seed)
    width = rng.choice([8, 12, 25, 32, 50, 64, 96, 99, 160, 200, 256])
    mixing = (rng.choice([1, 1, 2, 3, 4]), rng.choice([8, 16, 20, 32, 64, 128, 40]))      # kv heads and value width of layers that mix

    def feed_forward():
        kind = rng.random()
        if kind < 0.15:
            return None
        if kind < 0.45:
            return dense(rng.choice([8, 24, 30, 64, 13, 128, 200]))
        count = rng.choice([1, 1, 2, 3, 4])
        experts = count * rng.choice([1, 2, 3, 5])
        keep = rng.randint(1, count)
        return moe(experts, rng.randint(1, min(keep * (experts // count), 6)), count, keep, rng.choice([8, 24, 30, 64, 13, 128]),
                   rng.choice([0.6, 1.5, 7.0]), rng.choice([8, 24, 30, 64, 13, 128]), rng.choice([0.6, 1.5, 7.0]))

    def rotation(dim):
        even = [d for d in (2, 4, 6, 8, 16, 20, 32, 64, 128, dim) if d <= dim and d % 2 == 0]
        return rot(rng.choice([20.0, 500.0, 10000.0, 300000.0]), rng.choice(even))

    def layer():
        dim = rng.choice([8, 16, 24, 32, 64, 128, 20, 96, 10, 33])
        if rng.random() < 0.4:
            heads = rng.choice([1, 1, 2, 3, 5])
            return retention(heads, dim, rng.choice([dim, 8, 16, 20, 32, 64, 130, 7]), rotation(dim),
                             [rng.choice([0.3, 0.9, 0.97, 0.99, 0.998, 0.9995, 1.0]) for _ in range(heads)], feed_forward())
        v_mix = rng.random() < 0.6
        kv, vdim = mixing if v_mix else (rng.choice([1, 1, 2, 3, 4]), rng.choice([dim, dim, 8, 16, 20, 32, 64, 128, 40]))
        if v_mix and rng.random() < 0.4:
            dim = vdim
        return attention(kv * rng.choice([1, 2, 3, 4, 6, 8, 17]), kv, dim, vdim, rng.choice([1, 3, 8, 17, 40, 64, 100]),
                         rng.choice([0, 0, 1, 4, 16, 20, 33, 70]), rotation(dim), rng.uniform(0.05, 0.4), v_mix, feed_forward())

    return model(rng.randint(50, 700), width, rng.choice([1e-5, 1e-6]), rng.choice([0, 4, 8, 13, 24, 64]),
                 [layer() for _ in range(rng.randint(1, 5))], embedding_scale=rng.choice([1.0, 0.5, 6.0]))


@pytest.mark.parametrize("seed,dtype", [(s, "float32") for s in range(20)] + [(s, "bfloat16") for s in range(100, 116)])
def test_a_configuration_drawn_at_random(tmp_path, cuda_device, seed, dtype):
    drawn = draw_config(seed)
    # bfloat16 models take every expert: a choice between close logits is float32's to test
    config = drawn if dtype == "float32" else without_choice(drawn)
    folder = write_model(tmp_path / "model", config, seed=seed, dtype=DTYPES[dtype])
    rng = random.Random(seed + 1)
    requests = {f"r{i}": random_tokens(config["vocab"], rng.randint(1, 170), seed=seed * 10 + i) for i in range(6)}
    for build in (trace_mixed, trace_portions, functools.partial(trace_tail, tail=40)):
        steps = build(requests)
        rows = collect(steps, replay(folder, dtype, steps, page_size=rng.choice([16, 32, 64])))
        assert_rows_match(rows, requests, folder, dtype, f"seed {seed} {getattr(build, '__name__', 'trace_tail')}", least=0.3)
