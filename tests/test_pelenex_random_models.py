"""Pelenex configurations drawn at random (every size, count, constant, rank and the order of layers from a seeded
generator; keys that may be absent are absent now and then) through the engine against the plain implementation: whole, the
last tokens one by one, prompts in portions and an unequal batch.  What the hand-made models happen not to combine shows
here: larger widths and heads, states of more rows than columns, windows around the requests' lengths, kept tokens beyond
the window, layers of one kind only.

The 32-bit comparison covers every position.  In bfloat16 only the positions before a router's first close call are held
against the plain implementation; every other configuration therefore takes every expert and is compared at every position
in bfloat16 too."""
import random

import pytest

import plain_pelenex as plain
from conftest import random_ids
from engine_drives import drive_batches, drive_portions, drive_tail_one_by_one, drive_whole
from pelenex_models import both, delta, dense, layer, mlstm, moe, write_model
from test_pelenex import compare, poison_states

pytestmark = pytest.mark.gpu


def draw_mlp(r: random.Random, every: bool):
    x = r.random()
    if x < 0.12:
        return None
    if x < 0.5:
        return dense(r.choice([24, 40, 64, 100, 136, 304]))
    experts = r.choice([1, 2, 3, 4, 5] if every else [1, 2, 3, 4, 6, 11, 17, 40])
    top = experts if every else r.randint(1, min(experts, 6))
    return moe(r.choice([24, 40, 64, 96, 136]), experts, top, r.choice([None, 16, 40, 72, 200]))


def draw_mixer(r: random.Random, kind: str):
    dims, vdims = [4, 8, 13, 16, 24, 32, 48, 64, 72, 96, 128, 160], [4, 8, 15, 16, 24, 32, 40, 64, 96, 128, 136]
    if kind == "mlstm":
        return mlstm(r.choice([1, 2, 3, 4]), r.choice(dims), r.choice(vdims), r.choice([3.0, 9.0, 15.0]))
    if kind == "channel_delta":
        g = r.choice([1, 1, 2, 3])
        return delta(g * r.choice([1, 1, 2, 3]), g, r.choice(dims), r.choice(vdims), r.choice([1, 2, 3, 4, 4, 6, 9]))
    dim, kv = r.choice([8, 12, 16, 24, 32, 48, 64, 96, 128]), r.choice([1, 1, 2, 3])
    mask = None
    if r.random() < 0.85:
        mask = (r.choice([1, 5, 31, 64, 65, 100, 128, 140, 200]), r.choice([None, 0, 1, 24, 64, 70, 150]))
    left = (kv * r.choice([1, 2, 4, 5]), kv, dim, round(dim ** -0.5 * r.choice([0.7, 1.0, 2.0]), 4), mask)
    return both(left, (r.choice([1, 2, 3, 4]), r.choice(dims), r.choice(vdims), r.choice([1.0, 4.0, 16.0, 40.0])))


def draw_config(seed: int) -> dict:
    r = random.Random(seed)
    width = r.choice([48, 64, 72, 100, 128, 160, 192, 256, 320, 384])
    cfg = {"architecture": "Pelenex", "vocab": r.choice([97, 200, 333, 512, 777, 1500]), "width": width,
           "norm": {"eps": r.choice([1e-5, 1e-6, 1e-4])}}
    if r.random() < 0.8:
        cfg["norm"]["groups"] = r.choice([g for g in (1, 2, 3, 4, 5, 8) if width % g == 0])
    if r.random() < 0.8:
        cfg["logit_softcap"] = r.choice([5.0, 12.0, 30.0])
    kinds = r.choice([("mlstm", "channel_delta", "parallel")] * 4 + [("mlstm",), ("channel_delta",), ("parallel",)])
    cfg["layers"] = [layer(draw_mixer(r, r.choice(kinds)), draw_mlp(r, seed % 2 == 1)) for _ in range(r.choice([1, 2, 3, 4, 5]))]
    return cfg


@pytest.mark.parametrize("seed", range(14))
def test_a_random_model_whole_decoded_in_portions_and_batched(tmp_path, seed):
    from vlrf_b200.engine import Engine, load_model
    cfg = draw_config(5000 + seed)
    write_model(cfg, seed, tmp_path, ranks=1 + 3 * seed, slow=float(seed % 3), apart=0.0 if seed % 2 else 20.0)
    pc, w = plain.read_model_dir(tmp_path)
    reqs = [random_ids(cfg["vocab"], n, 37 * seed + i) for i, n in enumerate((1 + seed % 3, 66 + 5 * seed, 141, 230))]
    want = [plain.logits_all_positions(pc, w, ids) for ids in reqs]
    decided = [plain.decided_prefix(pc, w, ids) for ids in reqs]
    for dtype in ("float32", "bfloat16"):
        eng = Engine(load_model(tmp_path, dtype), max_tokens=768)
        poison_states(eng)
        name = f"random {seed}"
        compare(drive_whole(eng, reqs), want, dtype, "whole", name, decided)
        compare(drive_tail_one_by_one(eng, reqs, 36), want, dtype, "prefix + 36 single tokens", name, decided)
        compare(drive_portions(eng, reqs, 2 + seed % 9), want, dtype, "portions", name, decided)
        poison_states(eng)
        compare(drive_batches(eng, reqs, 4, [1, 33, 100, 199]), want, dtype, "unequal batch", name, decided)
        assert eng.cache.slots.n_held == 0
