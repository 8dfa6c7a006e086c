"""Vilodra configurations drawn at random (every size, count, constant and the order of layers from a seeded generator; keys that may
be absent are absent now and then) through the engine against the plain implementation: whole, the last tokens one by one,
prompts in portions and an unequal batch.  What the hand-made models happen not to combine shows here: larger widths and heads,
states of more rows than columns, windows around the requests' lengths, several readers of one layer's latents, layers of one
kind only.

The 32-bit comparison covers every position.  In bfloat16 only the positions before a router's first close call are held
against the plain implementation; every other configuration therefore takes every expert and is compared at every position
in bfloat16 too."""
import random

import pytest

import plain_vilodra as plain
from conftest import random_ids
from engine_drives import drive_batches, drive_portions, drive_tail_one_by_one, drive_whole
from test_vilodra import compare, poison_states
from vilodra_models import dense, diffatt, latent, layer, lightning, moe, write_model

pytestmark = pytest.mark.gpu


def draw_mlp(r: random.Random, every: bool):
    x = r.random()
    if x < 0.15:
        return None
    if x < 0.5:
        return dense(r.choice([24, 40, 64, 100, 136, 304]))
    experts = r.choice([1, 2, 3, 4, 5] if every else [1, 2, 3, 4, 6, 11, 17, 40])
    return moe(r.choice([24, 40, 64, 96, 136]), experts, experts if every else r.randint(1, min(experts, 6)), r.choice([0.5, 1.0, 2.2]))


def draw_mixer(r: random.Random, kind: str, layers: list):
    if kind == "lightning":
        n = r.choice([1, 2, 3, 5])
        return lightning(r.choice([4, 8, 13, 16, 32, 48, 64, 72, 96, 128, 160]), r.choice([4, 8, 15, 16, 32, 40, 64, 96, 128, 136]),
                         *[r.choice([0.3, 0.7, 0.9, 0.97, 0.995, 0.9995]) for _ in range(n)])
    if kind == "attention":
        kv, dim = r.choice([1, 1, 2, 3]), r.choice([8, 12, 16, 24, 32, 48, 64, 96, 128])
        rot = sc = None
        if r.random() < 0.9:
            rot = (r.choice([d for d in (2, 4, 8, 12, 16, 32, 64) if d <= dim]), r.choice([50.0, 1000.0, 10000.0, 500000.0]))
            sc = r.choice([None, (4.0, 1.0, 4.0, 64), (8.0, 0.5, 2.0, 512), (2.0, 1.0, 8.0, 128)])
        return diffatt(kv * r.choice([1, 2, 4, 5]), kv, dim, r.choice([8, 12, 16, 24, 40, 64, 96, 128]), round(dim ** -0.5 * r.choice([0.7, 1.0, 2.0]), 4),
                       r.choice([0.0, 0.2, 0.55, 0.8]), rot, sc)
    window = r.choice([None, 1, 5, 31, 64, 65, 100, 128, 140, 200])
    heads, dim, vdim = r.choice([1, 2, 3, 4, 6, 17]), r.choice([8, 12, 16, 24, 32, 48, 64]), r.choice([8, 12, 16, 24, 40, 64])
    owners = [i for i, lay in enumerate(layers) if lay["type"] == "latent_attention" and "kv_from" not in lay["mixer"]]
    if owners and r.random() < 0.6:
        j = r.choice(owners)
        o = layers[j]["mixer"]
        m = latent(heads, dim, o["rot_dim"], vdim, o["kv_rank"], 0.1, window, kv_from=j)
        m["mixer"]["rot"] = o["rot"]
    else:
        m = latent(heads, dim, r.choice([4, 6, 8, 16, 32]), vdim, r.choice([16, 32, 36, 40, 64, 96, 160]), 0.1, window, r.choice([100.0, 10000.0]),
                   r.choice([None, (4.0, 64, 8.0, 1.0), (2.0, 256, 32.0, 2.0)]))
    m["mixer"]["scale"] = round((dim + m["mixer"]["rot_dim"]) ** -0.5 * r.choice([0.8, 1.0, 2.0]), 4)
    return m


def draw_config(seed: int) -> dict:
    r = random.Random(seed)
    cfg = {"architecture": "Vilodra", "vocab": r.choice([97, 200, 333, 512, 777, 1500]), "width": r.choice([48, 64, 72, 100, 128, 192, 256, 320]),
           "norm": {"eps": r.choice([1e-5, 1e-6, 1e-4])}, "residual_mult": r.choice([0.25, 0.6, 1.0, 1.4])}
    kinds = r.choice([("lightning", "attention", "latent_attention")] * 3 + [("latent_attention",), ("lightning",), ("attention",)])
    cfg["layers"] = []
    for _ in range(r.choice([2, 3, 4, 5])):
        cfg["layers"].append(layer(draw_mixer(r, r.choice(kinds), cfg["layers"]), draw_mlp(r, seed % 2 == 1)))
    return cfg


@pytest.mark.parametrize("seed", range(16))
def test_a_random_model_whole_decoded_in_portions_and_batched(tmp_path, seed):
    from vlrf_b200.engine import Engine, load_model
    cfg = draw_config(7000 + seed)
    write_model(cfg, seed, tmp_path)
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
