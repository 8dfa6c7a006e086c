"""Vilodra through the engine against the plain implementation: whole requests, the last tokens one by one, prompts in
portions down to two tokens, unequal batches with reused slots, blocks and states, the first tokens, long decoding
past every window, a step of seventy sequences, greedy generation through the package's entry point and a replay through
bin/trace_run — in 32-bit and in bfloat16, on four small models whose sizes all differ."""
import pytest
import torch

import plain_vilodra as plain
from conftest import random_ids, record_error
from engine_drives import drive_batches, drive_portions, drive_tail_one_by_one, drive_whole, poison
from vilodra_models import MODELS, SHARP_FACTOR, every_expert, write_model

pytestmark = pytest.mark.gpu

#: largest absolute logit error over the largest absolute logit of the plain implementation
TOL = {"float32": 1e-4, "bfloat16": 5e-2}
DTYPES = ["float32", "bfloat16"]
LENGTHS = {"vil_a": [1 + 12, 17 + 12, 64 + 12, 65 + 12, 150, 215], "vil_b": [3 + 10, 63 + 10, 129 + 10, 200],
           "vil_odd": [2 + 8, 40 + 8, 100 + 8, 141], "vil_sharp": [5 + 16, 64 + 16, 127 + 16, 260]}
DECODE = {"vil_a": 12, "vil_b": 10, "vil_odd": 8, "vil_sharp": 16}
NAMES = list(MODELS)


def poison_states(engine):
    """NaN in every block of the cache and in the states of every slot that no sequence holds: a slot that is taken must be zeroed,
    not trusted."""
    poison(engine)
    for g in engine.cache._groups:
        if hasattr(g, "state"):
            for s in range(engine.cache.n_slots):
                if not engine.cache.slots.is_held(s):
                    g.state[:, s].fill_(float("nan"))


@pytest.fixture(scope="module")
def vil_dirs(tmp_path_factory):
    """(model, dtype) -> folder.  bfloat16 runs a model of the same layers whose tokens take every expert: then no choice rests on
    rounding, and every position can be held against the plain implementation."""
    out = {}
    for i, (name, cfg) in enumerate(MODELS.items()):
        for dtype in DTYPES:
            d = tmp_path_factory.mktemp(f"{name}_{dtype}")
            write_model(cfg if dtype == "float32" else every_expert(cfg), 60 + i, d, sharp=SHARP_FACTOR if name == "vil_sharp" else 1.0)
            out[name, dtype] = d
    return out


@pytest.fixture(scope="module")
def truth(vil_dirs):
    out = {}
    for (name, dtype), d in vil_dirs.items():
        cfg, w = plain.read_model_dir(d)
        reqs = [random_ids(cfg["vocab"], n, 11 + i) for i, n in enumerate(LENGTHS[name])]
        out[name, dtype] = (cfg, w, reqs, [plain.logits_all_positions(cfg, w, ids) for ids in reqs])
    return out


def make_engine(vil_dirs, name, dtype, max_tokens):
    from vlrf_b200.engine import Engine, load_model
    eng = Engine(load_model(vil_dirs[name, dtype], dtype), max_tokens=max_tokens)
    poison_states(eng)
    return eng


def compare(got, want, dtype, what, model, decided=None):
    """Every position; with `decided` (per request) and bfloat16 the positions before a router's first close call, since rounding may
    choose another expert there and everything later in the sequence depends on that token."""
    worst = 0.0
    for i, (g, t) in enumerate(zip(got, want)):
        assert g.shape == t.shape, f"{what}: request {i} has shape {tuple(g.shape)}, expected {tuple(t.shape)}"
        assert torch.isfinite(g).all(), f"{what}: request {i} has non-finite logits (something unwritten was read)"
        err = (g.double() - t).abs().max(dim=1).values / float(t.abs().max())
        if dtype != "float32" and decided is not None:
            err = err[:decided[i]]
            if err.numel() == 0:
                continue
        bad = (err > TOL[dtype]).nonzero()
        assert bad.numel() == 0, (f"{what} ({model}, {dtype}): request {i} (length {len(t)}) first differs at position "
                                  f"{int(bad[0])} with error {float(err[bad[0]]):.3e} of the logit scale")
        worst = max(worst, float(err.max()))
    record_error("vilodra " + what, model, dtype, worst)


def test_the_sharp_model_is_sharp_and_decided(truth):
    """Its last position must depend on single tokens: another one at the oldest position inside the first layer's window of 48, one
    right outside it, and the sequence's second each move the last logits far beyond rounding, and so does a model whose
    windows are one token wider or whose sinks are gone.  None of the routers of the models that bfloat16 runs has a choice to
    make, so it is compared at every position."""
    import copy
    cfg, w, reqs, want = truth["vil_sharp", "float32"]
    scale = want[3].abs().max()
    for place in (1, len(reqs[3]) - 49, len(reqs[3]) - 48):
        ids = [(t + 1) % cfg["vocab"] if i == place else t for i, t in enumerate(reqs[3])]
        moved = plain.logits_all_positions(cfg, w, ids)[-1]
        assert float((moved - want[3][-1]).abs().max() / scale) > 0.02, place
    wider = copy.deepcopy(cfg)
    for lay in wider["layers"]:
        if "mask" in lay["mixer"]:
            lay["mixer"]["mask"]["size"] += 1
    gone = {k: (v * 0 - 100.0 if k.endswith(".sink") else v) for k, v in w.items()}
    for c, ww in ((wider, w), (cfg, gone)):
        assert float((plain.logits_all_positions(c, ww, reqs[3]) - want[3]).abs().max() / scale) > 0.05
    for name in NAMES:
        cfg, w, reqs, _ = truth[name, "bfloat16"]
        assert [plain.decided_prefix(cfg, w, r) for r in reqs] == [len(r) for r in reqs], name


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_each_request_alone_and_whole(vil_dirs, truth, name, dtype):
    _, _, reqs, want = truth[name, dtype]
    eng = make_engine(vil_dirs, name, dtype, 320)
    compare(drive_whole(eng, reqs), want, dtype, "whole", name)
    eng.cache.check()
    assert eng.cache.slots.n_held == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_last_tokens_one_by_one(vil_dirs, truth, name, dtype):
    _, _, reqs, want = truth[name, dtype]
    eng = make_engine(vil_dirs, name, dtype, 320)
    compare(drive_tail_one_by_one(eng, reqs, 32), want, dtype, "prefix + 32 single tokens", name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [2, 3, 7, 64, 65])
def test_prompts_in_portions(vil_dirs, truth, portion, dtype):
    """Portions of an even and of an odd number of tokens (the two copies of a state), down to two tokens."""
    for name in ("vil_a", "vil_odd", "vil_sharp"):
        _, _, reqs, want = truth[name, dtype]
        eng = make_engine(vil_dirs, name, dtype, 320)
        compare(drive_portions(eng, reqs[1:], portion), want[1:], dtype, f"portions of {portion}", name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_with_reused_slots_blocks_and_states(vil_dirs, truth, name, dtype):
    _, _, reqs, want = truth[name, dtype]
    prompt_lens = [max(1, len(r) - DECODE[name]) for r in reqs]
    batch = 3
    order = list(reversed(range(len(reqs))))

    def need_of(rs):
        return max(sum((len(r) + 63) // 64 * 64 for r in rs[b:b + batch]) for b in range(0, len(rs), batch))

    eng = make_engine(vil_dirs, name, dtype, max(need_of(reqs), need_of([reqs[i] for i in order])))
    compare(drive_batches(eng, reqs, batch, prompt_lens), want, dtype, "unequal batches", name)
    assert eng.cache.slots.n_held == 0
    poison_states(eng)           # what the second pass reads it must have written (or zeroed) itself
    got = drive_batches(eng, [reqs[i] for i in order], batch, [prompt_lens[i] for i in order])
    compare(got, [want[i] for i in order], dtype, "unequal batches, reused cache", name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_first_tokens(vil_dirs, truth, name, dtype):
    cfg, w, _, _ = truth[name, dtype]
    reqs = [random_ids(cfg["vocab"], n, 70 + n) for n in (1, 2, 3, 1)]
    want = [plain.logits_all_positions(cfg, w, ids) for ids in reqs]
    eng = make_engine(vil_dirs, name, dtype, 256)
    compare(drive_whole(eng, reqs), want, dtype, "first tokens, whole", name)
    compare(drive_batches(eng, reqs, 4, [1, 1, 1, 1]), want, dtype, "first tokens, batch", name)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_from_one_token(vil_dirs, truth, dtype):
    for name in ("vil_b", "vil_sharp"):
        cfg, w, _, _ = truth[name, dtype]
        ids = random_ids(cfg["vocab"], 200, 5)
        want = plain.logits_all_positions(cfg, w, ids)
        eng = make_engine(vil_dirs, name, dtype, 256)
        compare(drive_tail_one_by_one(eng, [ids], tail=len(ids) - 1), [want], dtype, "decoding 200 positions", name)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_batch_of_seventy_sequences(vil_dirs, truth, dtype):
    """More rows in a decode step than the few-row products take."""
    cfg, w, _, _ = truth["vil_odd", dtype]
    reqs = [random_ids(cfg["vocab"], 4 + (i * 7) % 30, 300 + i) for i in range(70)]
    want = [plain.logits_all_positions(cfg, w, ids) for ids in reqs]
    eng = make_engine(vil_dirs, "vil_odd", dtype, 70 * 64)
    compare(drive_batches(eng, reqs, 70, [max(1, len(r) - 3) for r in reqs]), want, dtype, "seventy sequences", "vil_odd")


@pytest.mark.parametrize("name", ["vil_a", "vil_b"])
def test_greedy_generation_through_the_entry_point(tmp_path, name):
    """Seven requests over three rows: requests wait, take over rows (and states) of those that ended, and decode in the
    replayed session beside padding rows, whose first step runs twice; every request gets what it gets alone from the
    plain implementation (32-bit, so that no argmax rests on rounding)."""
    from vlrf_b200.api import Model
    from vlrf_b200.sampling.params import SamplingParams
    write_model(MODELS[name], 77, tmp_path)
    cfg, w = plain.read_model_dir(tmp_path)
    prompts = [random_ids(cfg["vocab"], n, 900 + n) for n in (3, 20, 1, 66, 9, 33, 5)]
    new = [6, 3, 9, 4, 7, 2, 8]
    model = Model.load(tmp_path, "float32", max_tokens=3 * 128, n_slots=3)
    params = [SamplingParams(max_new_tokens=n, do_sample=False) for n in new]
    results = model.generate_ids(prompts, params)
    want = [plain.greedy_generate(cfg, w, p, n) for p, n in zip(prompts, new)]
    assert [r.new_tokens for r in results] == want
    assert len({t for ts in want for t in ts}) > 10, "the model just repeats itself: the test would show nothing"
    assert model.engine.cache.slots.n_held == 0
    model.engine.cache.check()


def test_trace_replay_of_a_batch_of_unequal_requests(vil_dirs, truth, tmp_path):
    """`bin/trace_run` on a Vilodra folder: twelve requests of 1 to 70 tokens start together in one step, go on one token
    a step and end one after another.  32-bit, every wanted position."""
    from test_trace_run import Replay, read
    cfg, w, _, _ = truth["vil_a", "float32"]
    V = cfg["vocab"]
    reqs = {f"q{i}": random_ids(V, n, 500 + i) for i, n in enumerate([1, 2, 3, 5, 8, 13, 21, 34, 55, 70, 4, 1])}
    want = {k: plain.logits_all_positions(cfg, w, ids) for k, ids in reqs.items()}
    decode = 4
    fed = {k: max(1, len(ids) - decode) for k, ids in reqs.items()}
    rp = Replay(vil_dirs["vil_a", "float32"], "float32", tmp_path / "out", sum(len(v) for v in reqs.values()))
    f = rp.send([{"id": k, "tokens": ids[:fed[k]], "want": [fed[k] - 1]} for k, ids in reqs.items()],
                end=[k for k, ids in reqs.items() if fed[k] == len(ids)])
    got = read(f, V)
    for r, k in enumerate(reqs):
        assert float((got[r].double() - want[k][fed[k] - 1]).abs().max() / want[k].abs().max()) < TOL["float32"], (k, "prompt")
    live = [k for k, ids in reqs.items() if fed[k] < len(ids)]
    while live:
        f = rp.send([{"id": k, "tokens": [reqs[k][fed[k]]], "want": [0]} for k in live],
                    end=[k for k in live if fed[k] + 1 == len(reqs[k])])
        got = read(f, V)
        for r, k in enumerate(live):
            assert float((got[r].double() - want[k][fed[k]]).abs().max() / want[k].abs().max()) < TOL["float32"], (k, fed[k])
            fed[k] += 1
        live = [k for k in live if fed[k] < len(reqs[k])]
    rp.close()
