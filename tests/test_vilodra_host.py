"""Vilodra without a GPU: the configuration reader (every key read, absent keys, refusals), the tensor list, what layers keep and
share, the rotations' frequency tables, the factor on the second map, and the plain functions' own edge cases."""
import copy
import math

import pytest
import torch

import plain_vilodra as plain
from vilodra_models import MODELS, VIL_A, VIL_B, VIL_ODD


def parse(cfg):
    import vlrf_b200.models  # noqa: F401
    from vlrf_b200.registry import parse_config
    return parse_config(cfg)


def test_every_key_is_read():
    arch, c = parse(VIL_A)
    assert arch.name == "Vilodra" and (c.vocab, c.width, c.norm_eps, c.residual_mult) == (311, 96, 1e-5, 0.7)
    m = c.mixers[0]
    assert m.kind == "latent_attention" and (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale) == (3, 16, 8, 24, 40, 0.25)
    assert (m.rot.base, m.rot.dims, m.rot.scaling, m.window, m.kv_from) == (1000.0, 8, (4.0, 64.0, 8.0, 2.0), 40, None)
    m = c.mixers[1]
    assert m.kind == "attention" and (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.diff) == (6, 2, 16, 40, 0.3, 0.3)
    assert (m.rot.base, m.rot.dims, m.rot.scaling) == (500.0, 8, (4.0, 1.0, 4.0, 128.0))
    m = c.mixers[2]
    assert m.kind == "lightning" and (m.heads, m.dim, m.vdim, m.decay) == (3, 24, 16, (0.55, 0.93, 0.998))
    assert c.mixers[3].kv_from == 0 and c.mixers[3].heads == 5 and c.mixers[4].rot.scaling is None
    assert (c.mlps[1].kind, c.mlps[1].ff, c.mlps[1].experts, c.mlps[1].top, c.mlps[1].scale) == ("moe", 40, 5, 2, 1.5)
    assert (c.mlps[0].kind, c.mlps[0].ff) == ("dense", 72) and c.mlps[2] is None
    assert parse(c.to_dict())[1].to_dict() == c.to_dict()


def test_absent_keys():
    _, c = parse(VIL_ODD)
    assert c.mixers[3].window == 0 and c.mixers[1].rot.scaling is None and c.mixers[4].rot is None and c.mlps[3] is None
    cfg = copy.deepcopy(VIL_ODD)
    del cfg["residual_mult"]
    assert parse(cfg)[1].residual_mult == 1.0


@pytest.mark.parametrize("change,where", [
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(low=4.0), "low"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0), "scaling"),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask"),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=0), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=6), "rot_dim"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_rank=48), "kv_rank"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(base=999.0), "rot"),
    (lambda c: c["layers"][2]["mixer"].update(heads=4), "decay"),
    (lambda c: c["layers"][2]["mixer"].update(decay=0.5), "decay"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=0), "vdim"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "inner size"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "kind"),
    (lambda c: c["layers"][0].update(type="mlstm"), "type"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_refusals(change, where):
    from vlrf_b200.config import ConfigError
    cfg = copy.deepcopy(VIL_A)
    change(cfg)
    with pytest.raises(ConfigError, match=where):
        parse(cfg)


def test_tensor_list():
    arch, c = parse(VIL_A)
    specs = arch.weight_spec(c)
    spec = {s.name: s.shape for s in specs}
    assert len(spec) == len(specs)
    assert spec["embed"] == (311, 96) and spec["final.norm"] == (96,) and "head" not in spec
    assert spec["l0.mix.q"] == (3 * 24, 96) and spec["l0.mix.dkv"] == (48, 96) and spec["l0.mix.dkv.norm"] == (40,)
    assert spec["l0.mix.uk"] == (48, 40) and spec["l0.mix.uv"] == (72, 40) and spec["l0.mix.sink"] == (3,) and spec["l0.mix.o"] == (96, 72)
    assert spec["l1.mix.q"] == (6 * 2 * 16, 96) and spec["l1.mix.k"] == (2 * 2 * 16, 96) and spec["l1.mix.v"] == (80, 96)
    assert spec["l1.mix.lq1"] == spec["l1.mix.lk2"] == (16,) and spec["l1.mlp.router"] == (5, 96) and spec["l1.mlp.e4.down"] == (96, 40)
    assert "l1.mlp.e0.gate" not in spec and "l3.mix.dkv" not in spec and "l3.mix.dkv.norm" not in spec and spec["l3.mix.sink"] == (5,)
    assert spec["l2.mix.norm"] == (48,) and spec["l2.mix.g"] == (48, 96) and not any(n.startswith("l2.mlp") for n in spec)
    assert [s.optional for s in specs if s.name in ("l1.norm2", "l2.norm2")] == [False, True]
    drawn = arch.random_weights(c, torch.Generator().manual_seed(1))
    assert set(drawn) == set(spec) - {"l2.norm2"} and all(tuple(drawn[n].shape) == spec[n] for n in drawn)


def test_what_layers_keep_and_share():
    """A shared cache keeps what the widest window of its readers asks for, and every row as soon as one of them sees all."""
    from vlrf_b200.cache import KVNeed, LatentNeed, StateNeed
    from vlrf_b200.engine.model import BuildOptions
    from vlrf_b200.weights.spec import CheckedWeights
    for cfg, windows in ((VIL_A, {0: 70, 3: 70}), (VIL_B, {1: 130, 3: 130, 4: 130}), (VIL_ODD, {1: 0, 3: 0})):
        arch, c = parse(cfg)
        assert {i: c.cache_window(i) for i in windows} == windows
        w = arch.random_weights(c, torch.Generator().manual_seed(2))
        model = arch.build(c, CheckedWeights(w), BuildOptions(torch.float32, torch.device("cpu")))
        needs = model.cache_needs()
        for i, win in windows.items():
            m = c.mixers[i]
            own = LatentNeed(m.kv_rank + m.rot_dim, "window", win) if win else LatentNeed(m.kv_rank + m.rot_dim)
            assert model.layers[i].cache_need() == own and needs[i] == (own if m.kv_from is None else None)
            assert model.layers[i].mixer.window == m.window
    arch, c = parse(VIL_A)
    model = arch.build(c, CheckedWeights(arch.random_weights(c, torch.Generator().manual_seed(2))), BuildOptions(torch.float32, torch.device("cpu")))
    needs = model.cache_needs()
    assert needs[1] == KVNeed(2, 32, "full", v_dim=40) and needs[4] == KVNeed(1, 48, "full", v_dim=24)
    assert needs[2] == StateNeed((2, 3 * 24 * 16), torch.float32) and needs[5] == StateNeed((2, 2 * 8 * 40), torch.float32)
    assert parse(VIL_B)[1].mixers[2].vdim == 2 * parse(VIL_B)[1].mixers[2].dim
    # where the factor on a sublayer's output goes
    assert model.layers[0].mixer.out_factor == 0.7 and model.layers[0].feed_forward.out_factor == 0.7
    assert model.layers[1].mixer.out_factor == pytest.approx(0.7 * 0.7) and model.layers[1].feed_forward.weight_scale == pytest.approx(1.5 * 0.7)
    assert model.layers[2].mixer.out_factor == 0.7 and model.layers[2].feed_forward is None


def test_parts_refuse_what_does_not_fit():
    from vlrf_b200.parts import get_part
    w = torch.zeros
    att = get_part("mixer", "window_attention")
    ok = dict(n_heads=2, n_kv_heads=1, dim=4, vdim=6, scale=1.0, second_map=(0.5, 1e-5))
    assert att(w(16, 8), w(8, 8), w(6, 8), w(8, 12), **ok).in_width == 30
    for bad, match in ((dict(sink=w(2)), "sinks"), (dict(w_gate=w(2, 8)), "sinks"), (dict(second_map=(0.5, 0.0)), "eps")):
        with pytest.raises(ValueError, match=match):
            att(w(16, 8), w(8, 8), w(6, 8), w(8, 12), **{**ok, **bad})
    with pytest.raises(ValueError, match="twice the rows"):
        att(w(8, 8), w(4, 8), w(6, 8), w(8, 12), **ok)
    lat = get_part("mixer", "latent_attention")
    base = dict(n_heads=2, dim=3, vdim=4, kv_rank=5, scale=1.0, w_uk=w(6, 5), w_uv=w(8, 5), w_out=w(8, 8), w_q=w(6, 8), w_dkv=w(5, 8), dkv_norm=w(5))
    assert lat(**base, window=7, cache_window=9).cache_need().window == 9 and lat(**base, window=7, cache_window=0).cache_need().kind == "full"
    for bad in (dict(window=9, cache_window=7), dict(window=0, cache_window=7), dict(window=-1)):
        with pytest.raises(ValueError, match="window"):
            lat(**base, **bad)
    with pytest.raises(ValueError, match="sink"):
        lat(**base, sink=w(3))
    with pytest.raises(ValueError, match="decays"):
        get_part("mixer", "fixed_memory")(w(6, 8), w(6, 8), w(8, 8), w(8, 8), w(8), w(8, 8), n_heads=2, dim=3, vdim=4, decay=[0.5], eps=1e-5)
    moe = get_part("feed_forward", "routed_experts")
    with pytest.raises(ValueError, match="one already"):
        moe(w(3, 8), None, None, w(3, 5, 8), w(3, 8, 5), top=1, renormalize=True)
    with pytest.raises(ValueError, match="activation"):
        moe(w(3, 8), None, None, w(3, 5, 8), w(3, 8, 5), top=1, scoring="softmax_all", activation="tanh")


@pytest.mark.parametrize("dims,base,sc", [(32, 10000.0, (4.0, 1.0, 4.0, 128)), (16, 500.0, (8.0, 1.0, 4.0, 1024)), (48, 20.0, (2.0, 0.5, 8.0, 64)),
                                          (8, 3.0, (4.0, 1.0, 2.0, 8192))])
def test_frequencies_by_wavelength(dims, base, sc):
    from vlrf_b200.parts import RotaryPositions
    part = RotaryPositions(base, dims, "cpu", pairing="interleaved", wavelengths=sc)
    f = plain.frequencies({"base": base, "dims": dims})
    want = plain.stretched(f, dict(zip(("factor", "low", "high", "original"), sc)))
    assert part.inv_freq.tolist() == pytest.approx(want, rel=1e-6) and part.magnitude == 1.0
    with pytest.raises(ValueError, match="wavelength"):
        RotaryPositions(base, dims, "cpu", wavelengths=(4.0, 2.0, 2.0, 64))
    with pytest.raises(ValueError, match="wavelength"):
        RotaryPositions(base, dims, "cpu", wavelengths=sc, yarn=(4.0, 64, 8.0, 1.0))


def test_wavelength_scaling_has_three_ranges():
    """A table that reaches all three, with the blend continuous at both ends."""
    sc = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64.0}
    two_pi = 2 * math.pi
    f = [two_pi / 15.0, two_pi / 16.0, two_pi / 40.0, two_pi / 64.0, two_pi / 65.0]
    got = plain.stretched(f, sc)
    assert got[0] == f[0] and got[1] == pytest.approx(f[1]) and got[3] == pytest.approx(f[3] / 4) and got[4] == f[4] / 4
    s = (64 / 40 - 1) / 3
    assert got[2] == pytest.approx((1 - s) * f[2] / 4 + s * f[2]) and f[2] / 4 < got[2] < f[2]


def test_factor_on_the_second_map():
    from vlrf_b200.models.vilodra import second_map_factor
    g = torch.Generator().manual_seed(4)
    v = [(0.4 * torch.randn(12, generator=g)).bfloat16() for _ in range(4)]
    w = {"p.lq1": v[0].double(), "p.lk1": v[1].double(), "p.lq2": v[2].double(), "p.lk2": v[3].double()}
    assert second_map_factor(*v, 0.35) == pytest.approx(float(plain.mix_of_maps(w, "p.", 0.35)), rel=1e-12)
    z = torch.zeros(3)
    assert second_map_factor(z, z, z, z, 0.6) == 0.6


def test_plain_attention_edges():
    # equal scores: a window of 2 averages the last two values; a sink of the keys' score takes its share
    q = k = torch.zeros(4, 1, 2, dtype=torch.float64)
    v = torch.tensor([[[1.0]], [[10.0]], [[100.0]], [[1000.0]]], dtype=torch.float64)
    assert plain.attend(q, k, v, 1.0, 2)[:, 0, 0].tolist() == pytest.approx([1.0, 5.5, 55.0, 550.0])
    assert plain.attend(q, k, v, 1.0)[3, 0, 0] == pytest.approx(1111 / 4)
    sink = torch.zeros(1, dtype=torch.float64)
    assert plain.attend(q, k, v, 7.0, 2, sink)[:, 0, 0].tolist() == pytest.approx([0.5, 11 / 3, 110 / 3, 1100 / 3])
    big = torch.full((1,), 800.0, dtype=torch.float64)           # (a sink far above every score leaves nothing, and no overflow)
    assert float(plain.attend(q, k, v, 1.0, None, big).abs().max()) < 1e-300


def test_plain_recurrence_and_experts_written_out():
    t = lambda *v: torch.tensor(v, dtype=torch.float64).view(-1, 1, 1)   # noqa: E731
    got = plain.fading_memory(t(2.0, 3.0, 1.0), t(5.0, 7.0, 0.0), t(0.5, -1.0, 9.0), torch.tensor([0.25], dtype=torch.float64)).flatten().tolist()
    assert got == pytest.approx([2 * 2.5, 3 * (0.25 * 2.5 - 7.0), 0.25 * (0.25 * 2.5 - 7.0)])
    d = lambda x: torch.tensor([[x]], dtype=torch.float64)   # noqa: E731
    w = {"p.router": torch.tensor([[1.0], [3.0], [2.0]], dtype=torch.float64)}
    for e, (up, down) in enumerate(((1.0, 1.0), (0.5, 2.0), (-1.0, 3.0))):
        w[f"p.e{e}.up"], w[f"p.e{e}.down"] = d(up), d(down)
    s = [math.exp(v) for v in (1.0, 3.0, 2.0)]
    gelu = lambda z: 0.5 * z * (1 + math.erf(z / 2 ** 0.5))   # noqa: E731
    want = 1.7 * (s[1] * 2.0 * gelu(0.5) + s[2] * 3.0 * gelu(-1.0)) / (s[1] + s[2])
    assert float(plain.routed_ff(d(1.0), w, "p.", {"router": {"top": 2, "experts": 3, "scale": 1.7}})) == pytest.approx(want)


def test_configurations_differ():
    sizes = [(c["width"], c["vocab"], len(c["layers"]), c["residual_mult"]) for c in MODELS.values()]
    assert len(set(sizes)) == len(sizes) and VIL_ODD["width"] % 8 != 0
