"""Pelenex without a GPU: the configuration reader (every key read, absent keys, refusals), the tensor list with sizes that
only the tensors say, what every layer keeps, the block's joint matrices, and the plain functions' own edge cases."""
import copy
import math

import pytest
import torch

import plain_pelenex as plain
from pelenex_models import MODELS, PEL_A, PEL_B, PEL_ODD


def parse(cfg):
    import vlrf_b200.models  # noqa: F401
    from vlrf_b200.registry import parse_config
    return parse_config(cfg)


def test_every_key_is_read():
    arch, c = parse(PEL_A)
    assert arch.name == "Pelenex" and (c.vocab, c.width, c.norm_eps, c.norm_groups, c.logit_softcap) == (311, 96, 1e-5, 3, 20.0)
    m = c.mixers[0]
    assert m.kind == "parallel" and (m.attention.heads, m.attention.kv_heads, m.attention.dim, m.attention.vdim) == (6, 2, 16, 16)
    assert (m.attention.scale, m.attention.window, m.attention.keep_first) == (0.3, 37, 5)
    assert (m.memory.heads, m.memory.dim, m.memory.vdim, m.memory.tau) == (3, 24, 16, 8.0)
    assert (c.mixers[3].attention.window, c.mixers[3].attention.keep_first) == (70, 0)
    m = c.mixers[1]
    assert m.kind == "mlstm" and (m.memory.heads, m.memory.dim, m.memory.vdim, m.memory.gate_cap) == (3, 16, 40, 9.0)
    m = c.mixers[2]
    assert m.kind == "channel_delta" and (m.memory.heads, m.memory.kv_heads, m.memory.dim, m.memory.vdim, m.memory.conv) == (4, 2, 24, 16, 4)
    assert (c.mlps[0].kind, c.mlps[0].ff, c.mlps[0].experts, c.mlps[0].top, c.mlps[0].shared_ff) == ("moe", 40, 5, 2, 56)
    assert (c.mlps[1].kind, c.mlps[1].ff) == ("dense", 72) and c.mlps[3] is None and c.mlps[5].shared_ff == 0
    assert parse(c.to_dict())[1].to_dict() == c.to_dict()


def test_absent_keys():
    _, c = parse(PEL_B)
    assert c.norm_groups == 1 and c.logit_softcap is None and c.mixers[1].attention.window == 0 and c.mlps[0] is None


@pytest.mark.parametrize("change,where", [
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=24), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(tau=0.0), "tau"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].update(dim=0), "dim"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][2]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0), "shared"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gated"), "kind"),
    (lambda c: c["layers"][1].update(type="attention"), "type"),
    (lambda c: c["norm"].update(groups=7), "groups"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c.update(logit_softcap=0.0), "softcap"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_refusals(change, where):
    from vlrf_b200.config import ConfigError
    cfg = copy.deepcopy(PEL_A)
    change(cfg)
    with pytest.raises(ConfigError, match=where):
        parse(cfg)


def test_tensor_list():
    arch, c = parse(PEL_A)
    specs = arch.weight_spec(c)
    spec = {s.name: s.drawn_shape for s in specs}
    assert len(spec) == len(specs)
    assert spec["embed"] == spec["head"] == (311, 96) and spec["final.norm"] == (96,)
    assert spec["l0.mix.left.q"] == (96, 96) and spec["l0.mix.left.k"] == (32, 96) and "l0.mix.left.v" not in spec
    assert spec["l0.mix.right.norm"] == (16,) and spec["l0.mix.right.a2.b"] == (72,) and spec["l0.mix.right.out"] == (96,)
    assert spec["l1.mix.norm"] == (120,) and spec["l1.mix.i"] == (3, 96) and spec["l1.mix.f.b"] == (3,) and spec["l1.mix.o"] == (96, 120)
    assert spec["l2.mix.q"] == (48, 96) and spec["l2.mix.v.conv"] == (64, 4) and spec["l2.mix.A_log"] == (4,) and spec["l2.mix.dt_bias"] == (96,)
    assert spec["l2.mix.norm"] == (16,) and spec["l0.mlp.e4.down"] == (96, 40) and spec["l0.mlp.shared.gate"] == (56, 96)
    assert "l5.mlp.shared.gate" not in spec and not any(n.startswith("l3.mlp") for n in spec) and "l0.norm2" not in spec
    drawn = arch.random_weights(c, torch.Generator().manual_seed(1))
    assert set(drawn) == set(spec) and all(tuple(drawn[n].shape) == sh for n, sh in spec.items())


def test_sizes_that_only_the_tensors_say():
    """A rank is whatever the two tensors that share it agree on; one that disagrees is named."""
    from vlrf_b200.weights import FreeSize, TensorSpec, WeightError, check_tensors
    arch, c = parse(PEL_A)
    found = arch.random_weights(c, torch.Generator().manual_seed(1))
    found["l2.mix.a1"], found["l2.mix.a2"] = torch.zeros(7, 96), torch.zeros(96, 7)
    assert check_tensors(found, arch.weight_spec(c))["l2.mix.a1"].shape == (7, 96)
    found["l2.mix.a2"] = torch.zeros(96, 5)
    with pytest.raises(WeightError, match="l2.mix.a2"):
        check_tensors(found, arch.weight_spec(c))
    spec = [TensorSpec("a", (FreeSize("r", 4), 3)), TensorSpec("b", (2, FreeSize("r", 4)))]
    assert spec[0].drawn_shape == (4, 3)
    with pytest.raises(WeightError, match="b: expected"):
        check_tensors({"a": torch.zeros(6, 3), "b": torch.zeros(2, 5)}, spec)
    with pytest.raises(WeightError, match="a: expected"):
        check_tensors({"a": torch.zeros(6), "b": torch.zeros(2, 6)}, spec)


def test_what_layers_keep():
    from vlrf_b200.cache import KVNeed, StateNeed
    from vlrf_b200.parts import get_part
    w = torch.zeros
    decayed = get_part("mixer", "decayed_memory")(w(6, 10), w(6, 10), w(10, 10), w(10, 10), w(3, 10), w(6, 3), w(6), w(5), w(10, 10), n_heads=2,
                                                  dim=3, vdim=5, tau=4.0, eps=1e-5)
    assert decayed.cache_need() == StateNeed((2, 32), torch.float32) and decayed.in_width == 6 + 6 + 10 + 10 + 3
    stab = get_part("mixer", "stabilized_memory")(w(6, 10), w(6, 10), w(10, 10), w(10, 10), w(2, 10), w(2) + 1, w(2, 10), w(2) + 2, w(10), w(10, 10),
                                                  n_heads=2, dim=3, vdim=5, gate_cap=4.0, eps=1e-5)
    assert stab.cache_need() == StateNeed((2, 48), torch.float32)            # 2 · (5 + 1) · (3 + 1)
    assert stab.in_bias[-4:].tolist() == [1, 1, 2, 2] and not stab.in_bias[:-4].any()
    delta = get_part("mixer", "delta_memory")(w(6, 10), w(6, 10), w(20, 10), w(4, 10), w(6, 3), w(6, 3), w(20, 3), w(3, 10), w(12, 3), w(4), w(12), w(2, 10),
                                              w(20, 2), w(5), w(10, 20), n_heads=4, n_groups=2, dim=3, vdim=5, eps=1e-5)
    assert delta.cache_need() == StateNeed((2, 60 + 2 * 32), torch.float32) and delta.conv_off == 60
    att = get_part("mixer", "window_attention")(w(24, 10), w(8, 10), None, w(10, 24), n_heads=3, n_kv_heads=1, dim=8, vdim=8, scale=1.0, window=9,
                                                keep_first=2, qk_norm="head", norm_eps=1e-5, slopes=w(3))
    assert torch.equal(att.q_norm, torch.ones(8)) and torch.equal(att.k_norm, torch.ones(8))
    pair = get_part("mixer", "parallel")(att, decayed, left_scale=0.5, right_scale=0.5, out_norms=(w(10), w(10), 1e-5))
    assert pair.cache_need() == (KVNeed(1, 8, "window", 9, keep_first=2), decayed.cache_need()) and pair.out_weight is None
    with pytest.raises(ValueError, match="slope"):
        get_part("mixer", "window_attention")(w(24, 10), w(8, 10), None, w(10, 24), n_heads=3, n_kv_heads=1, dim=8, vdim=8, scale=1.0, slopes=w(2))
    with pytest.raises(ValueError, match="one scale"):
        get_part("mixer", "parallel")(att, decayed, left_scale=0.5, right_scale=0.6, out_norms=(w(10), w(10), 1e-5))
    with pytest.raises(ValueError, match="rank"):
        get_part("mixer", "decayed_memory")(w(6, 10), w(6, 10), w(10, 10), w(10, 10), w(3, 10), w(6, 2), w(6), w(5), w(10, 10), n_heads=2, dim=3, vdim=5,
                                            tau=4.0, eps=1e-5)


def test_a_block_joins_its_products_and_its_parts_let_go_of_their_own():
    from vlrf_b200.parts import get_part
    g = torch.Generator().manual_seed(3)
    r = lambda *s: torch.randn(*s, generator=g)   # noqa: E731
    d, H, n, mv = 16, 2, 3, 4
    mixer = get_part("mixer", "stabilized_memory")(r(6, d), r(6, d), r(8, d), r(8, d), r(2, d), r(2), r(2, d), r(2), r(8), r(d, 8), n_heads=H, dim=n, vdim=mv,
                                                   gate_cap=4.0, eps=1e-5)
    own_in, own_bias, own_out = mixer.in_weight.clone(), mixer.in_bias.clone(), mixer.out_weight.clone()
    ff = get_part("feed_forward", "routed_experts")(r(3, d), None, r(3, 5, d), r(3, 5, d), r(3, d, 5), top=1, shared=(r(6, d), r(6, d), r(d, 6), None),
                                                    scoring="sigmoid", weights_on="input")
    ff_in, ff_down = ff.in_weight.clone(), ff.out_weight.clone()
    block = get_part("block", "parallel_sublayers")(get_part("norm", "group_rmsnorm")(r(d), 1e-5, 2), mixer, ff)
    assert block.joint_in and block.joint_out and block.ff_at == 32
    assert torch.equal(block.in_weight[:32], own_in) and torch.equal(block.in_weight[32:32 + 15], ff_in) and not block.in_weight[47:].any()
    assert torch.equal(block.in_bias[:32], own_bias) and not block.in_bias[32:].any()
    assert torch.equal(block.out_weight, torch.cat([own_out, ff_down], 1))
    for t in (mixer.in_weight, ff.w_in, ff.shared[0]):
        assert t.untyped_storage().data_ptr() == block.in_weight.untyped_storage().data_ptr()
    for t in (mixer.out_weight, ff.shared[1]):
        assert t.untyped_storage().data_ptr() == block.out_weight.untyped_storage().data_ptr()
    assert torch.equal(ff.shared[0], ff_in[3:]) and ff.leading_rows(64) == 15 and ff.leading_rows(65) == 3


def test_weights_on_the_input_take_no_identity_experts():
    from vlrf_b200.parts import get_part
    w = torch.zeros
    with pytest.raises(ValueError, match="input"):
        get_part("feed_forward", "routed_experts")(w(4, 8), None, w(3, 5, 8), w(3, 5, 8), w(3, 8, 5), top=1, scoring="sigmoid", n_identity=1,
                                                   weights_on="input")


def test_sinusoid_frequencies_of_the_part_match_the_plain_ones():
    from vlrf_b200.parts import get_part
    part = get_part("position", "sinusoidal")(10, "cpu")
    want = plain.sinusoid(torch.tensor([3]), 10)[0]
    for i, f in enumerate(part.frequencies.tolist()):
        assert math.sin(3 * f) == pytest.approx(float(want[2 * i])) and math.cos(3 * f) == pytest.approx(float(want[2 * i + 1]))
    assert plain.sinusoid(torch.tensor([0]), 4)[0].tolist() == [0, 1, 0, 1]


def test_plain_attention_edges():
    mask = {"size": 4, "keep_first": 2}
    assert [j for j in range(10) if plain.visible(9, j, mask)] == [0, 1, 6, 7, 8, 9]
    assert [j for j in range(10) if plain.visible(9, j, {"size": 4})] == [6, 7, 8, 9]
    assert plain.slopes(2) == [2.0 ** -4, 2.0 ** -8] and plain.slopes(1) == [2.0 ** -8]
    # two keys of equal score: the farther one weighs e^(−slope) as much
    q = k = torch.zeros(2, 1, 2, dtype=torch.float64)
    v = torch.tensor([[[1.0]], [[0.0]]], dtype=torch.float64)
    out = plain.attend(q, k, v, 1.0, None, [0.5])
    assert float(out[1, 0, 0]) == pytest.approx(math.exp(-0.5) / (1 + math.exp(-0.5)))


def test_plain_recurrences_written_out():
    """Two tokens of each recurrence by hand, one head with a state of one number."""
    t = lambda *v: torch.tensor(v, dtype=torch.float64).view(-1, 1, 1)   # noqa: E731
    q, k, v = t(2.0, 3.0), t(5.0, 7.0), t(0.5, -1.0)
    assert plain.decayed_memory(q, k, v, t(0.9, 0.25)).flatten().tolist() == pytest.approx([2 * 2.5, 3 * (0.25 * 2.5 - 7.0)])
    beta = torch.tensor([[0.5], [0.1]], dtype=torch.float64)
    s1 = 5.0 * 0.5 * 0.5
    s2 = 0.25 * s1
    s2 += 7.0 * 0.1 * (-1.0 - 7.0 * s2)
    assert plain.delta_memory(q, k, v, t(0.9, 0.25), beta).flatten().tolist() == pytest.approx([2 * s1, 3 * s2])
    li, lf = torch.tensor([[-2.0], [1.0]], dtype=torch.float64), torch.tensor([[-0.5], [-0.25]], dtype=torch.float64)
    m1 = max(-0.5 + 0.0, -2.0)                                     # the maximum starts at 0: token 0 keeps −0.5, not −2
    s1, n1 = math.exp(-2.0 - m1) * 2.5, math.exp(-2.0 - m1) * 5.0
    m2 = max(-0.25 + m1, 1.0)
    a, b = math.exp(-0.25 + m1 - m2), math.exp(1.0 - m2)
    s2, n2 = a * s1 - b * 7.0, a * n1 + b * 7.0
    want = [2 * s1 / (max(abs(2 * n1), math.exp(-m1)) + 1e-6), 3 * s2 / (max(abs(3 * n2), math.exp(-m2)) + 1e-6)]
    assert plain.stabilized_memory(q, k, v, li, lf).flatten().tolist() == pytest.approx(want)


def test_plain_convolution_and_experts():
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=torch.float64)
    w = torch.tensor([[0.5, 3.0]], dtype=torch.float64)            # the last tap is the current token's
    s = lambda x: x / (1 + math.exp(-x))   # noqa: E731
    assert plain.short_convolution(u, w).flatten().tolist() == pytest.approx([s(3.0), s(6.5), s(13.0)])
    d = lambda x: torch.tensor([[x]], dtype=torch.float64)   # noqa: E731
    wts = {"p.router": torch.tensor([[1.0], [2.0]], dtype=torch.float64), "p.e0.gate": d(1.0), "p.e0.up": d(1.0), "p.e0.down": d(1.0),
           "p.e1.gate": d(1.5), "p.e1.up": d(2.0), "p.e1.down": d(-1.0)}
    sc = 1 / (1 + math.exp(-2.0))
    got = plain.routed_ff(d(1.0), wts, "p.", {"router": {"top": 1, "experts": 2}})
    assert float(got) == pytest.approx(-s(1.5 * sc) * 2.0 * sc)    # the weight acts on the input, inside the gate


def test_configurations_differ():
    sizes = [(c["width"], c["vocab"], len(c["layers"])) for c in MODELS.values()]
    assert len(set(sizes)) == len(sizes) and PEL_ODD["width"] % 8 != 0
