"""Each mechanism of the Vilodra design alone: the kernel against the plain function on inputs of its own — queries and keys of two
maps prepared and kept, differential attention at its edges, latent attention with windows, sinks and a factor by all three
kernels, the rotations with a factor on cosines and sines, the recurrence with a fixed decay over steps of every cut, the wide
read-out, the gate with a factor, renormalized routing and experts without a gate."""
import os
import types

import pytest
import torch
import torch.nn.functional as F

import plain_vilodra as plain
from test_kuvusun_kernels import paged, step_tables
from test_rakelorn_kernels import SLOTS, STEPS, close, dev, run_steps, step_ctx
from test_suposun_kernels import PagedKV

pytestmark = pytest.mark.gpu

DT = [torch.float32, torch.bfloat16]
F64 = torch.float64
TOTAL = [sum(s[i] for s in STEPS) for i in range(3)]


def tol(dt):
    return 2e-5 if dt == torch.float32 else 1.2e-2


def i32(v):
    return dev(torch.as_tensor(v), torch.int32)


# ---- differential attention -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt,t", [(torch.float32, 1e-4), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("H,G,n,m,rot,sc", [(4, 2, 16, 40, 8, (4.0, 1.0, 4.0, 64)), (3, 3, 13, 7, 6, None), (5, 1, 24, 24, 24, (2.0, 1.0, 2.0, 512)),
                                            (2, 1, 64, 16, 0, None), (20, 1, 8, 16, 4, None)])
def test_two_maps_prepared(H, G, n, m, rot, sc, dt, t):
    """Tokens of three sequences across block borders and far out: every map of every query and key head rotated by itself, a
    key head's maps side by side in the cache, values untouched; a second layer that writes no cache gets the same queries."""
    from vlrf_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 10 + n)
    positions, slot_of = [0, 1, 63, 64, 65, 1000, 4000], [0, 0, 1, 1, 1, 2, 2]
    T = len(positions)
    q, k, v = torch.randn(T, H * 2 * n, generator=g), torch.randn(T, G * 2 * n, generator=g), torch.randn(T, G * m, generator=g)
    wide = torch.full((T, q.shape[1] + k.shape[1] + v.shape[1] + 3), float("nan"))
    wide[:, 2:-1] = torch.cat([q, k, v], 1)
    wide = dev(wide)
    f = plain.frequencies({"base": 300.0, "dims": rot}) if rot else []
    if sc:
        f = plain.stretched(f, dict(zip(("factor", "low", "high", "original"), sc)))
    fr = dev(torch.tensor(f, dtype=F64).float()) if rot else None
    cache = PagedKV(3, 4096, G, 2 * n, m, dt)
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    qo = torch.full((T, H * 2 * n), float("nan"), dtype=dt, device="cuda")
    args = (fr, rot, qo, cache.k, cache.v, cache.table, i32(slot_of), i32(positions), T, H, G, n, m)
    ops.qkv_rope_append(wide[:, 2:-1], 0, H * 2 * n, (H + G) * 2 * n, *args, True, err, interleaved=True, maps=2)
    assert int(err.item()) == 0
    pos = torch.tensor(positions)
    turned = lambda x, heads: plain.rotate(x.double().view(T, heads * 2, n), pos, f).view(T, heads, 2 * n)   # noqa: E731
    close(qo.view(T, H, 2 * n), turned(q, H), t, "queries")
    kk, vv = turned(k, G), v.double().view(T, G, m)
    for i, (s, p) in enumerate(zip(slot_of, positions)):
        blk = int(cache.table[s, p // 64])
        close(cache.k[blk, :, p % 64], kk[i], t, f"keys of token {i}")
        close(cache.v[blk, :, p % 64], vv[i], t, f"values of token {i}")
    assert (~torch.isnan(cache.k.float())).sum().item() == T * G * 2 * n and (~torch.isnan(cache.v.float())).sum().item() == T * G * m
    before, first = cache.k.clone(), qo.clone()
    ops.qkv_rope_append(wide[:, 2:2 + q.shape[1]], 0, 0, 0, *args, False, err, interleaved=True, maps=2)
    assert torch.equal(first, qo) and torch.equal(torch.nan_to_num(before), torch.nan_to_num(cache.k))


def differential_case(H, G, n, m, window, lens, seed):
    """Random maps (bfloat16 values, exact in both dtypes).  For the last query of every sequence each map has a loud key of its own,
    through the first query head of each key/value head: map 1 the oldest visible one, map 2 one in the middle; with a window the
    key just outside it is louder still in both maps."""
    g = torch.Generator().manual_seed(seed)
    T = sum(lens)
    rd = lambda *shape: torch.randn(*shape, generator=g).bfloat16().double()   # noqa: E731
    q, k, v = rd(T, H, 2, n), rd(T, G, 2, n), rd(T, G, m)
    start = 0
    for length in lens:
        last, inside = start + length - 1, max(0, length - window) if window else 0
        for hk in range(G):
            for j, (place, loud) in enumerate(((inside, 5.0), (inside + (length - inside) // 2, 5.5))):
                unit = q[last, hk * (H // G), j] / float(q[last, hk * (H // G), j].norm())
                k[start + place, hk, j] = (loud * unit).bfloat16().double()
                if inside > 0:
                    k[start + inside - 1, hk, j] = (9.0 * unit).bfloat16().double()
        start += length
    return q, k, v


def plain_differential(q, k, v, lens, scale, window, lam, eps, factor):
    out, start = [], 0
    for length in lens:
        sl = slice(start, start + length)
        a = [plain.attend(q[sl, :, j], k[sl, :, j], v[sl], scale, window or None) for j in range(2)]
        out.append(plain.over_rms(a[0] - lam * a[1], eps) * factor)
        start += length
    return torch.cat(out)


LAM, FACTOR = 0.43, 0.6


def run_differential(q, k, v, lens, scale, window, eps, dt, tail, splits=None):
    """Everything is appended to a NaN-filled cache under a permuted block table; then the last `tail` tokens of every sequence
    (None: all of them, by the kernel that takes a warp per token and head) attend."""
    from vlrf_b200.csrc import ops
    from vlrf_b200.parts.context import Workspace
    T, H, _, n = q.shape
    G, m = v.shape[1], v.shape[2]
    slot_of = [s for s, length in enumerate(lens) for _ in range(length)]
    positions = [p for length in lens for p in range(length)]
    cache = PagedKV(len(lens), max(lens), G, 2 * n, m, dt)
    proj = dev(torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], dim=1), torch.float32)
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    qo = torch.full((T, H * 2 * n), float("nan"), dtype=dt, device="cuda")
    ops.qkv_rope_append(proj, 0, H * 2 * n, (H + G) * 2 * n, None, 0, qo, cache.k, cache.v, cache.table, i32(slot_of), i32(positions), T, H, G, n, m,
                        True, err, maps=2)
    if tail is None:
        out = torch.full((T, H * m), float("nan"), dtype=dt, device="cuda")
        ops.attention_window(qo, cache.k, cache.v, cache.table, i32(slot_of), i32(positions), out, T, H, G, n, m, scale, window, FACTOR, err,
                             second_map=(LAM, eps))
        rows = list(range(T))
    else:
        rows, seq_start, seq_pos0, start = [], [0], [], 0
        for length in lens:
            new = min(tail, length)
            rows += list(range(start + length - new, start + length))
            seq_start.append(seq_start[-1] + new)
            seq_pos0.append(length - new)
            start += length
        idx = torch.tensor(rows)
        ctx = types.SimpleNamespace(n_tokens=len(rows), n_seqs=len(lens), max_new=min(tail, max(lens)), max_context=max(lens), ws=Workspace("cuda"),
                                    dev_err=err, tok_slot=i32(torch.tensor(slot_of)[idx]), tok_pos=i32(torch.tensor(positions)[idx]),
                                    seq_slot=i32(torch.arange(len(lens))), seq_start=i32(seq_start), seq_pos0=i32(seq_pos0))
        wide = torch.full((len(rows), H * m + 4), float("nan"), dtype=dt, device="cuda")
        out = wide[:, 2:2 + H * m]
        if splits:
            os.environ["VLRF_B200_DECODE_SPLITS"] = str(splits)
        try:
            ops.attention_window_step(qo[idx.to("cuda")].contiguous(), cache.k, cache.v, cache.table, out, ctx, H, G, n, m, scale, window, FACTOR,
                                      second_map=(LAM, eps))
        finally:
            os.environ.pop("VLRF_B200_DECODE_SPLITS", None)
        assert torch.isnan(wide[:, :2].float()).all() and torch.isnan(wide[:, 2 + H * m:].float()).all()
    assert int(err.item()) == 0
    return out.reshape(len(rows), H, m), rows


@pytest.mark.parametrize("dt,t", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("H,G,n,m,window", [(4, 2, 16, 24, 0), (6, 2, 32, 64, 0), (3, 1, 24, 40, 50), (2, 2, 64, 128, 0), (5, 5, 40, 8, 64), (16, 1, 48, 96, 0),
                                            (1, 1, 128, 128, 0), (8, 2, 96, 32, 33), (5, 1, 12, 20, 0), (20, 1, 16, 16, 0), (3, 3, 13, 9, 7),
                                            (2, 1, 128, 64, 0), (2, 1, 160, 200, 0)])
def test_differential_attention_at_the_edges(H, G, n, m, window, dt, t):
    """Sequences of 1, 2, 64, 65, 129, 200 and 333 tokens in one step: as one prompt step (both kernels), as a later portion of 70, 3
    and 2 tokens, and as a decode step whose contexts are whole, cut in 2 and cut in 5 parts."""
    lens = [1, 2, 64, 65, 129, 200, 333]
    scale, eps = 0.9 * n ** -0.5 if n > 32 else 0.3, 1e-5
    q, k, v = differential_case(H, G, n, m, window, lens, n * 7 + m)
    want = plain_differential(q, k, v, lens, scale, window, LAM, eps, FACTOR)
    got, _ = run_differential(q, k, v, lens, scale, window, eps, dt, None)
    close(got, want, t, "a warp per token and head")
    for tail, splits in ((10 ** 6, None), (70, None), (3, None), (2, None), (1, 1), (1, 2), (1, 5)):
        got, rows = run_differential(q, k, v, lens, scale, window, eps, dt, tail, splits)
        close(got, want[torch.tensor(rows)], t, f"the last {tail} tokens, contexts in {splits} parts")


def test_the_second_map_and_a_far_key_would_show():
    """On those inputs: exchanging the maps, another factor, leaving out the oldest key, or moving a window by one changes the expected
    result of the last queries by far more than the kernels' tolerance."""
    lens, last = [200, 333], [199, 532]
    for window in (0, 50):
        q, k, v = differential_case(4, 2, 16, 24, window, lens, 3)
        want = plain_differential(q, k, v, lens, 0.3, window, LAM, 1e-5, FACTOR)
        others = [plain_differential(q.flip(2), k.flip(2), v, lens, 0.3, window, LAM, 1e-5, FACTOR),
                  plain_differential(q, k, v, lens, 0.3, window, 0.5 * LAM, 1e-5, FACTOR),
                  plain_differential(q, k, v, lens, 0.3, window - 1 if window else 332, LAM, 1e-5, FACTOR)]
        if window:
            others.append(plain_differential(q, k, v, lens, 0.3, window + 1, LAM, 1e-5, FACTOR))
        for i, other in enumerate(others):
            rows = last if window or i < 2 else last[1:]
            assert float((other[rows] - want[rows]).abs().max() / want.abs().max()) > 0.1, (window, i)


@pytest.mark.parametrize("dt", DT)
def test_the_heads_norm_has_its_eps_inside_the_root(dt):
    """Values so small that eps decides: what is left is the difference times the factor over sqrt(eps), nearly."""
    q, k, v = differential_case(2, 1, 16, 32, 0, [40], 9)
    v = (v * 1e-4).bfloat16().double()
    want = plain_differential(q, k, v, [40], 0.3, 0, LAM, 1e-5, FACTOR)
    assert float(want.abs().max()) < 0.1
    for tail in (None, 40, 1):
        got, rows = run_differential(q, k, v, [40], 0.3, 0, 1e-5, dt, tail, 1)
        close(got, want[torch.tensor(rows)], 3e-5 if dt == torch.float32 else 3e-2, f"tail {tail}")


# ---- latent attention -------------------------------------------------------------------------------------------------------
def one_query(q, rows, C, scale, pos, window, sink, factor):
    """q [H, C + R] at `pos` over rows [n, C + R]: the plain attention of the last of pos + 1 tokens."""
    first = max(0, pos - window + 1) if window else 0
    s = (rows[first:pos + 1].double() @ q.double().T) * scale                       # [keys, H]
    s = torch.cat([s, sink.double()[None]], 0)
    return (torch.softmax(s, 0)[:-1].T @ rows[first:pos + 1, :C].double()) * factor


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("C,R,H,splits", [(64, 16, 3, None), (64, 16, 3, 1), (64, 16, 3, 4), (96, 32, 20, None), (96, 32, 20, 2), (40, 8, 5, None),
                                          (256, 16, 16, 3), (36, 6, 2, None), (512, 64, 4, None)])
def test_latent_attention_with_windows_and_sinks(C, R, H, splits, dt, monkeypatch):
    """Windows whose edge falls inside a tile, on a tile's and on a block's border (and none), sinks from next to nothing to above every
    score, a factor on the result; per head the oldest visible row is made loud, and the row before it louder still."""
    from vlrf_b200.csrc import ops
    if splits is not None:
        monkeypatch.setenv("VLRF_B200_DECODE_SPLITS", str(splits))
    g = torch.Generator().manual_seed(C + H)
    n, D, scale, factor = 420, C + R, 0.3, 0.55
    order = [5, 2, 6, 0, 4, 1, 3]
    if splits is None:
        positions, runs = list(range(130, 130 + 71)) + [0, 1] + [419], [71, 2, 1]                # portions of a prompt
    else:
        positions = [419, 0, 31, 32, 63, 64, 65, 300, 1, 127, 128]                               # single tokens
        runs = [1] * len(positions)
    sink = torch.linspace(-6.0, 9.0, H) if H > 1 else torch.tensor([2.0])
    for window in (0, 33, 64, 100):
        rows = torch.randn(n, D, generator=g).to(torch.bfloat16)
        qp = torch.randn(len(positions), H, D, generator=g) * (0.5 / D ** 0.5)
        for i, p in enumerate(positions):
            inside = max(0, p - window + 1) if window else 0
            for h in range(H):
                key = rows[inside].float()
                qp[i, h] += key * (6.0 / (scale * float(key @ key)))
                if inside:
                    out = rows[inside - 1].float()
                    qp[i, h] += out * (9.0 / (scale * float(out @ out)))
        qp = qp.to(torch.bfloat16)
        want = torch.stack([one_query(qp[i], rows, C, scale, p, window, sink, factor) for i, p in enumerate(positions)])
        if window:                                     # (the edge would show)
            other = one_query(qp[0], rows, C, scale, positions[0], window + 1, sink, factor)
            assert float((other - want[0]).abs().max() / want.abs().max()) > 0.1
        cache, table = paged(7, order, D, dt)
        for b in range(7):
            cache[order[b], :min(64, n - 64 * b)] = rows[64 * b:64 * b + 64].to(dt).cuda()
        ctx = step_tables(positions, runs)
        err = torch.zeros(1, dtype=torch.int32, device="cuda")
        for use in (ctx, None):
            out = torch.full((len(positions), H * C), float("nan"), dtype=dt, device="cuda")
            ops.attention_latent(qp.view(len(positions), -1).to(dt).cuda(), cache, C, R, table, i32([1] * len(positions)), i32(positions), out,
                                 len(positions), H, scale, window, err, ctx=use, sink=dev(sink), out_scale=factor)
            assert int(err.item()) == 0
            close(out.view(len(positions), H, C), want, 2e-5 if dt == torch.float32 else 1.2e-2, f"window {window}, step tables {use is not None}")


@pytest.mark.parametrize("dim,R,vdim,H,window", [(16, 16, 24, 2, 40), (48, 16, 64, 3, 64), (64, 32, 128, 2, 0), (64, 0, 48, 2, 33), (128, 64, 16, 1, 1),
                                                 (96, 32, 8, 2, 100), (192, 64, 128, 1, 65), (16, 16, 40, 4, 500)])
def test_prompt_attention_over_plain_rows_with_windows_and_sinks(dim, R, vdim, H, window):
    """Sequences of 1 to 200 tokens; per query the oldest visible key is loud and the one before it louder still."""
    from vlrf_b200.csrc import ops
    g = torch.Generator().manual_seed(dim + R + window)
    lens = [1, 70, 64, 200, 33, 65]
    T, bf, scale, factor = sum(lens), torch.bfloat16, 0.29, 0.7
    kn, v = torch.randn(T, H, dim, generator=g).to(bf), torch.randn(T, H, vdim, generator=g).to(bf)
    kr = torch.randn(T, R, generator=g).to(bf)
    q = torch.randn(T, H, dim + R, generator=g) * 0.05
    starts = [sum(lens[:i]) for i in range(len(lens) + 1)]
    for a, b in zip(starts, starts[1:]):
        for i in range(b - a):
            inside = max(0, i - window + 1) if window else 0
            for h in range(H):
                for place, loud in ((inside, 5.0), (inside - 1, 8.0)):
                    if place >= 0:
                        key = torch.cat([kn[a + place, h], kr[a + place]]).float()
                        q[a + i, h] += key * (loud / (scale * float(key @ key)))
    q = q.to(bf)
    sink = torch.linspace(4.0, -3.0, H)
    full = torch.cat([kn, kr[:, None].expand(T, H, R)], -1).double()
    want = torch.cat([plain.attend(q[a:b].double(), full[a:b], v[a:b].double(), scale, window or None, sink.double()) for a, b in zip(starts, starts[1:])])
    out = torch.full((T, H * vdim), float("nan"), dtype=bf, device="cuda")
    ops.attention_rows(dev(q[..., :dim].reshape(T, -1)), dev(q[..., dim:].reshape(T, -1)) if R else None, dev(kn.view(T, -1)), dev(kr) if R else None,
                       dev(v.view(T, -1)), i32(starts), out, len(lens), max(lens), H, dim, R, vdim, scale, window=window, sink=dev(sink), out_scale=factor)
    close(out.view(T, H, vdim), want * factor, 1.2e-2, "rows")


@pytest.mark.parametrize("dt", DT)
def test_rotations_with_a_factor_on_cosines_and_sines(dt):
    """A token's cache row and the queries' rows with scaled frequencies and the magnitude that goes with them."""
    from vlrf_b200.csrc import ops
    from vlrf_b200.parts import RotaryPositions
    H, dim, C, R, T = 3, 12, 20, 16, 6
    sc = (4.0, 64, 16.0, 1.0)
    part = RotaryPositions(400.0, R, "cuda", pairing="interleaved", yarn=sc)
    f, mag = plain.yarn(plain.frequencies({"base": 400.0, "dims": R}), dict(zip(("factor", "original", "fast", "slow"), sc)), 400.0, R)
    assert part.inv_freq.tolist() == pytest.approx(f, rel=1e-6) and part.magnitude == pytest.approx(mag) and mag > 1.1
    g = torch.Generator().manual_seed(2)
    positions = torch.tensor([0, 1, 63, 64, 300, 1000])
    q, proj = torch.randn(T, H, dim + R, generator=g), torch.randn(T, C + R, generator=g)
    w = 1 + 0.2 * torch.randn(C, generator=g)
    qn, qp = torch.zeros(T, H * dim, dtype=dt, device="cuda"), torch.zeros(T, H * (C + R), dtype=dt, device="cuda")
    ops.latent_q_rows(dev(q.view(T, -1)), H, dim, R, part.inv_freq, R, i32(positions), qn, qp, C, T, interleaved=True, magnitude=part.magnitude)
    t = 6e-5 if dt == torch.float32 else 6e-3
    close(qn.view(T, H, dim), q[..., :dim], t, "unrotated")
    close(qp.view(T, H, C + R)[..., C:], plain.rotate(q[..., dim:].double(), positions, f, mag), t, "rotated")
    cache, table = paged(16, list(range(15, -1, -1)), C + R, dt)
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    ops.latent_append(dev(proj), C, R, dev(w), 1e-5, part.inv_freq, R, cache, table, i32([1] * T), i32(positions), T, err, interleaved=True,
                      magnitude=part.magnitude)
    want = torch.cat([plain.over_rms(proj[:, :C].double(), 1e-5) * w.double(), plain.rotate(proj[:, None, C:].double(), positions, f, mag)[:, 0]], -1)
    for i, p in enumerate(positions.tolist()):
        close(cache[15 - p // 64, p % 64], want[i], t, f"row at {p}")
    assert int(err.item()) == 0


# ---- the recurrence ---------------------------------------------------------------------------------------------------------
#: (heads, rows, columns, columns a lane): rows around every size the kernel is instantiated for, columns that fill, cross and leave
#: over a CTA's, sizes that are no multiples of 4
SHAPES = [(2, 16, 16, 0), (3, 13, 22, 0), (4, 48, 32, 1), (2, 64, 40, 2), (1, 128, 128, 4), (6, 33, 7, 4), (2, 160, 24, 0), (1, 512, 20, 0), (2, 72, 130, 2),
          (1, 4, 1, 1), (2, 256, 33, 2), (5, 64, 64, 0), (3, 128, 64, 0)]


def draw_memory(H, K, V, totals, seed):
    g = torch.Generator().manual_seed(seed)
    rd = lambda *s: torch.randn(*s, generator=g).double()   # noqa: E731
    decay = torch.tensor([[0.6, 0.9, 0.99, 0.3, 0.999, 1.0][h % 6] for h in range(H)], dtype=torch.float32).double()
    return [dict(q=rd(n, H, K), k=rd(n, H, K), v=rd(n, H, V)) for n in totals], decay


def plain_memory(d, decay, act):
    f = F.silu if act == "silu" else (lambda x: x)
    return plain.fading_memory(f(d["q"]), f(d["k"]), f(d["v"]), decay)


def memory_step(d, decay, state, ctx, act):
    """One step's recurrence from [q | k | v] side by side in wider rows (an odd number of columns ahead of them now and then)."""
    from vlrf_b200.csrc import ops
    T, H, K = d["q"].shape
    V = d["v"].shape[2]
    lead = 4 if (K + V) % 2 == 0 else 3
    wide = dev(torch.cat([torch.full((T, lead), float("nan"), dtype=F64)] + [d[n].reshape(T, -1) for n in "qkv"], 1), torch.float32)
    q, k, v = wide[:, lead:lead + H * K], wide[:, lead + H * K:lead + 2 * H * K], wide[:, lead + 2 * H * K:]
    y = torch.full((T, H * V), float("nan"), device="cuda")
    ops.matrix_state_scan("fixed", q, k, v, state, ctx, y, H, H, K, V, q_scale=1.0, decay=dev(decay, torch.float32), input_act=act)
    return y.view(T, H, V)


@pytest.mark.parametrize("act", ["silu", "none"])
@pytest.mark.parametrize("H,K,V,columns", SHAPES)
def test_fixed_memory_over_steps(H, K, V, columns, act):
    from vlrf_b200.csrc import call_host
    warps = {0: 0, 1: 2, 2: 1, 4: 4}[columns]
    seqs, decay = draw_memory(H, K, V, TOTAL, K * 7 + V)
    want = [plain_memory(d, decay, act) for d in seqs]
    state = torch.full((8, 2, -(-H * K * V // 4) * 4), float("nan"), device="cuda")
    for s in SLOTS:
        state[s] = 0.0
    pad = {name: torch.full((1,) + tuple(t.shape[1:]), float("nan"), dtype=F64) for name, t in seqs[0].items()}

    def fn(ctx, runs):
        rows = {name: torch.cat([seqs[SLOTS.index(s)][name][p0:p0 + m] if s >= 0 else pad[name] for s, p0, m in runs]) for name in pad}
        out = memory_step(rows, decay, state, ctx, act)
        if ctx.max_new == 1:                               # a step of single tokens may run twice
            assert torch.equal(torch.nan_to_num(memory_step(rows, decay, state, ctx, act)), torch.nan_to_num(out))
        return out

    call_host("vlrf_matrix_state_force", columns, warps)
    try:
        got = run_steps(fn, [0, 0, 0], 8, None, None)
    finally:
        call_host("vlrf_matrix_state_force", 0, 0)
    for i in range(3):
        close(got[i], want[i], 2e-5, f"sequence {i}")
    assert torch.isnan(state[[s for s in range(8) if s not in SLOTS]]).all(), "a state of another slot was written"


@pytest.mark.parametrize("lens", [[15, 16, 17, 31, 32, 33, 63, 64, 65, 66, 127, 128, 129], [700, 1, 333]])
def test_fixed_memory_at_the_batches_edges(lens):
    """Prompts that end at, before and behind the edges of staged batches and chunks, in one step, then one more token each."""
    H, K, V = 3, 64, 48
    seqs, decay = draw_memory(H, K, V, [n + 1 for n in lens], 9)
    state = torch.zeros(len(lens), 2, H * K * V, device="cuda")
    for upto in (0, 1):
        part = [(0, n) if upto == 0 else (n, n + 1) for n in lens]
        ctx, _ = step_ctx([(s, a, b - a) for s, (a, b) in enumerate(part)])
        y = memory_step({name: torch.cat([d[name][a:b] for d, (a, b) in zip(seqs, part)]) for name in "qkv"}, decay, state, ctx, "silu").cpu()
        at = 0
        for s, (a, b) in enumerate(part):
            close(y[at:at + b - a], plain_memory(seqs[s], decay, "silu")[a:b], 2e-5, f"sequence of {lens[s]}, {upto}")
            at += b - a


def test_fixed_memory_carries_a_far_token():
    """700 tokens, then three single ones: what the first token alone wrote under a key that only the last ones ask for comes back
    faded by the decay and nothing else; other keys are loud."""
    H, K, V, n = 2, 24, 20, 703
    (d,), _ = draw_memory(H, K, V, [n], 5)
    decay = torch.tensor([0.9995, 0.999], dtype=torch.float32).double()
    d["k"][0, :, 0], d["k"][1:, :, 0], d["q"][700:] = 4.0, 0.0, 0.0
    d["q"][700:, :, 0] = 3.0
    d["v"][0] = 5.0
    want = plain_memory(d, decay, "none")
    assert float((want[702, 0, 0] - 60.0 * decay[0] ** 702).abs()) < 1e-9
    state = torch.zeros(2, 2, H * K * V, device="cuda")
    got = []
    for p0, m in ((0, 700), (700, 1), (701, 1), (702, 1)):
        ctx, _ = step_ctx([(1, p0, m)])
        got.append(memory_step({name: t[p0:p0 + m] for name, t in d.items()}, decay, state, ctx, "none"))
    close(torch.cat(got), want, 5e-5, "all")
    close(torch.cat(got)[700:], want[700:], 5e-5, "the far token")


def test_fixed_memory_of_seventy_single_tokens():
    H, K, V = 3, 32, 48
    seqs, decay = draw_memory(H, K, V, [4] * 70, 9)
    state = torch.zeros(70, 2, H * K * V, device="cuda")
    got = [[] for _ in seqs]
    for t in range(4):
        ctx, _ = step_ctx([(s, t, 1) for s in range(70)])
        y = memory_step({name: torch.cat([d[name][t:t + 1] for d in seqs]) for name in "qkv"}, decay, state, ctx, "silu")
        for s in range(70):
            got[s].append(y[s:s + 1])
    for s in range(70):
        close(torch.cat(got[s]), plain_memory(seqs[s], decay, "silu"), 2e-5, f"sequence {s}")


def chunk_step(d, decay, state, ctx, scale=1.0):
    """One step in chunks from bfloat16 rows [q | k | v]; the scratch is NaN before."""
    from vlrf_b200.csrc import ops
    T, H, K = d["q"].shape
    V = d["v"].shape[2]
    n = H * (2 * K + V)
    wide = dev(torch.cat([torch.full((T, 8), float("nan"), dtype=F64)] + [d[x].reshape(T, -1) for x in "qkv"], 1), torch.bfloat16)[:, 8:]
    ctx.ws.get("fixed_state_chunks", (T // 64 + ctx.n_seqs) * H, K * V, torch.float32).fill_(float("nan"))
    y = torch.full((T, H * V), float("nan"), device="cuda")
    assert wide.shape[1] == n and ops.fixed_state_chunks_takes(torch.bfloat16, types.SimpleNamespace(max_new=64, n_tokens=T, n_seqs=ctx.n_seqs), H, K, V, state.shape[2])
    ops.fixed_state_chunks(wide[:, :H * K], wide[:, H * K:2 * H * K], wide[:, 2 * H * K:], dev(decay, torch.float32), state, ctx, y, H, K, V, q_scale=scale)
    return y.view(T, H, V)


@pytest.mark.parametrize("H,K,V", [(2, 16, 16), (3, 24, 40), (1, 128, 128), (5, 64, 64), (2, 72, 136), (1, 256, 32), (6, 8, 8), (3, 48, 264), (2, 136, 96)])
def test_fixed_memory_in_chunks(H, K, V):
    """Nine sequences at and around the chunks' edges in one step, twice (the second step goes on from states at odd and even
    positions), a padding sequence among them; then the token-by-token kernel goes on from the states that the chunks left."""
    from vlrf_b200.parts.context import Workspace
    lens = [1, 63, 64, 65, 127, 128, 129, 200, 33]
    more = [64, 1, 130, 2, 65, 63, 7, 128, 96]
    seqs, decay = draw_memory(H, K, V, [a + b + 1 for a, b in zip(lens, more)], K + V)
    seqs = [{name: t.bfloat16().double() for name, t in d.items()} for d in seqs]
    want = [plain_memory(d, decay, "none") * 0.8 for d in seqs]
    slots = [7, 3, 0, 9, 5, 1, 2, 8, 4]
    state = torch.full((11, 2, H * K * V), float("nan"), device="cuda")
    state[slots] = 0.0
    pad = {name: torch.full((1,) + tuple(t.shape[1:]), float("nan"), dtype=F64) for name, t in seqs[0].items()}
    done = [0] * len(lens)
    for step, news in enumerate((lens, more, [1] * len(lens))):
        ctx, runs = step_ctx([(s, p, n) for s, p, n in zip(slots, done, news)], pad_rows=(2,))
        ctx.ws = Workspace("cuda")
        rows = {name: torch.cat([seqs[slots.index(s)][name][p:p + n] if s >= 0 else pad[name] for s, p, n in runs]) for name in pad}
        if step < 2:
            y = chunk_step(rows, decay, state, ctx, 0.8)
        else:
            y = memory_step(rows, decay, state, ctx, "none") * 0.8
        at = 0
        for s, p, n in runs:
            if s >= 0:
                i = slots.index(s)
                close(y[at:at + n], want[i][p:p + n], 1e-4, f"step {step}, sequence {i}")
            at += n
        done = [a + n for a, n in zip(done, news)]
    assert torch.isnan(state[[6, 10]]).all(), "a state of another slot was written"


def test_fixed_memory_in_chunks_carries_a_far_token():
    """What the first of 1,500 tokens wrote under a key that only the last ones ask for."""
    from vlrf_b200.parts.context import Workspace
    H, K, V, n = 2, 24, 24, 1500
    (d,), _ = draw_memory(H, K, V, [n], 5)
    decay = torch.tensor([0.9995, 0.998], dtype=torch.float32).double()
    d["k"][0, :, 0], d["k"][1:, :, 0], d["q"][n - 3:] = 4.0, 0.0, 0.0
    d["q"][n - 3:, :, 0], d["v"][0] = 3.0, 5.0
    d = {name: t.bfloat16().double() for name, t in d.items()}
    want = plain_memory(d, decay, "none")
    state = torch.zeros(2, 2, H * K * V, device="cuda")
    ctx, _ = step_ctx([(1, 0, n)])
    ctx.ws = Workspace("cuda")
    got = chunk_step(d, decay, state, ctx)
    close(got, want, 1e-4, "all")
    close(got[n - 3:], want[n - 3:], 1e-4, "the far token")


@pytest.mark.parametrize("M,N,K", [(70, 96, 64), (300, 200, 128), (129, 37, 72), (2000, 640, 256)])
def test_a_product_with_silu_in_its_epilogue(M, N, K):
    from vlrf_b200.csrc import KernelError, ops
    g = torch.Generator().manual_seed(M)
    x, w = torch.randn(M, K, generator=g).bfloat16(), (3 * torch.randn(N, K, generator=g) / K ** 0.5).bfloat16()
    want = F.silu(x.double() @ w.double().T)
    for od, t in ((torch.bfloat16, 5e-3), (torch.float32, 1e-5)):
        out = torch.full((M, N), float("nan"), dtype=od, device="cuda")
        ops.linear(dev(x), dev(w), None, out, act="silu")
        close(out, want, t, f"to {od}")
    big = torch.full((M, K), 60.0).bfloat16()              # (both ends: sums of some thousand, and of minus some thousand)
    out = torch.zeros(M, N, dtype=torch.bfloat16, device="cuda")
    ones = torch.ones(N, K).bfloat16()
    ones[::2] = -1.0
    ops.linear(dev(big), dev(ones), None, out, act="silu")
    assert float(out[:, ::2].float().abs().max()) == 0.0
    close(out[:, 1::2], (60.0 * K * torch.ones(M, N // 2)).double(), 5e-3, "large")
    with pytest.raises(KernelError, match="epilogue"):
        ops.linear(dev(x[:8]), dev(w), None, out[:8], act="silu")


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("H,V", [(1, 700), (1, 1024), (1, 2048), (1, 513), (2, 3000), (1, 8192), (1, 9001), (3, 516)])
def test_the_read_out_of_wide_rows(H, V, dt):
    """Rows of all heads normed together, a CTA each: widths held in registers by 1, 2, 4 and 8 quads a thread, and others."""
    from vlrf_b200.csrc import ops
    T, eps = 11, 1e-5
    g = torch.Generator().manual_seed(V)
    y, gate, w = torch.randn(T, H, V, generator=g), torch.randn(T, H * V + 6, generator=g) * 3, 1.0 + 0.3 * torch.randn(H * V, generator=g)
    y[3] *= 1e-5                                           # (so small that eps decides)
    want = plain.over_rms(y.double(), eps) * w.double().view(H, V) * torch.sigmoid(gate[:, 4:4 + H * V].double().view(T, H, V)) * 0.7
    wide = torch.full((T + 1, H * V + 8), float("nan"), dtype=dt, device="cuda")
    gd = dev(gate)
    ops.head_rows(dev(y.reshape(T, -1)), dev(w), gd[:, 4:4 + H * V], "sigmoid", wide[:, 4:4 + H * V], T, H, V, eps, 0.7)
    close(wide[:T, 4:4 + H * V].float().view(T, H, V), want, tol(dt), "read-out")
    close(wide[3, 4:4 + H * V].float().view(H, V), want[3], tol(dt), "the small row")
    assert torch.isnan(wide[:, :4].float()).all() and torch.isnan(wide[:, 4 + H * V:].float()).all() and torch.isnan(wide[T].float()).all()


# ---- feed-forwards ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("cols", [64, 30])
def test_a_gate_with_a_factor(cols):
    from vlrf_b200.csrc import KernelError, ops
    g = torch.Generator().manual_seed(cols)
    a, b = torch.randn(9, 2 * cols, generator=g), None
    want = lambda x, y: F.silu(x.double()) * y.double() * 0.37   # noqa: E731
    ad = dev(a)
    for od in DT:                                          # float32 gate and values
        out = torch.zeros(9, cols, dtype=od, device="cuda")
        ops.gate_mul(ad[:, :cols], ad[:, cols:], out, "silu", 9, cols, factor=0.37)
        close(out, want(a[:, :cols], a[:, cols:]), 2e-6 if od == torch.float32 else 5e-3, f"to {od}")
    ah = a.bfloat16()
    out = torch.zeros(9, cols, dtype=torch.bfloat16, device="cuda")
    hd = dev(ah)
    ops.gate_mul(hd[:, :cols], hd[:, cols:], out, "silu", 9, cols, factor=0.37)
    close(out, want(ah[:, :cols], ah[:, cols:]), 5e-3, "bfloat16")
    with pytest.raises(KernelError, match="factor"):
        ops.gate_mul(ad[:, :2], ad[:, :cols], ad[:, :cols], "silu", 9, cols, per=cols // 2, factor=0.5)


@pytest.mark.parametrize("E,top", [(5, 2), (16, 1), (3, 3), (40, 6), (70, 4), (130, 8), (1, 1)])
def test_router_with_renormalized_scores(E, top):
    from vlrf_b200.csrc import ops
    g = torch.Generator().manual_seed(E)
    T = 33
    z = (torch.randn(T, E, generator=g) * 2).double().float()
    slot = torch.zeros(T, dtype=torch.int32)
    slot[7] = -1
    ids = torch.zeros(T, top, dtype=torch.int32, device="cuda")
    rank, wts, counts = torch.zeros_like(ids), torch.zeros(T, top, device="cuda"), torch.zeros(E, dtype=torch.int32, device="cuda")
    for scoring in ("softmax", "sigmoid"):
        counts.zero_()
        ops.moe_route_scored(dev(z), E, top, 1, 1, 0, 1.9, torch.zeros(E, device="cuda"), dev(slot), ids, wts, rank, counts, T, scoring=scoring,
                             renormalize=True)
        s = torch.softmax(z.double(), -1) if scoring == "softmax" else torch.sigmoid(z.double())
        order = torch.sort(s, dim=-1, descending=True, stable=True)
        live = [t for t in range(T) if t != 7]
        assert ids.cpu()[live].tolist() == order.indices[live, :top].tolist() and ids.cpu()[7].tolist() == [-1] * top
        chosen = order.values[:, :top]
        close(wts[live], (chosen / chosen.sum(-1, keepdim=True) * 1.9)[live], 2e-6, scoring)
        if top > 1 and E > top:
            assert float((chosen.sum(-1) - 1.0).abs().max()) > 0.05          # (without renormalizing it would show)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("width,E,top,ff,T", [(64, 5, 2, 40, 37), (96, 4, 1, 32, 9), (100, 3, 3, 28, 70), (64, 6, 4, 48, 130), (128, 8, 2, 64, 1)])
def test_experts_without_a_gate_and_with_renormalized_scores(width, E, top, ff, T, dt):
    """The whole part against the plain one, on choices that lie apart; relu² in place of the exact GELU would differ."""
    from vlrf_b200.parts import get_part
    from vlrf_b200.parts.context import Workspace
    g = torch.Generator().manual_seed(width + E)
    rd = lambda *s: (torch.randn(*s, generator=g) / s[-1] ** 0.5).bfloat16()   # noqa: E731
    h = torch.randn(T, width, generator=g).bfloat16()
    h[:, :E] = torch.stack([torch.randperm(E, generator=g) for _ in range(T)]).bfloat16()
    w = {"r.router": (0.5 * torch.eye(E, width)).bfloat16()}
    for e in range(E):
        w[f"r.e{e}.up"], w[f"r.e{e}.down"] = 2 * rd(ff, width), rd(width, ff)
    ml = {"router": {"top": top, "experts": E, "scale": 1.3}}
    want = plain.routed_ff(h.double(), {n: t.double() for n, t in w.items()}, "r.", ml)
    stack = lambda n: dev(torch.stack([w[f"r.e{e}.{n}"] for e in range(E)]), dt)   # noqa: E731
    ctx, _ = step_ctx([(0, 0, T)])
    ctx.ws, ctx.act_dtype = Workspace("cuda"), dt
    for act, same in (("gelu_erf", True), ("relu2", False)):
        part = get_part("feed_forward", "routed_experts")(dev(w["r.router"], dt), None, None, stack("up"), stack("down"), top=top, scoring="softmax_all",
                                                          renormalize=True, weight_scale=1.3, activation=act)
        x = dev(torch.ones(T, width))
        part.forward(dev(h, dt), x, ctx)
        if same:
            close(x - 1.0, want, tol(dt), "experts")
        else:
            assert float((x.double().cpu() - 1.0 - want).abs().max() / want.abs().max()) > 0.1
