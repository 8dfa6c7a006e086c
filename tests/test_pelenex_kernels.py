"""Each mechanism of the Pelenex design alone: the kernel against the plain function on inputs of its own — the three
recurrences over steps of every cut (both copies of their states, other slots full of NaN, padding rows) and over long
prompts, the convolution with its unit norms and kept inputs, the low-rank decays and gates, the read-out of a head, the
pair of normed outputs, attention with distance slopes at its edges, sinusoidal positions, expert weights on the inputs."""
import os
import types

import pytest
import torch
import torch.nn.functional as F

import plain_pelenex as plain
from test_rakelorn_kernels import SLOTS, STEPS, close, dev, run_steps, step_ctx
from test_suposun_kernels import PagedKV

pytestmark = pytest.mark.gpu

DT = [torch.float32, torch.bfloat16]
F64 = torch.float64
TOTAL = [sum(s[i] for s in STEPS) for i in range(3)]


def tol(dt):
    return 2e-5 if dt == torch.float32 else 1.2e-2


#: (heads, query/key heads, rows, columns, columns a lane): rows around every size the kernel is instantiated for, columns
#: that fill, cross and leave over a CTA's, sizes that are no multiples of 4
SHAPES = [(2, 1, 16, 16, 0), (3, 3, 13, 22, 0), (4, 2, 48, 32, 1), (2, 2, 64, 40, 2), (1, 1, 128, 128, 4), (6, 3, 33, 7, 4), (2, 2, 160, 24, 0),
          (1, 1, 512, 20, 0), (2, 1, 72, 130, 2), (1, 1, 4, 1, 1), (2, 2, 256, 33, 2)]


def draw_recurrence(kind, H, G, K, V, totals, seed):
    """Per sequence float64 inputs of a recurrence; keys and values of size 1, decays from forgetful to nearly none."""
    g = torch.Generator().manual_seed(seed)
    rd = lambda *s: torch.randn(*s, generator=g, dtype=F64)   # noqa: E731
    out = []
    for n in totals:
        d = dict(q=rd(n, G, K), k=rd(n, G, K), v=rd(n, H, V), decay=torch.sigmoid(2.0 + 2.0 * rd(n, H, K)), s0=rd(n, H), s1=rd(n, H) + 2.0)
        if kind == "delta":
            d["q"], d["k"] = plain.unit(d["q"]), plain.unit(d["k"])
            d["s1"] = (d["q"] * d["k"]).sum(-1)
        if kind == "stabilized":
            d["s0"] = 3.0 * d["s0"]
        out.append({name: t.float().double() for name, t in d.items()})
    return out


def plain_recurrence(kind, d, H, G, K, cap):
    share = [h // (H // G) for h in range(H)]
    q, k = d["q"][:, share] * K ** -0.5, d["k"][:, share]
    if kind == "decayed":
        return plain.decayed_memory(q, k, d["v"], d["decay"])
    if kind == "delta":
        return plain.delta_memory(q, k, d["v"], d["decay"], torch.sigmoid(d["s0"]))
    return plain.stabilized_memory(q, k, d["v"], cap * torch.tanh(d["s0"] / cap), F.logsigmoid(cap * torch.tanh(d["s1"] / cap)))


def scan(kind, rows, state, ctx, H, G, K, V, cap):
    """One step's recurrence from [q | k | v | decay | s0 | s1] side by side in wider rows (an odd column ahead of them, so that
    shapes that could be copied in quads sometimes are and sometimes are not)."""
    from vlrf_b200.csrc import ops
    parts = [rows["q"].reshape(-1, G * K), rows["k"].reshape(-1, G * K), rows["v"].reshape(-1, H * V), rows["decay"].reshape(-1, H * K),
             rows["s0"], rows["s1"]]
    lead = 4 if (K + V) % 2 == 0 else 3
    wide = dev(torch.cat([torch.full((parts[0].shape[0], lead), float("nan"), dtype=F64)] + parts, dim=1), torch.float32)
    at, cols = lead, []
    for p in parts:
        cols.append(wide[:, at:at + p.shape[1]])
        at += p.shape[1]
    q, k, v, decay, s0, s1 = cols
    T = ctx.n_tokens
    y = torch.full((T, H * V), float("nan"), device="cuda")
    den = torch.full((T, 2 * H), float("nan"), device="cuda")
    ops.matrix_state_scan(kind, q, k, v, state, ctx, y, H, G, K, V, q_scale=K ** -0.5, decay=decay if kind != "stabilized" else None,
                          s0=s0 if kind != "decayed" else None, s1=s1 if kind != "decayed" else None, cap=cap,
                          den=den if kind == "stabilized" else None)
    y = y.view(T, H, V)
    if kind == "stabilized":
        den = den.view(T, H, 2)
        y = y / (torch.maximum(den[..., 0].abs(), den[..., 1]) + 1e-6)[..., None]
    return y


def state_numbers(kind, H, K, V):
    return H * (V + 1) * (K + 1) if kind == "stabilized" else H * K * V


@pytest.mark.parametrize("H,G,K,V,columns", SHAPES)
@pytest.mark.parametrize("kind", ["decayed", "delta", "stabilized"])
def test_recurrence_over_steps(kind, H, G, K, V, columns):
    from vlrf_b200.csrc import call_host
    warps = {0: 0, 1: 2, 2: 1, 4: 4}[columns]
    if kind != "delta":
        G = H
    seqs = draw_recurrence(kind, H, G, K, V, TOTAL, K * 7 + V)
    want = [plain_recurrence(kind, d, H, G, K, 6.0) for d in seqs]
    n = -(-state_numbers(kind, H, K, V) // 4) * 4
    state = torch.full((8, 2, n), float("nan"), device="cuda")
    for s in SLOTS:
        state[s] = 0.0
    pad = {name: torch.full((1,) + tuple(t.shape[1:]), float("nan"), dtype=F64) for name, t in seqs[0].items()}

    def fn(ctx, runs):
        rows = {name: torch.cat([seqs[SLOTS.index(s)][name][p0:p0 + m] if s >= 0 else pad[name] for s, p0, m in runs]) for name in pad}
        out = scan(kind, rows, state, ctx, H, G, K, V, 6.0)
        if ctx.max_new == 1:                               # a step of single tokens may run twice
            again = scan(kind, rows, state, ctx, H, G, K, V, 6.0)
            assert torch.equal(torch.nan_to_num(again), torch.nan_to_num(out))
        return out

    call_host("vlrf_matrix_state_force", columns, warps)
    try:
        got = run_steps(fn, [0, 0, 0], 8, None, None)
    finally:
        call_host("vlrf_matrix_state_force", 0, 0)
    for i in range(3):
        close(got[i], want[i], 2e-5, f"{kind}, sequence {i}")
    assert torch.isnan(state[[s for s in range(8) if s not in SLOTS]]).all(), "a state of another slot was written"


@pytest.mark.parametrize("kind", ["decayed", "delta", "stabilized"])
def test_recurrence_carries_a_far_token_through_a_long_prompt(kind):
    """700 tokens in one step, then three single ones: one key, written by the first token alone and asked for by the last
    ones, lives in a channel that hardly decays; every other token writes elsewhere and is loud."""
    H, K, V, n = 2, 24, 20, 703
    d = draw_recurrence(kind, H, H, K, V, [n], 5)[0]
    d["k"][0, :, 0], d["k"][1:, :, 0], d["q"][700:] = 4.0, 0.0, 0.0
    d["q"][700:, :, 0] = 3.0
    d["decay"][:, :, 0] = 0.9999
    d["v"][0] = 5.0
    if kind == "delta":
        d["k"] = plain.unit(d["k"])
        d["q"] = plain.unit(d["q"])
        d["s1"] = (d["q"] * d["k"]).sum(-1).float().double()
    if kind == "stabilized":
        d["s0"][0], d["s1"][:] = 5.9, 30.0                 # (a gate nearly open in, a forget gate that forgets nothing)
    d = {name: t.float().double() for name, t in d.items()}
    want = plain_recurrence(kind, d, H, H, K, 6.0)
    gone = {name: t.clone() for name, t in d.items()}
    gone["v"][0] = -5.0
    assert float((plain_recurrence(kind, gone, H, H, K, 6.0)[700:] - want[700:]).abs().max() / want[700:].abs().max()) > 1e-2
    state = torch.zeros(2, 2, -(-state_numbers(kind, H, K, V) // 4) * 4, device="cuda")
    got = []
    for p0, m in ((0, 700), (700, 1), (701, 1), (702, 1)):
        ctx, _ = step_ctx([(1, p0, m)])
        got.append(scan(kind, {name: t[p0:p0 + m] for name, t in d.items()}, state, ctx, H, H, K, V, 6.0))
    # (a stabilized read-out is divided by n · q, which comes near zero at some of the 700 tokens)
    close(torch.cat(got), want, 5e-5 if kind != "stabilized" else 1e-2, kind)
    close(torch.cat(got)[700:], want[700:], 5e-5, kind + ", the far token")


def test_recurrence_of_seventy_single_tokens_and_a_full_batch_edge():
    """Many sequences in one decode step; and prompts of 15, 16, 17, 31, 32 and 33 tokens (the staged batches' edges)."""
    H, K, V = 3, 32, 48
    seqs = draw_recurrence("delta", H, H, K, V, [4] * 70, 9)
    state = torch.zeros(70, 2, H * K * V, device="cuda")
    got = [[] for _ in seqs]
    for t in range(4):
        ctx, _ = step_ctx([(s, t, 1) for s in range(70)])
        y = scan("delta", {name: torch.cat([d[name][t:t + 1] for d in seqs]) for name in seqs[0]}, state, ctx, H, H, K, V, 0.0)
        for s in range(70):
            got[s].append(y[s:s + 1])
    for s in range(70):
        close(torch.cat(got[s]), plain_recurrence("delta", seqs[s], H, H, K, 0.0), 2e-5, f"sequence {s}")
    lens = [15, 16, 17, 31, 32, 33]
    for kind in ("decayed", "stabilized"):
        seqs = draw_recurrence(kind, H, H, K, V, lens, 10)
        state = torch.zeros(6, 2, -(-state_numbers(kind, H, K, V) // 4) * 4, device="cuda")
        ctx, _ = step_ctx([(s, 0, n) for s, n in enumerate(lens)])
        y = scan(kind, {name: torch.cat([d[name] for d in seqs]) for name in seqs[0]}, state, ctx, H, H, K, V, 6.0)
        close(y, torch.cat([plain_recurrence(kind, d, H, H, K, 6.0) for d in seqs]), 2e-5, kind)


@pytest.mark.parametrize("H,G,K,V,taps", [(4, 2, 24, 16, 4), (2, 2, 32, 40, 3), (1, 1, 64, 48, 1), (6, 3, 9, 11, 5), (2, 1, 128, 128, 4),
                                          (1, 1, 200, 72, 2), (1, 1, 300, 500, 4), (3, 3, 16, 8, 16), (1, 1, 512, 16, 9)])
def test_convolution_and_unit_norms_over_steps(H, G, K, V, taps):
    from vlrf_b200.csrc import ops
    ch = 2 * G * K + H * V
    g = torch.Generator().manual_seed(ch + taps)
    us = [torch.randn(n, ch, generator=g).double() for n in TOTAL]
    w = torch.randn(ch, taps, generator=g).double()
    want, want_kq = [], []
    for u in us:
        c = plain.short_convolution(u, w)
        q, k = plain.unit(c[:, :G * K].reshape(-1, G, K)), plain.unit(c[:, G * K:2 * G * K].reshape(-1, G, K))
        want.append(torch.cat([q.reshape(-1, G * K), k.reshape(-1, G * K), c[:, 2 * G * K:]], dim=1))
        want_kq.append((q * k).sum(-1))
    off = 12
    state = torch.full((8, 2, off + (taps - 1) * ch + 3), float("nan"), device="cuda")
    for s in SLOTS:
        state[s] = 0.0
    wd = dev(w, torch.float32)

    def fn(ctx, runs):
        rows = torch.cat([us[SLOTS.index(s)][p0:p0 + n] if s >= 0 else torch.full((n, ch), float("nan"), dtype=F64) for s, p0, n in runs])
        wide = dev(torch.cat([torch.full((rows.shape[0], 5), float("nan"), dtype=F64), rows], dim=1), torch.float32)
        out = torch.full((ctx.n_tokens, ch), float("nan"), device="cuda")
        kq = torch.full((ctx.n_tokens, G), float("nan"), device="cuda")
        ops.conv_unit(wide, 5, wd, state, off, ctx, out, kq, H, G, K, V)
        return torch.cat([out, kq], dim=1)

    got = run_steps(fn, [0, 0, 0], 8, None, None)
    for i in range(3):
        close(got[i][:, :ch], want[i], 1e-5, f"sequence {i}")
        close(got[i][:, ch:], want_kq[i], 1e-5, f"k · q of sequence {i}")
        if taps > 1:                                       # the kept inputs, in the copy of the parity of the length
            kept = state[SLOTS[i], TOTAL[i] & 1, off:off + (taps - 1) * ch].view(taps - 1, ch)
            close(kept, torch.cat([torch.zeros(taps - 1, ch, dtype=F64), us[i]])[-(taps - 1):], 1e-6, "kept inputs")
    assert torch.isnan(state[[s for s in range(8) if s not in SLOTS]]).all()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("T,rank,rank2,H,K,V", [(1, 16, 24, 2, 32, 16), (200, 256, 24, 1, 200, 40), (90, 264, 8, 1, 60, 24), (70, 5, 33, 3, 24, 10), (64, 64, 8, 4, 33, 40), (3, 1, 128, 1, 130, 7), (129, 40, 40, 2, 64, 64)])
def test_low_rank_decays_and_gates(T, rank, rank2, H, K, V, dt):
    from vlrf_b200.csrc import ops
    g = torch.Generator().manual_seed(T + rank)
    a = torch.randn(T, rank + rank2 + 3, generator=g)
    a1, g1 = a[:, 1:1 + rank], a[:, 2 + rank:2 + rank + rank2]
    w1, w2 = (torch.randn(H * K, rank, generator=g) / rank ** 0.5).to(dt), (torch.randn(H * V, rank2, generator=g) / rank2 ** 0.5).to(dt)
    bias, a_log = torch.randn(H * K, generator=g), torch.randn(H, generator=g)
    bias[0], bias[1] = 40.0, -40.0                         # (both ends of softplus and of the sigmoid)
    ad = dev(a)
    d1, d2 = ad[:, 1:1 + rank], ad[:, 2 + rank:2 + rank + rank2]
    z = a1.double() @ w1.double().T + bias.double()
    want = torch.exp(-torch.exp(a_log.double()).repeat_interleave(K) * F.softplus(z))
    out = torch.full((T + 1, H * K + 2), float("nan"), device="cuda")
    gate = torch.full((T + 1, H * V), float("nan"), device="cuda")
    ops.lowrank_rows([(d1, dev(w1), out, "softplus_decay", dict(bias=dev(bias), a_log=dev(a_log), per=K)), (d2, dev(w2), gate, "plain", {})], T)
    close(out[:T, :H * K], want, 3e-5, "softplus decay")
    close(gate[:T], g1.double() @ w2.double().T, 3e-5, "gate")
    assert torch.isnan(out[T]).all() and torch.isnan(out[:, H * K:]).all() and torch.isnan(gate[T]).all()
    ops.lowrank_rows([(d1, dev(w1), out, "sigmoid_power", dict(bias=dev(bias), tau=16.0))], T)
    close(out[:T, :H * K], torch.sigmoid(z) ** (1 / 16.0), 3e-5, "power of a sigmoid")
    # a decay next to one is what a long memory rests on: its distance from one, too
    slow = torch.exp(F.logsigmoid(z) / 16.0)
    err = ((1 - out[:T, :H * K].double().cpu()) - (1 - slow)).abs().max()
    assert float(err) < 3e-5


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("H,V,per_head,divided,act", [(3, 16, False, False, "silu"), (2, 40, True, True, "sigmoid"), (4, 7, True, True, "sigmoid"),
                                                      (1, 512, False, False, "sigmoid"), (2, 600, False, True, "silu"), (5, 128, False, False, "silu")])
def test_a_heads_read_out(H, V, per_head, divided, act, dt):
    from vlrf_b200.csrc import ops
    T, eps = 37, 1e-5
    g = torch.Generator().manual_seed(V)
    y, gate = torch.randn(T, H, V, generator=g) * 0.01, torch.randn(T, H * V + 6, generator=g) * 3
    y[3] *= 1e-4                                           # (a head so small that eps decides)
    w = 1.0 + 0.3 * torch.randn(H * V if per_head else V, generator=g)
    den = torch.stack([torch.randn(T, H, generator=g), 0.4 * torch.rand(T, H, generator=g)], dim=-1)
    o = y.double()
    if divided:
        o = o / (torch.maximum(den[..., 0].double().abs(), den[..., 1].double()) + 1e-6)[..., None]
    z = gate[:, 4:4 + H * V].double().view(T, H, V)
    want = plain.over_rms(o, eps) * w.double().view(-1, V) * (F.silu(z) if act == "silu" else torch.sigmoid(z)) * 0.7
    wide = torch.full((T + 1, H * V + 8), float("nan"), dtype=dt, device="cuda")
    gd = dev(gate)
    ops.head_rows(dev(y.reshape(T, -1)), dev(w), gd[:, 4:4 + H * V], act, wide[:, 4:4 + H * V], T, H, V, eps, 0.7,
                  den=dev(den.reshape(T, -1)) if divided else None)
    close(wide[:T, 4:4 + H * V].float().view(T, H, V), want, tol(dt), "read-out")
    close(wide[3, 4:4 + H * V].float().view(H, V), want[3], tol(dt), "the small head")
    assert torch.isnan(wide[:, :4].float()).all() and torch.isnan(wide[:, 4 + H * V:].float()).all() and torch.isnan(wide[T].float()).all()


@pytest.mark.parametrize("d", [64, 100, 1000, 4096])
def test_a_pair_of_normed_outputs_is_added(d):
    from vlrf_b200.csrc import ops
    g = torch.Generator().manual_seed(d)
    T = 9
    a, b, x = torch.randn(T, d, generator=g), 30 * torch.randn(T, d, generator=g), torch.randn(T + 1, d, generator=g)
    wa, wb = 1 + 0.2 * torch.randn(d, generator=g), 1 + 0.2 * torch.randn(d, generator=g)
    pair = 0.5 * (plain.over_rms(a.double(), 1e-5) * wa.double() + plain.over_rms(b.double(), 1e-5) * wb.double())
    xd = dev(x)
    ops.norm_pair_add(dev(a), dev(b), dev(wa), dev(wb), xd, T, 1e-5, 0.5)
    close(xd[:T], x[:T].double() + pair, 1e-6, "added")
    assert torch.equal(xd[T].cpu(), x[T])
    ops.norm_pair_add(dev(a), dev(b), dev(wa), dev(wb), xd, T, 1e-5, 0.5, accumulate=False)
    close(xd[:T], pair, 1e-6, "replaced")


def slope_case(H, G, dk, window, keep, lens, seed):
    """As in the tests of attention at its edges: for the last query of every sequence the oldest key inside the window and the
    last kept key are loud through the first head of each key/value head, the keys just outside louder still, all of them
    by enough to outweigh what the slopes take off at that distance."""
    g = torch.Generator().manual_seed(seed)
    T = sum(lens)
    rd = lambda *shape: torch.randn(*shape, generator=g).bfloat16().double()   # noqa: E731
    q, k, v = rd(T, H, dk), rd(T, G, dk), rd(T, G, dk)
    slope = torch.tensor(plain.slopes(H), dtype=F64) * 0.2
    start = 0
    for n in lens:
        last, inside = start + n - 1, max(0, n - window) if window else 0
        for hk in range(G):
            h = hk * (H // G)
            size = float(q[last, h].norm())

            def loud(j, score):                            # a key whose score behind the slope comes out as `score`
                k[start + j, hk] = ((score + float(slope[h]) * (n - 1 - j)) / 0.5 / size ** 2 * q[last, h]).bfloat16().double()
            loud(inside, 6.0)
            if inside > keep:
                loud(inside - 1, 12.0)
                if keep > 0:
                    loud(keep - 1, 7.0)
                    if inside - 1 > keep:
                        loud(keep, 12.0)
        start += n
    mask = {"size": window, "keep_first": keep} if window else None
    want, start = [], 0
    for n in lens:
        sl = slice(start, start + n)
        want.append(plain.attend(q[sl], k[sl], v[sl], 0.5, mask, slope.tolist()))
        start += n
    return q, k, v, slope, torch.cat(want)


def run_slopes(q, k, v, slope, lens, window, keep, dtype, tail, splits=None):
    """Keys and values in a NaN-filled cache under a permuted block table; the last `tail` tokens of every sequence attend (None:
    all of them by the kernel that takes a warp per token and head)."""
    from vlrf_b200.csrc import ops
    from vlrf_b200.parts.context import Workspace
    T, H, dk = q.shape
    G = k.shape[1]
    slot_of = [s for s, n in enumerate(lens) for _ in range(n)]
    positions = [p for n in lens for p in range(n)]
    cache = PagedKV(len(lens), max(lens), G, dk, dk, dtype)
    proj = dev(torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], dim=1), torch.float32)
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    qo = torch.full((T, H * dk), float("nan"), dtype=dtype, device="cuda")
    tok_slot, tok_pos = dev(torch.tensor(slot_of), torch.int32), dev(torch.tensor(positions), torch.int32)
    ops.qkv_rope_append(proj, 0, H * dk, H * dk + G * dk, None, 0, qo, cache.k, cache.v, cache.table, tok_slot, tok_pos, T, H, G, dk, dk, True, err)
    sl = dev(slope, torch.float32)
    if tail is None:
        out = torch.full((T, H * dk), float("nan"), dtype=dtype, device="cuda")
        ops.attention_window(qo, cache.k, cache.v, cache.table, tok_slot, tok_pos, out, T, H, G, dk, dk, 0.5, window, 1.0, err, keep_first=keep, slopes=sl)
        rows = list(range(T))
    else:
        rows, seq_start, seq_pos0, start = [], [0], [], 0
        for n in lens:
            m = min(tail, n)
            rows += list(range(start + n - m, start + n))
            seq_start.append(seq_start[-1] + m)
            seq_pos0.append(n - m)
            start += n
        idx = torch.tensor(rows)
        i32 = lambda t: dev(torch.as_tensor(t), torch.int32)   # noqa: E731
        ctx = types.SimpleNamespace(n_tokens=len(rows), n_seqs=len(lens), max_new=min(tail, max(lens)), max_context=max(lens), ws=Workspace("cuda"),
                                    dev_err=err, tok_slot=i32(torch.tensor(slot_of)[idx]), tok_pos=i32(torch.tensor(positions)[idx]),
                                    seq_slot=i32(torch.arange(len(lens))), seq_start=i32(seq_start), seq_pos0=i32(seq_pos0))
        out = torch.full((len(rows), H * dk), float("nan"), dtype=dtype, device="cuda")
        if splits:
            os.environ["VLRF_B200_DECODE_SPLITS"] = str(splits)
        try:
            ops.attention_window_step(qo[idx.to("cuda")].contiguous(), cache.k, cache.v, cache.table, out, ctx, H, G, dk, dk, 0.5, window, 1.0,
                                      keep_first=keep, slopes=sl)
        finally:
            os.environ.pop("VLRF_B200_DECODE_SPLITS", None)
    assert int(err.item()) == 0
    return out.view(len(rows), H, dk), rows


@pytest.mark.parametrize("dtype,t", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("H,G,dk,window,keep", [(4, 1, 16, 40, 5), (6, 2, 32, 70, 0), (4, 4, 8, 64, 64), (8, 2, 16, 33, 70), (5, 1, 12, 7, 3),
                                                (3, 3, 64, 130, 1), (2, 1, 24, 0, 0), (16, 1, 64, 100, 24), (2, 2, 128, 65, 63), (20, 1, 16, 40, 9)])
def test_attention_with_distance_slopes_at_the_edges(H, G, dk, window, keep, dtype, t):
    lens = [1, 2, 64, 65, 129, 200, 333]
    q, k, v, slope, want = slope_case(H, G, dk, window, keep, lens, dk * 7 + window)
    got, rows = run_slopes(q, k, v, slope, lens, window, keep, dtype, None)
    close(got, want, t, "a warp per token and head")
    for tail, splits in ((10 ** 6, None), (70, None), (3, None), (1, 1), (1, 2), (1, 5)):
        got, rows = run_slopes(q, k, v, slope, lens, window, keep, dtype, tail, splits)
        close(got, want[torch.tensor(rows)], t, f"the last {tail} tokens, contexts in {splits} parts")


def test_an_edge_or_a_slope_would_show():
    """On those inputs: moving the window by one, keeping one token more or fewer, or leaving the slopes out changes the
    expected result of the last queries by far more than the kernels' tolerance."""
    lens = [200, 333]
    q, k, v, slope, want = slope_case(4, 1, 16, 40, 5, lens, 1)
    last = [199, 532]
    for mask, sl in (({"size": 41, "keep_first": 5}, slope), ({"size": 39, "keep_first": 5}, slope), ({"size": 40, "keep_first": 6}, slope),
                     ({"size": 40, "keep_first": 4}, slope), ({"size": 40, "keep_first": 5}, 0 * slope), ({"size": 40, "keep_first": 5}, slope.flip(0))):
        out = torch.cat([plain.attend(q[a:b], k[a:b], v[a:b], 0.5, mask, sl.tolist()) for a, b in ((0, 200), (200, 533))])
        assert float((out[last] - want[last]).abs().max() / want.abs().max()) > 0.05, mask


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("d", [96, 33, 1000])
def test_sinusoidal_positions(d, dt):
    from vlrf_b200.csrc import ops
    from vlrf_b200.parts import get_part
    g = torch.Generator().manual_seed(d)
    table = torch.randn(50, d, generator=g).to(dt)
    ctx, _ = step_ctx([(1, 0, 3), (0, 777, 2), (2, 131000, 5)], pad_rows=(1,))
    pos = ctx.tok_pos.cpu()
    tokens = torch.arange(ctx.n_tokens) * 5 % 50
    ctx.tokens, ctx.dev_err = dev(tokens, torch.int32), torch.zeros(1, dtype=torch.int32, device="cuda")
    out = torch.full((ctx.n_tokens + 1, d), float("nan"), device="cuda")
    ops.embed_sinusoid(dev(table), get_part("position", "sinusoidal")(d, "cuda").frequencies, 1.5, ctx, out)
    live = [i for i in range(ctx.n_tokens) if i != 3]
    close(out[live], (table.double()[tokens] * 1.5 + plain.sinusoid(pos, d))[live], 1e-6, "embedded")
    assert torch.isnan(out[[3, ctx.n_tokens]]).all() and int(ctx.dev_err.item()) == 0


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("width,E,top,ff,shared,T", [(64, 5, 2, 40, 24, 37), (96, 4, 1, 32, None, 9), (100, 3, 3, 28, 20, 70), (64, 6, 4, 48, 40, 130)])
def test_experts_whose_weights_act_on_their_inputs(width, E, top, ff, shared, T, dt):
    """The whole part against the plain one; the same weights on the outputs would differ."""
    from vlrf_b200.parts import get_part
    from vlrf_b200.parts.context import Workspace
    g = torch.Generator().manual_seed(width + E)
    rd = lambda *s: (torch.randn(*s, generator=g) / s[-1] ** 0.5).bfloat16()   # noqa: E731
    h = torch.randn(T, width, generator=g).bfloat16()
    order = torch.stack([torch.randperm(E, generator=g) for _ in range(T)]).float()
    h[:, :E] = order.bfloat16()                            # (scores that lie apart: no choice rests on rounding)
    w = {"r.router": (0.5 * torch.eye(E, width)).bfloat16()}
    for e in range(E):
        w[f"r.e{e}.gate"], w[f"r.e{e}.up"], w[f"r.e{e}.down"] = 2 * rd(ff, width), rd(ff, width), rd(width, ff)
    ml = {"router": {"top": top, "experts": E}}
    sh = None
    if shared is not None:
        w["r.shared.gate"], w["r.shared.up"], w["r.shared.down"] = rd(shared, width), rd(shared, width), rd(width, shared)
        ml["shared"] = {"ff": shared}
        sh = tuple(dev(w[f"r.shared.{n}"], dt) for n in ("gate", "up", "down")) + (None,)
    stack = lambda n: dev(torch.stack([w[f"r.e{e}.{n}"] for e in range(E)]), dt)   # noqa: E731
    part = get_part("feed_forward", "routed_experts")(dev(w["r.router"], dt), None, stack("gate"), stack("up"), stack("down"), top=top, shared=sh,
                                                      scoring="sigmoid", weights_on="input")
    w64 = {n: t.double() for n, t in w.items()}
    want = plain.routed_ff(h.double(), w64, "r.", ml)
    on_output = sum(torch.sigmoid(h.double() @ w64["r.router"].T).gather(1, plain.route(h.double(), w64, "r.", ml)[0][:, j:j + 1])
                    * torch.stack([plain.gated_ff(h[t].double(), w64, f"r.e{int(e)}.") for t, e in enumerate(plain.route(h.double(), w64, "r.", ml)[0][:, j])])
                    for j in range(top))
    if shared is None:
        assert float((on_output - want).abs().max() / want.abs().max()) > 0.02
    ctx, _ = step_ctx([(0, 0, T)])
    ctx.ws, ctx.act_dtype = Workspace("cuda"), dt
    x = dev(torch.ones(T, width))
    part.forward(dev(h, dt), x, ctx)
    close(x - 1.0, want, tol(dt), "experts")
