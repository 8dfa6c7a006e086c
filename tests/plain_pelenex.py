"""A plain, slow implementation of the Pelenex design in float64, one function per mechanism, written from the
design's equations and sharing no code with the package (it reads model folders with the tests' own reader).

Notation: T tokens, width d.  Linear weights are [out, in] and applied as x · Wᵀ.  Everything runs over a whole
sequence from its first token and every recurrence is a loop over tokens, so there is no cache here and a state is a
local variable that starts at zero.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F

from plain_gpt2 import read_model_dir  # noqa: F401  (the tests' own reader of config.json + model.safetensors)


def over_rms(x, eps):
    """x / sqrt(mean(x²) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, w, groups, eps):
    """Every one of `groups` equal consecutive parts divided by its own root mean square, the whole times w."""
    shape = x.shape
    return over_rms(x.reshape(*shape[:-1], groups, shape[-1] // groups), eps).reshape(shape) * w


def sinusoid(positions, width):
    """Entry 2i: sin(p · 10000^(−2i/width)); entry 2i + 1: the cosine of the same angle."""
    out = torch.zeros(len(positions), width, dtype=torch.float64)
    for c in range(width):
        ang = positions.to(torch.float64) * 10000.0 ** (-(c - c % 2) / width)
        out[:, c] = torch.cos(ang) if c % 2 else torch.sin(ang)
    return out


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def visible(i, j, mask):
    """Query i sees key j: not later, and inside the window or among the first kept tokens."""
    if j > i:
        return False
    return mask is None or i - j < mask["size"] or j < (mask.get("keep_first") or 0)


def attend(q, k, v, scale, mask, slope):
    """q [T, H, n], k [T, G, n], v [T, G, m] → [T, H, m]; score = (q · k) · scale − slope_h · (i − j), softmax over the
    visible keys."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        js = torch.tensor([j for j in range(i + 1) if visible(i, j, mask)])
        for h in range(H):
            g = h // (H // G)
            s = (k[js, g] @ q[i, h]) * scale - slope[h] * (i - js).to(q.dtype)
            out[i, h] = torch.softmax(s, 0) @ v[js, g]
    return out


def windowed_attention(h, w, p, m, eps):
    """Values are the keys as projected; queries and keys divided by their root mean square per head; no rotation."""
    T, H, G, n = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[p + "q"].T).view(T, H, n)
    k = (h @ w[p + "k"].T).view(T, G, n)
    o = attend(over_rms(q, eps), over_rms(k, eps), k, m["scale"], m.get("mask"), slopes(H))
    return o.reshape(T, -1) @ w[p + "o"].T


def decayed_memory(q, k, v, alpha):
    """S_t = diag(alpha_t) S_(t−1) + k_t v_tᵀ, o_t = S_tᵀ q_t.  q, k, alpha [T, H, n], v [T, H, m] → [T, H, m]."""
    T, H, n = q.shape
    S = torch.zeros(H, n, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def gated_linear_attention(h, w, p, m, eps):
    T, H, n, mv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, n) * n ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, n)
    v = (h @ w[p + "v"].T).view(T, H, mv)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    alpha = torch.exp(F.logsigmoid(z) / m["tau"]).view(T, H, n)
    o = over_rms(decayed_memory(q, k, v, alpha), eps) * w[p + "norm"]
    return (o.reshape(T, -1) * F.silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def side_by_side(h, w, p, m, eps):
    """Half the sum of the two mixers' outputs, each normed over the width with a weight of its own."""
    left = windowed_attention(h, w, p + "left.", m["left"], eps)
    right = gated_linear_attention(h, w, p + "right.", m["right"], eps)
    return 0.5 * (over_rms(left, eps) * w[p + "left.out"] + over_rms(right, eps) * w[p + "right.out"])


def stabilized_memory(q, k, v, log_i, log_f):
    """The matrix memory with a running maximum m (starting at 0) taken out of the exponential gates; q, k [T, H, n],
    v [T, H, m], log gates [T, H] → [T, H, m]."""
    T, H, n = q.shape
    S = torch.zeros(H, n, v.shape[2], dtype=q.dtype)
    norm = torch.zeros(H, n, dtype=q.dtype)
    mx = torch.zeros(H, dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        new = torch.maximum(log_f[t] + mx, log_i[t])
        keep, take = torch.exp(log_f[t] + mx - new), torch.exp(log_i[t] - new)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        norm = keep[:, None] * norm + take[:, None] * k[t]
        mx = new
        den = torch.maximum((norm * q[t]).sum(-1).abs(), torch.exp(-mx)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(1) / den[:, None]
    return out


def mlstm(h, w, p, m, eps):
    T, H, n, mv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).view(T, H, n) * n ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, n)
    v = (h @ w[p + "v"].T).view(T, H, mv)
    log_i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    log_f = F.logsigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o = over_rms(stabilized_memory(q, k, v, log_i, log_f), eps).reshape(T, -1) * w[p + "norm"]
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def short_convolution(u, taps_w):
    """y_t = Σ_j w[:, j] u_(t − taps + 1 + j) per channel, zeros before the start, then x · sigmoid(x)."""
    T, taps = u.shape[0], taps_w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += taps_w[:, j] * u[s]
    return F.silu(out)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_memory(q, k, v, g, beta):
    """S ← g ⊙ S (rows), u = beta (v − Sᵀ k), S ← S + k uᵀ, o = Sᵀ q.  q, k, g [T, H, n], v [T, H, m], beta [T, H]."""
    T, H, n = q.shape
    S = torch.zeros(H, n, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def channel_delta(h, w, p, m, eps):
    T, H, G, n, mv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_convolution(h @ w[p + "q"].T, w[p + "q.conv"]).view(T, G, n)
    k = short_convolution(h @ w[p + "k"].T, w[p + "k.conv"]).view(T, G, n)
    v = short_convolution(h @ w[p + "v"].T, w[p + "v.conv"]).view(T, H, mv)
    share = [hh // (H // G) for hh in range(H)]
    q, k = unit(q)[:, share] * n ** -0.5, unit(k)[:, share]
    beta = torch.sigmoid(h @ w[p + "b"].T)
    z = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(T, H, n)
    g = torch.exp(-torch.exp(w[p + "A_log"])[:, None] * F.softplus(z))
    o = over_rms(delta_memory(q, k, v, g, beta), eps) * w[p + "norm"]
    return (o.reshape(T, -1) * torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)) @ w[p + "o"].T


def gated_ff(h, w, p):
    return (F.silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, ml, margins=None):
    """(chosen experts [T, top], their scores [T, top]): scores sigmoid(W_router h), the largest chosen, not renormalized."""
    top = ml["router"]["top"]
    z = h @ w[p + "router"].T
    order = torch.sort(z, dim=-1, descending=True, stable=True)
    if margins is not None and z.shape[1] > top:
        margins.append(order.values[:, top - 1] - order.values[:, top])
    return order.indices[:, :top], torch.sigmoid(order.values[:, :top])


def routed_ff(h, w, p, ml, margins=None):
    """Σ expert(score · h) over the chosen experts, and the shared expert on h itself."""
    idx, wt = route(h, w, p, ml, margins)
    rows = []
    for t in range(h.shape[0]):
        y = torch.zeros_like(h[t])
        for j in range(idx.shape[1]):
            y = y + gated_ff(wt[t, j] * h[t], w, p + f"e{int(idx[t, j])}.")
        rows.append(y)
    out = torch.stack(rows)
    return out + gated_ff(h, w, p + "shared.") if ml.get("shared") is not None else out


MIXERS = {"mlstm": mlstm, "parallel": side_by_side, "channel_delta": channel_delta}


def forward(cfg, w, ids, keep_layers=False, margins=None):
    """ids [T] → logits [T, vocab] (and the residual after every layer, if asked)."""
    w = {k: (v.to(torch.float64) if v.is_floating_point() else v) for k, v in w.items()}
    ids = torch.as_tensor(ids, dtype=torch.long)
    eps, groups = cfg["norm"]["eps"], cfg["norm"].get("groups", 1)
    x = w["embed"][ids] + sinusoid(torch.arange(len(ids)), cfg["width"])
    kept = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = group_norm(x, w[p + "norm1"], groups, eps)
        y = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
        ml = layer.get("mlp")
        if ml is not None:
            y = y + (gated_ff(h, w, p + "mlp.") if ml["kind"] == "dense" else routed_ff(h, w, p + "mlp.", ml, margins))
        x = x + y
        kept.append(x)
    logits = group_norm(x, w["final.norm"], groups, eps) @ w["head"].T
    cap = cfg.get("logit_softcap")
    if cap is not None:
        logits = cap * torch.tanh(logits / cap)
    return (logits, torch.stack(kept)) if keep_layers else logits


def logits_all_positions(cfg, w, ids):
    return forward(cfg, w, ids)


def decided_prefix(cfg, w, ids, least=0.05):
    """Positions before the first token whose routing (in any layer) has two logits closer together than `least` where the
    chosen end."""
    margins = []
    forward(cfg, w, ids, margins=margins)
    if not margins:
        return len(ids)
    close = torch.nonzero(torch.stack(margins).min(0).values < least)
    return int(close[0]) if len(close) else len(ids)


def greedy_generate(cfg, w, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(torch.argmax(forward(cfg, w, ids)[-1])))
    return ids[len(prompt):]
