"""A plain, slow implementation of the Vilodra design in float64, one function per mechanism, written from the design's
equations and sharing no code with the package (it reads model folders with the tests' own reader).

Notation: T tokens, width d.  Linear weights are [out, in] and applied as x · Wᵀ.  Everything runs over a whole sequence
from its first token and the recurrence is a loop over tokens, so there is no cache here: a layer that reads another
layer's latents is handed that layer's as a value, and a state is a local variable that starts at zero.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F

from plain_gpt2 import read_model_dir  # noqa: F401  (the tests' own reader of config.json + model.safetensors)


def over_rms(x, eps):
    """x / sqrt(mean(x²) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """The stored weight is the factor's offset from one."""
    return over_rms(x, eps) * (1.0 + w)


# ---- rotation ------------------------------------------------------------------------------------------------------------
def frequencies(rot):
    return [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]


def stretched(freqs, sc):
    """By wavelength: short ones stay, long ones are `factor` times longer, a linear blend of the two frequencies between."""
    out = []
    for f in freqs:
        length = 2.0 * math.pi / f
        if length < sc["original"] / sc["high"]:
            out.append(f)
        elif length > sc["original"] / sc["low"]:
            out.append(f / sc["factor"])
        else:
            s = (sc["original"] / length - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1.0 - s) * f / sc["factor"] + s * f)
    return out


def yarn(freqs, sc, base, dims):
    """(frequencies, factor on cosines and sines): pairs below the index that turns `fast` times over `original` positions
    stay, those beyond the one that turns `slow` times are divided by `factor`, a linear ramp over the index between."""
    def index_of(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(index_of(sc["fast"])), 0), min(math.ceil(index_of(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, freqs, magnitude=1.0):
    """The first 2 · len(freqs) entries of the last axis in neighbouring pairs; x [T, heads, n]."""
    out = x.clone()
    for i, f in enumerate(freqs):
        a = positions.to(torch.float64) * f
        c, s = (magnitude * torch.cos(a))[:, None], (magnitude * torch.sin(a))[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


# ---- softmax attention ---------------------------------------------------------------------------------------------------
def attend(q, k, v, scale, window=None, sink=None):
    """q [T, H, n], k [T, G, n], v [T, G, m] → [T, H, m].  Query i sees keys i − window < j ≤ i (no window: every j ≤ i);
    with `sink` the denominator of head h has one more term exp(sink_h)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        first = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            g = h // (H // G)
            s = (k[first:i + 1, g] @ q[i, h]) * scale
            top = float(s.max()) if sink is None else max(float(s.max()), float(sink[h]))
            e = torch.exp(s - top)
            den = e.sum() + (0.0 if sink is None else torch.exp(sink[h] - top))
            out[i, h] = (e / den) @ v[first:i + 1, g]
    return out


def mix_of_maps(w, p, diff):
    """The factor on the second map: exp(lq1 · lk1) − exp(lq2 · lk2) + diff."""
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def differential_attention(h, w, p, m, eps):
    """Two attention maps a head over the same values, the second taken off the first."""
    T, H, G, n, mv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, 2, n)
    k = (h @ w[p + "k"].T).view(T, G, 2, n)
    v = (h @ w[p + "v"].T).view(T, G, mv)
    rot = m.get("rot")
    maps = []
    for j in range(2):
        qj, kj = q[:, :, j], k[:, :, j]
        if rot is not None:
            f = frequencies(rot)
            f = stretched(f, rot["scaling"]) if rot.get("scaling") is not None else f
            pos = torch.arange(T)
            qj, kj = rotate(qj, pos, f), rotate(kj, pos, f)
        maps.append(attend(qj, kj, v, m["scale"]))
    o = over_rms(maps[0] - mix_of_maps(w, p, m["diff"]) * maps[1], eps) * (1.0 - m["diff"])
    return o.reshape(T, -1) @ w[p + "o"].T


def latent_rotation(m):
    rot = m["rot"]
    f = frequencies(rot)
    return yarn(f, rot["scaling"], rot["base"], rot["dims"]) if rot.get("scaling") is not None else (f, 1.0)


def latents(h, w, p, m, eps):
    """(normed latent [T, kv_rank], rotated key part [T, rot_dim]): what a token leaves behind."""
    C = m["kv_rank"]
    u = h @ w[p + "dkv"].T
    f, mag = latent_rotation(m)
    r = rotate(u[:, None, C:], torch.arange(h.shape[0]), f, mag)[:, 0]
    return over_rms(u[:, :C], eps) * w[p + "dkv.norm"], r


def latent_attention(h, w, p, m, c, r):
    """Keys and values written out from the latents c and the shared rotated part r."""
    T, H, n, R, mv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, n + R)
    f, mag = latent_rotation(m)
    q = torch.cat([q[..., :n], rotate(q[..., n:], torch.arange(T), f, mag)], -1)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, n), r[:, None].expand(T, H, R)], -1)
    v = (c @ w[p + "uv"].T).view(T, H, mv)
    o = attend(q, k, v, m["scale"], m["mask"]["size"] if m.get("mask") is not None else None, w[p + "sink"])
    return o.reshape(T, -1) @ w[p + "o"].T


# ---- the recurrence ------------------------------------------------------------------------------------------------------
def fading_memory(q, k, v, decay):
    """S_t = decay_h S_(t−1) + k_t v_tᵀ, o_t = S_tᵀ q_t.  q, k [T, H, n], v [T, H, m], decay [H] → [T, H, m]."""
    T, H, n = q.shape
    S = torch.zeros(H, n, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def lightning(h, w, p, m, eps):
    T, H, n, mv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = F.silu(h @ w[p + "q"].T).view(T, H, n)
    k = F.silu(h @ w[p + "k"].T).view(T, H, n)
    v = F.silu(h @ w[p + "v"].T).view(T, H, mv)
    o = fading_memory(q, k, v, torch.tensor(m["decay"], dtype=torch.float64)).reshape(T, -1)
    return (over_rms(o, eps) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- feed-forward --------------------------------------------------------------------------------------------------------
def gated_ff(h, w, p):
    return (F.silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def route(h, w, p, ml, margins=None):
    """(chosen experts [T, top], their weights [T, top]): softmax over all logits, the largest chosen, renormalized, scaled."""
    top = ml["router"]["top"]
    z = h @ w[p + "router"].T
    s = torch.softmax(z, -1)
    order = torch.sort(s, dim=-1, descending=True, stable=True)
    if margins is not None and z.shape[1] > top:
        zs = torch.sort(z, dim=-1, descending=True).values
        margins.append(zs[:, top - 1] - zs[:, top])
    chosen = order.values[:, :top]
    return order.indices[:, :top], chosen / (chosen.sum(-1, keepdim=True) + 1e-20) * ml["router"]["scale"]


def routed_ff(h, w, p, ml, margins=None):
    idx, wt = route(h, w, p, ml, margins)
    rows = []
    for t in range(h.shape[0]):
        y = torch.zeros_like(h[t])
        for j in range(idx.shape[1]):
            e = p + f"e{int(idx[t, j])}."
            y = y + wt[t, j] * (gelu(h[t] @ w[e + "up"].T) @ w[e + "down"].T)
        rows.append(y)
    return torch.stack(rows)


# ---- the model -----------------------------------------------------------------------------------------------------------
def forward(cfg, w, ids, keep_layers=False, margins=None):
    """ids [T] → logits [T, vocab] (and the residual after every layer, if asked)."""
    w = {k: (v.to(torch.float64) if v.is_floating_point() else v) for k, v in w.items()}
    ids = torch.as_tensor(ids, dtype=torch.long)
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][ids]
    kept, left_behind = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = offset_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "lightning":
            y = lightning(h, w, p + "mix.", m, eps)
        elif layer["type"] == "attention":
            y = differential_attention(h, w, p + "mix.", m, eps)
        else:
            if m.get("kv_from") is None:
                left_behind[i] = latents(h, w, p + "mix.", m, eps)
            y = latent_attention(h, w, p + "mix.", m, *left_behind[i if m.get("kv_from") is None else m["kv_from"]])
        x = x + mult * y
        ml = layer.get("mlp")
        if ml is not None:
            h = offset_norm(x, w[p + "norm2"], eps)
            x = x + mult * (gated_ff(h, w, p + "mlp.") if ml["kind"] == "dense" else routed_ff(h, w, p + "mlp.", ml, margins))
        kept.append(x)
    logits = offset_norm(x, w["final.norm"], eps) @ w["embed"].T
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
