"""Small Pelenex configurations for the tests: every size differs from layer to layer and between the models, and what a
configuration could make equal by accident (heads and query/key heads, key size and value size, ranks of the low-rank
products, groups of the norm, one tap, one head, windows of a block, kept tokens of more than a block, top = 1, top = every
expert, an absent mask, cap, shared expert and feed-forward) is covered somewhere."""
import json
from pathlib import Path

import torch


def mlstm(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def both(left, right):
    """left: (heads, kv_heads, dim, scale, mask or None); right: (heads, dim, vdim, tau)."""
    heads, kv_heads, dim, scale, mask = left
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if mask is not None:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]} if mask[1] is not None else {"size": mask[0]}
    return {"type": "parallel", "mixer": {"left": m, "right": dict(zip(("heads", "dim", "vdim", "tau"), right))}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


#: every kind of layer with every kind of feed-forward; windows of 37 and 70 with 5 and no kept tokens
PEL_A = {"architecture": "Pelenex", "vocab": 311, "width": 96, "norm": {"eps": 1e-5, "groups": 3}, "logit_softcap": 20.0, "layers": [
    layer(both((6, 2, 16, 0.3, (37, 5)), (3, 24, 16, 8.0)), moe(40, 5, 2, shared=56)),
    layer(mlstm(3, 16, 40, 9.0), dense(72)),
    layer(delta(4, 2, 24, 16, 4), moe(24, 3, 3, shared=32)),
    layer(both((2, 1, 32, 0.18, (70, None)), (2, 16, 48, 16.0)), None),
    layer(delta(2, 2, 16, 32, 3), dense(56)),
    layer(mlstm(2, 40, 24, 15.0), moe(32, 4, 1)),
]}
#: one group in the norm and no cap; an attention over all keys, kept tokens of more than a block under a window of 33; one
#: head of everything; one tap; layers without feed-forward
PEL_B = {"architecture": "Pelenex", "vocab": 257, "width": 128, "norm": {"eps": 1e-6}, "layers": [
    layer(delta(1, 1, 64, 48, 1), None),
    layer(both((4, 4, 16, 0.25, None), (1, 64, 32, 4.0)), dense(96)),
    layer(mlstm(1, 64, 16, 30.0), None),
    layer(both((8, 2, 8, 0.4, (33, 70)), (4, 8, 24, 32.0)), moe(48, 6, 1, shared=40)),
]}
#: sizes that are no multiples of 8 or 4 (the attention kernels of the CUDA cores, the recurrences' plain copies)
PEL_ODD = {"architecture": "Pelenex", "vocab": 199, "width": 100, "norm": {"eps": 1e-5, "groups": 5}, "logit_softcap": 8.0, "layers": [
    layer(mlstm(3, 13, 22, 6.0), moe(28, 7, 3, shared=20)),
    layer(both((5, 1, 12, 0.28, (7, 3)), (3, 10, 7, 12.0)), dense(44)),
    layer(delta(6, 3, 9, 11, 5), moe(36, 2, 1)),
    layer(both((3, 3, 20, 0.3, (130, 1)), (1, 33, 18, 16.0)), None),
]}
#: attention made sharp (its query and key norms leave only the scale to do it) and slow decays, so that a wrong key, an edge
#: or a lost state moves the logits by far more than rounding does; every expert is taken, so that no choice rests on
#: rounding and bfloat16 can be held against the plain implementation at every position
PEL_SHARP = {"architecture": "Pelenex", "vocab": 307, "width": 64, "norm": {"eps": 1e-5, "groups": 2}, "logit_softcap": 30.0, "layers": [
    layer(both((4, 2, 16, 1.0, (48, 9)), (2, 24, 16, 64.0)), moe(64, 3, 3, shared=24)),
    layer(mlstm(2, 24, 16, 12.0), dense(80)),
    layer(delta(4, 2, 16, 8, 4), moe(48, 2, 2, shared=16)),
    layer(both((2, 1, 32, 0.5, (100, 20)), (4, 16, 8, 48.0)), dense(48)),
]}
MODELS = {"pel_a": PEL_A, "pel_b": PEL_B, "pel_odd": PEL_ODD, "pel_sharp": PEL_SHARP}


def write_model(cfg: dict, seed: int, out_dir, ranks: int | None = None, slow: float = 0.0, apart: float = 0.0) -> None:
    """The package's random draw for the configuration; `ranks`: the low-rank products get ranks of their own, from `ranks` on;
    `slow` is added to the forget gates' and the decays' biases and taken off the steps' biases (states that last longer).
    `apart` > 0 keeps the experts' scores apart, so that few choices rest on rounding (see the plain `decided_prefix`): of
    every token's embedding the first entries, one per expert, are an order of the experts of its own (values from −apart to
    apart), and a router's rows mostly read them."""
    import vlrf_b200.models  # noqa: F401
    from vlrf_b200.registry import parse_config
    from vlrf_b200.weights import write_safetensors
    arch, parsed = parse_config(cfg)
    gen = torch.Generator().manual_seed(seed)
    tensors = arch.random_weights(parsed, gen)
    routers = [n for n in sorted(tensors) if n.endswith("router")]
    if apart and routers:
        most = max(tensors[n].shape[0] for n in routers)
        for t in range(cfg["vocab"]):
            tensors["embed"][t, :most] = torch.linspace(-apart, apart, most)[torch.randperm(most, generator=gen)]
        for n in routers:
            tensors[n] = 0.1 * tensors[n]
            tensors[n][:, :tensors[n].shape[0]] += torch.eye(tensors[n].shape[0])
    for name in tensors:
        # keys that lean towards the queries of the same token: a first token's read-out is (q · k) v divided by its own size, so
        # that where q · k happens to be near zero its sign, and with it everything behind, would rest on rounding
        for p in ("mix.k", "mix.right.k", "mix.k.conv"):
            if name.endswith(p):
                q = tensors[name[:-len(p)] + p.replace(".k", ".q")]
                tensors[name] = 0.6 * q + 0.8 * tensors[name]
    for i, name in enumerate(sorted(tensors)):
        if name.endswith(".f.b") or name.endswith(".a2.b"):
            tensors[name] = tensors[name] + slow
        if name.endswith(".dt_bias"):
            tensors[name] = tensors[name] - slow
        if ranks is not None and (name.endswith(".a1") or name.endswith(".g1")):
            second = name[:-1] + "2"
            n = ranks + i % 7
            tensors[name] = torch.randn(n, tensors[name].shape[1], generator=gen) / tensors[name].shape[1] ** 0.5
            tensors[second] = torch.randn(tensors[second].shape[0], n, generator=gen) / n ** 0.5
    Path(out_dir).mkdir(parents=True, exist_ok=True)
    (Path(out_dir) / "config.json").write_text(json.dumps(cfg, indent=2))
    write_safetensors(Path(out_dir) / "model.safetensors",
                      {k: (v.to(torch.bfloat16) if v.is_floating_point() else v) for k, v in tensors.items()})
