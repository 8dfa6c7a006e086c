"""Small Vilodra configurations for the tests: every size differs from layer to layer and between the models, and what a
configuration could make equal by accident (query heads and key/value heads, a map's size and the value size, rotated and whole
size, head counts and windows of two layers that share latents, a factor of one, one head, top = 1, top = every expert, an
absent mask, scaling, rotation and feed-forward) is covered somewhere."""
import json
from pathlib import Path

import torch


def diffatt(heads, kv_heads, dim, vdim, scale, diff, rot=None, scaling=None):
    """rot: (dims, base); scaling: (factor, low, high, original)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, window=None, base=10000.0, scaling=None, kv_from=None):
    """scaling: (factor, original, fast, slow)."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def lightning(dim, vdim, *decay):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, scale):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


#: every kind of layer with every kind of feed-forward; a layer reading another's latents with other heads, sizes and a wider
#: window; values larger than, equal to and smaller than a map
VIL_A = {"architecture": "Vilodra", "vocab": 311, "width": 96, "norm": {"eps": 1e-5}, "residual_mult": 0.7, "layers": [
    layer(latent(3, 16, 8, 24, 40, 0.25, 40, 1000.0, (4.0, 64, 8.0, 2.0)), dense(72)),
    layer(diffatt(6, 2, 16, 40, 0.3, 0.3, (8, 500.0), (4.0, 1.0, 4.0, 128)), moe(40, 5, 2, 1.5)),
    layer(lightning(24, 16, 0.55, 0.93, 0.998), None),
    layer(latent(5, 12, 8, 16, 40, 0.3, 70, 1000.0, (4.0, 64, 8.0, 2.0), kv_from=0), moe(24, 3, 3, 0.8)),
    layer(diffatt(2, 1, 24, 24, 0.2, 0.55, (24, 10000.0)), dense(56)),
    layer(lightning(8, 40, 0.9, 0.7), moe(32, 4, 1, 2.5)),
]}
#: sizes of the tensor-core kernels; a factor of one; a reader with a narrower and one with a wider window than the owner's;
#: values as wide as both maps; one head of everything
VIL_B = {"architecture": "Vilodra", "vocab": 257, "width": 128, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "layers": [
    layer(lightning(64, 48, 0.97), None),
    layer(latent(4, 32, 32, 16, 64, 0.2, 65, 5000.0, (8.0, 128, 16.0, 1.0)), moe(48, 6, 1, 1.0)),
    layer(diffatt(4, 4, 32, 64, 0.18, 0.8, (16, 2000.0), (8.0, 1.0, 2.0, 64)), None),
    layer(latent(1, 64, 32, 48, 64, 0.15, 33, 5000.0, (8.0, 128, 16.0, 1.0), kv_from=1), dense(96)),
    layer(latent(8, 16, 32, 8, 64, 0.22, 130, 5000.0, (8.0, 128, 16.0, 1.0), kv_from=1), moe(32, 4, 2, 0.5)),
    layer(diffatt(1, 1, 64, 32, 0.125, 0.2, (64, 100.0), (2.0, 0.5, 8.0, 256)), dense(40)),
]}
#: sizes that are no multiples of 8 or 4 (the attention kernels of the CUDA cores, the recurrence's plain copies); no mask, no
#: rotation, no scaling; a factor above one
VIL_ODD = {"architecture": "Vilodra", "vocab": 199, "width": 100, "norm": {"eps": 1e-5}, "residual_mult": 1.3, "layers": [
    layer(diffatt(5, 1, 12, 20, 0.28, 0.4, (6, 3000.0), (2.0, 1.0, 3.0, 32)), moe(28, 7, 3, 1.2)),
    layer(latent(3, 10, 6, 7, 36, 0.3, 7, 700.0), dense(44)),
    layer(lightning(13, 11, 0.8, 0.99, 0.5), moe(36, 2, 1, 0.7)),
    layer(latent(2, 20, 6, 18, 36, 0.22, None, 700.0, kv_from=1), None),
    layer(diffatt(3, 3, 20, 9, 0.22, 0.1), dense(36)),
]}
#: attention made sharp (the query projections are drawn larger, see `write_model`) and slow decays, so that a wrong key, an edge, a
#: sink or a lost state moves the logits by far more than rounding does; every expert is taken, so that no choice rests on
#: rounding and bfloat16 can be held against the plain implementation at every position
VIL_SHARP = {"architecture": "Vilodra", "vocab": 307, "width": 64, "norm": {"eps": 1e-5}, "residual_mult": 0.9, "layers": [
    layer(latent(4, 16, 16, 16, 32, 0.2, 48, 2000.0, (4.0, 32, 4.0, 1.0)), moe(64, 3, 3, 1.4)),
    layer(diffatt(4, 2, 16, 24, 0.25, 0.35, (16, 1000.0), (4.0, 1.0, 4.0, 64)), dense(80)),
    layer(lightning(24, 16, 0.96, 0.99, 0.999), None),
    layer(latent(2, 48, 16, 24, 32, 0.15, 100, 2000.0, (4.0, 32, 4.0, 1.0), kv_from=0), moe(48, 2, 2, 0.9)),
]}
SHARP_FACTOR = 2.0
MODELS = {"vil_a": VIL_A, "vil_b": VIL_B, "vil_odd": VIL_ODD, "vil_sharp": VIL_SHARP}


def every_expert(cfg: dict) -> dict:
    """The same model with every token taking every expert."""
    out = json.loads(json.dumps(cfg))
    for lay in out["layers"]:
        if lay["mlp"] is not None and lay["mlp"]["kind"] == "moe":
            lay["mlp"]["router"]["top"] = lay["mlp"]["router"]["experts"]
    return out


def write_model(cfg: dict, seed: int, out_dir, sharp: float = 1.0) -> None:
    """The package's random draw for the configuration, the matrices that make the attentions' queries multiplied by `sharp`."""
    import vlrf_b200.models  # noqa: F401
    from vlrf_b200.registry import parse_config
    from vlrf_b200.weights import write_safetensors
    arch, parsed = parse_config(cfg)
    tensors = arch.random_weights(parsed, torch.Generator().manual_seed(seed))
    for i, lay in enumerate(cfg["layers"]):
        if lay["type"] != "lightning":
            tensors[f"l{i}.mix.q"] = tensors[f"l{i}.mix.q"] * sharp
    Path(out_dir).mkdir(parents=True, exist_ok=True)
    (Path(out_dir) / "config.json").write_text(json.dumps(cfg, indent=2))
    write_safetensors(Path(out_dir) / "model.safetensors", {k: v.to(torch.bfloat16) for k, v in tensors.items()})
