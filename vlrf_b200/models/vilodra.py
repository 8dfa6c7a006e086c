"""Vilodra: a decoder whose layers are differential attention, latent attention with a window and sinks, or a recurrence with a
fixed decay per head, each before a dense or routed feed-forward, with a factor on what every sublayer adds.

Tensors (all linear weights [out, in]): `embed` [vocab, width], which is the head as well; per layer i `l<i>.norm1` and, with a
feed-forward, `l<i>.norm2` (offsets from one); the mixer's `l<i>.mix.*`; the feed-forward's `l<i>.mlp.*`; `final.norm`.

  mixer "attention"         mix.q [heads·2·dim, width], mix.k [kv_heads·2·dim, width] (two maps a head), mix.v, mix.lq1, mix.lk1,
                            mix.lq2, mix.lk2 [dim] (the factor on the second map), mix.o
  mixer "latent_attention"  mix.q (per head [dim | rot_dim]), mix.dkv [kv_rank + rot_dim, width], mix.dkv.norm, mix.uk, mix.uv,
                            mix.sink [heads], mix.o; with kv_from no mix.dkv and mix.dkv.norm
  mixer "lightning"         mix.q, mix.k [heads·dim, width], mix.v, mix.g [heads·vdim, width], mix.norm [heads·vdim], mix.o
  mlp "dense"               mlp.gate, mlp.up, mlp.down
  mlp "moe"                 mlp.router [experts, width], mlp.e<k>.up / .down (no gate)

  x = embed[token];  per layer  x += residual_mult · mixer(norm1(x));  x += residual_mult · ffn(norm2(x));  logits = embed · norm(x)

residual_mult never meets the residual as an operation of its own: every sublayer is linear behind the place where its inner rows
are written (heads, the gated rows, the experts' weights), and takes the factor there, in float32.
"""
from __future__ import annotations

import torch

from ..config.vilodra import VilodraConfig
from ..engine.model import BuildOptions, DecoderModel, LayerCall
from ..parts import LMHead, TokenEmbedding, get_part
from ..registry import Architecture, register_architecture
from ..weights.spec import CheckedWeights, TensorSpec, place

#: positions a sequence may reach: the design has no position table, so this only sizes the block tables
MAX_POSITIONS = 1 << 17


def weight_spec(cfg: VilodraConfig) -> list[TensorSpec]:
    d = cfg.width
    specs = [TensorSpec("embed", (cfg.vocab, d))]
    for i, (m, ml) in enumerate(zip(cfg.mixers, cfg.mlps)):
        p = f"l{i}."
        specs += [TensorSpec(p + "norm1", (d,), "vector"), TensorSpec(p + "norm2", (d,), "vector", optional=ml is None)]
        q = p + "mix."
        if m.kind == "attention":
            specs += [TensorSpec(q + "q", (m.heads * 2 * m.dim, d)), TensorSpec(q + "k", (m.kv_heads * 2 * m.dim, d)),
                      TensorSpec(q + "v", (m.kv_heads * m.vdim, d))]
            specs += [TensorSpec(q + name, (m.dim,), "vector") for name in ("lq1", "lk1", "lq2", "lk2")]
        elif m.kind == "latent_attention":
            specs.append(TensorSpec(q + "q", (m.heads * (m.dim + m.rot_dim), d)))
            if m.kv_from is None:
                specs += [TensorSpec(q + "dkv", (m.kv_rank + m.rot_dim, d)), TensorSpec(q + "dkv.norm", (m.kv_rank,), "vector")]
            specs += [TensorSpec(q + "uk", (m.heads * m.dim, m.kv_rank)), TensorSpec(q + "uv", (m.heads * m.vdim, m.kv_rank)),
                      TensorSpec(q + "sink", (m.heads,), "vector")]
        else:
            specs += [TensorSpec(q + "q", (m.heads * m.dim, d)), TensorSpec(q + "k", (m.heads * m.dim, d)),
                      TensorSpec(q + "v", (m.heads * m.vdim, d)), TensorSpec(q + "g", (m.heads * m.vdim, d)),
                      TensorSpec(q + "norm", (m.heads * m.vdim,), "vector")]
        specs.append(TensorSpec(q + "o", (d, m.heads * m.vdim)))
        if ml is not None:
            q = p + "mlp."
            if ml.kind == "dense":
                specs += [TensorSpec(q + "gate", (ml.ff, d)), TensorSpec(q + "up", (ml.ff, d)), TensorSpec(q + "down", (d, ml.ff))]
            else:
                for e in range(ml.experts):
                    specs += [TensorSpec(q + f"e{e}.up", (ml.ff, d)), TensorSpec(q + f"e{e}.down", (d, ml.ff))]
                specs.append(TensorSpec(q + "router", (ml.experts, d)))
    specs.append(TensorSpec("final.norm", (d,), "vector"))
    return specs


def random_weights(cfg: VilodraConfig, gen: torch.Generator) -> dict:
    """Matrices N(0, 1/in); the norms whose stored weights are offsets from one N(0, 0.1), the others 1 + N(0, 0.1); sinks N(0, 1);
    the vectors of the second map's factor N(0, 0.3 / dim^(1/4)), so that their two products differ from each other and from
    zero: no term of a formula is hidden by a zero or a one.  The embedding is drawn with rows of size 0.06, since with the
    embedding as head a token's own row otherwise dominates its logits and a random model does nothing but repeat its last
    token whatever its layers compute."""
    out = {}
    for spec in weight_spec(cfg):
        if spec.optional:
            continue
        name = spec.name
        t = torch.randn(spec.shape, generator=gen, dtype=torch.float32)
        if name.endswith(".sink"):
            pass
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = t * (0.3 / spec.shape[0] ** 0.25)
        elif name.endswith((".dkv.norm", ".mix.norm")):
            t = 1.0 + 0.1 * t
        elif spec.kind == "vector":
            t = 0.1 * t
        elif name == "embed":
            t = 0.06 * t
        else:
            t = t / float(spec.shape[-1]) ** 0.5
        out[name] = t
    return out


def second_map_factor(lq1, lk1, lq2, lk2, diff: float) -> float:
    """exp(lq1 · lk1) − exp(lq2 · lk2) + diff, one number for a layer."""
    dot = lambda a, b: float((a.double() * b.double()).sum().exp())   # noqa: E731
    return dot(lq1, lk1) - dot(lq2, lk2) + diff


def build(cfg: VilodraConfig, weights: CheckedWeights, options: BuildOptions) -> DecoderModel:
    dt, dev = options.dtype, options.device
    factor = cfg.residual_mult

    def matrix(name):
        return place(weights[name], "matrix", dt, dev)

    def vector(name):
        return place(weights[name], "vector", dt, dev)

    norm_cls, block_cls = get_part("norm", "group_rmsnorm"), get_part("block", "pre_norm")

    def offset_norm(name):
        return norm_cls(vector(name), cfg.norm_eps, 1, offset=1.0)

    rotations: dict = {}

    def rotary(kind, rot):
        if rot is None:
            return None
        if (kind, rot) not in rotations:
            scaling = {"wavelengths" if kind == "attention" else "yarn": rot.scaling}
            rotations[kind, rot] = get_part("position", "rotary")(rot.base, rot.dims, dev, pairing="interleaved", **scaling)
        return rotations[kind, rot]

    layers, schedule = [], []
    for i, (m, ml) in enumerate(zip(cfg.mixers, cfg.mlps)):
        p = f"l{i}.mix."
        kv_from = None
        if m.kind == "attention":
            lam = second_map_factor(*(weights[p + name] for name in ("lq1", "lk1", "lq2", "lk2")), m.diff)
            mixer = get_part("mixer", "window_attention")(
                matrix(p + "q"), matrix(p + "k"), matrix(p + "v"), matrix(p + "o"), n_heads=m.heads, n_kv_heads=m.kv_heads, dim=m.dim,
                vdim=m.vdim, scale=m.scale, rotary=rotary(m.kind, m.rot), second_map=(lam, cfg.norm_eps), out_factor=(1.0 - m.diff) * factor)
        elif m.kind == "latent_attention":
            kv_from = m.kv_from
            own = kv_from is None
            mixer = get_part("mixer", "latent_attention")(
                n_heads=m.heads, dim=m.dim, vdim=m.vdim, kv_rank=m.kv_rank, rot_dim=m.rot_dim, scale=m.scale, eps=cfg.norm_eps,
                w_q=matrix(p + "q"), w_dkv=matrix(p + "dkv") if own else None, dkv_norm=vector(p + "dkv.norm") if own else None,
                w_uk=matrix(p + "uk"), w_uv=matrix(p + "uv"), w_out=matrix(p + "o"), rotary=rotary(m.kind, m.rot), window=m.window,
                cache_window=cfg.cache_window(i), sink=vector(p + "sink"), out_factor=factor)
        else:
            mixer = get_part("mixer", "fixed_memory")(
                matrix(p + "q"), matrix(p + "k"), matrix(p + "v"), matrix(p + "g"), vector(p + "norm"), matrix(p + "o"), n_heads=m.heads,
                dim=m.dim, vdim=m.vdim, decay=m.decay, eps=cfg.norm_eps, out_factor=factor)
        ffn = norm2 = None
        if ml is not None:
            q = f"l{i}.mlp."
            norm2 = offset_norm(f"l{i}.norm2")
            if ml.kind == "dense":
                ffn = get_part("feed_forward", "gated_mlp")(matrix(q + "gate"), matrix(q + "up"), matrix(q + "down"), activation="silu",
                                                            out_factor=factor)
            else:
                def stack(what):
                    return torch.stack([matrix(q + f"e{e}.{what}") for e in range(ml.experts)]).contiguous()
                ffn = get_part("feed_forward", "routed_experts")(
                    matrix(q + "router"), None, None, stack("up"), stack("down"), top=ml.top, scoring="softmax_all", renormalize=True,
                    weight_scale=ml.scale * factor, activation="gelu_erf")
        layers.append(block_cls(offset_norm(f"l{i}.norm1"), mixer, norm2, ffn))
        schedule.append(LayerCall(i, reads_cache_of=kv_from))
    embed = matrix("embed")
    return DecoderModel(config=cfg, embedding=TokenEmbedding(embed, None), layers=layers, schedule=schedule,
                        final_norm=offset_norm("final.norm"), head=LMHead(embed), options=options, max_seq_len=MAX_POSITIONS)


VILODRA = register_architecture(Architecture(
    name="Vilodra", config_cls=VilodraConfig, weight_spec=weight_spec, random_weights=random_weights, build=build))
