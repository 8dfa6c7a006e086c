"""Pelenex: a decoder of recurrent layers (mLSTM, a gated delta rule with a decay per channel, windowed attention beside
gated linear attention) with dense or routed feed-forwards, the mixer and the feed-forward of a layer side by side behind
one norm, and sinusoidal positions at the embedding.

Tensors (all linear weights [out, in]): `embed`, `head` [vocab, width]; per layer i `l<i>.norm1` [width], the mixer's
`l<i>.mix.*` and the feed-forward's `l<i>.mlp.*`; `final.norm` [width].  A rank (`a1`, `g1`) is what the tensors say.

  mixer "mlstm"          mix.q, .k, .v, .g, .o, mix.i, .f [heads, width] with biases .i.b, .f.b, mix.norm [heads·vdim]
  mixer "channel_delta"  mix.q, .k, .v with .conv [channels, taps] each, mix.b [heads, width], mix.A_log [heads], mix.a1 [rank,
                         width], mix.a2 [heads·dim, rank], mix.dt_bias [heads·dim], mix.g1, mix.g2 [heads·vdim, rank], mix.norm
                         [vdim], mix.o
  mixer "parallel"       mix.left.q, .k, .o (the values are the projected keys), mix.right.q, .k, .v, .g, .o, .norm [vdim], .a1, .a2,
                         .a2.b [heads·dim], mix.left.out, mix.right.out [width]
  mlp "dense"            mlp.gate, mlp.up, mlp.down
  mlp "moe"              mlp.router, mlp.e<k>.gate / .up / .down, mlp.shared.gate / .up / .down

  x = embed[token] + sinusoids(position)
  per layer: h = norm1(x) (RMS norm in groups), x += mixer(h) + ffn(h)
  logits = cap · tanh(head · norm(x) / cap)
"""
from __future__ import annotations

import torch

from ..config.pelenex import PelenexConfig
from ..engine.model import BuildOptions, DecoderModel, LayerCall
from ..parts import LMHead, TokenEmbedding, get_part
from ..registry import Architecture, register_architecture
from ..weights.spec import CheckedWeights, FreeSize, TensorSpec, place

#: positions a sequence may reach: the design has no position table, so this only sizes the block tables
MAX_POSITIONS = 1 << 17


def _rank(cfg: PelenexConfig, name: str) -> FreeSize:
    return FreeSize(name, max(8, cfg.width // 16))


def weight_spec(cfg: PelenexConfig) -> list[TensorSpec]:
    d = cfg.width
    specs = [TensorSpec("embed", (cfg.vocab, d))]

    def matrices(prefix, **shapes):
        specs.extend(TensorSpec(prefix + name, shape) for name, shape in shapes.items())

    def vectors(prefix, names):
        specs.extend(TensorSpec(prefix + name, shape, "vector") for name, shape in names.items())

    for i, (m, ml) in enumerate(zip(cfg.mixers, cfg.mlps)):
        p = f"l{i}."
        vectors(p, {"norm1": (d,)})
        q, r = p + "mix.", m.memory
        H, n, mv = r.heads, r.dim, r.vdim
        if m.kind == "mlstm":
            matrices(q, q=(H * n, d), k=(H * n, d), v=(H * mv, d), g=(H * mv, d), o=(d, H * mv), i=(H, d), f=(H, d))
            vectors(q, {"norm": (H * mv,), "i.b": (H,), "f.b": (H,)})
        elif m.kind == "channel_delta":
            G, ra, rg = r.kv_heads, _rank(cfg, q + "a1"), _rank(cfg, q + "g1")
            matrices(q, q=(G * n, d), k=(G * n, d), v=(H * mv, d), b=(H, d), a1=(ra, d), a2=(H * n, ra), g1=(rg, d), g2=(H * mv, rg),
                     o=(d, H * mv))
            vectors(q, {"q.conv": (G * n, r.conv), "k.conv": (G * n, r.conv), "v.conv": (H * mv, r.conv), "A_log": (H,), "norm": (mv,),
                        "dt_bias": (H * n,)})
        else:
            a, ra = m.attention, _rank(cfg, q + "right.a1")
            matrices(q + "left.", q=(a.heads * a.dim, d), k=(a.kv_heads * a.dim, d), o=(d, a.heads * a.vdim))
            matrices(q + "right.", q=(H * n, d), k=(H * n, d), v=(H * mv, d), g=(H * mv, d), o=(d, H * mv), a1=(ra, d), a2=(H * n, ra))
            vectors(q, {"right.norm": (mv,), "right.a2.b": (H * n,), "left.out": (d,), "right.out": (d,)})
        if ml is None:
            continue
        q = p + "mlp."
        if ml.kind == "dense":
            matrices(q, gate=(ml.ff, d), up=(ml.ff, d), down=(d, ml.ff))
        else:
            for e in range(ml.experts):
                matrices(q + f"e{e}.", gate=(ml.ff, d), up=(ml.ff, d), down=(d, ml.ff))
            matrices(q, router=(ml.experts, d))
            if ml.shared_ff:
                matrices(q + "shared.", gate=(ml.shared_ff, d), up=(ml.shared_ff, d), down=(d, ml.shared_ff))
    vectors("", {"final.norm": (d,)})
    matrices("", head=(cfg.vocab, d))
    return specs


def random_weights(cfg: PelenexConfig, gen: torch.Generator) -> dict:
    """Matrices N(0, 1/in); norm weights 1 + N(0, 0.1); the mLSTM's input gate biases N(0, 1) and forget gate biases
    3 + N(0, 1), the decays' biases 1 + N(0, 1.5) and step biases −4 … 0 with rates exp(A_log) of 0.2 … 2, so that some
    channels forget within a few tokens and others keep hundreds; the embedding and the head N(0, 1) and N(0, 4/width)."""
    out = {}
    for spec in weight_spec(cfg):
        name, shape = spec.name, spec.drawn_shape
        t = torch.randn(shape, generator=gen, dtype=torch.float32)
        if name.endswith(".i.b"):
            pass
        elif name.endswith(".f.b"):
            t = 3.0 + t
        elif name.endswith(".a2.b"):
            t = 1.0 + 1.5 * t
        elif name.endswith(".dt_bias"):
            t = -4.0 * torch.rand(shape, generator=gen)
        elif name.endswith(".A_log"):
            t = torch.log(0.2 + 1.8 * torch.rand(shape, generator=gen))
        elif name.endswith(".conv"):
            t = t / float(shape[-1]) ** 0.5
        elif spec.kind == "vector":
            t = 1.0 + 0.1 * t
        elif name == "head":
            t = t * 2.0 / float(shape[-1]) ** 0.5
        elif name != "embed":
            t = t / float(shape[-1]) ** 0.5
        out[name] = t
    return out


def build(cfg: PelenexConfig, weights: CheckedWeights, options: BuildOptions) -> DecoderModel:
    dt, dev, eps = options.dtype, options.device, cfg.norm_eps

    def matrix(name):
        return place(weights[name], "matrix", dt, dev)

    def vector(name):
        return place(weights[name], "vector", dt, dev)

    def mixer_of(m, p):
        r = m.memory
        sizes = dict(n_heads=r.heads, dim=r.dim, vdim=r.vdim, eps=eps)
        if m.kind == "mlstm":
            return get_part("mixer", "stabilized_memory")(
                matrix(p + "q"), matrix(p + "k"), matrix(p + "v"), matrix(p + "g"), matrix(p + "i"), vector(p + "i.b"), matrix(p + "f"),
                vector(p + "f.b"), vector(p + "norm"), matrix(p + "o"), gate_cap=r.gate_cap, **sizes)
        if m.kind == "channel_delta":
            return get_part("mixer", "delta_memory")(
                matrix(p + "q"), matrix(p + "k"), matrix(p + "v"), matrix(p + "b"), vector(p + "q.conv"), vector(p + "k.conv"),
                vector(p + "v.conv"), matrix(p + "a1"), matrix(p + "a2"), vector(p + "A_log"), vector(p + "dt_bias"), matrix(p + "g1"),
                matrix(p + "g2"), vector(p + "norm"), matrix(p + "o"), n_groups=r.kv_heads, **sizes)
        a, ql, qr = m.attention, p + "left.", p + "right."
        slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / a.heads) for h in range(a.heads)], dtype=torch.float32, device=dev)
        left = get_part("mixer", "window_attention")(
            matrix(ql + "q"), matrix(ql + "k"), None, matrix(ql + "o"), n_heads=a.heads, n_kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim,
            scale=a.scale, window=a.window, keep_first=a.keep_first, qk_norm="head", norm_eps=eps, slopes=slopes)
        right = get_part("mixer", "decayed_memory")(
            matrix(qr + "q"), matrix(qr + "k"), matrix(qr + "v"), matrix(qr + "g"), matrix(qr + "a1"), matrix(qr + "a2"),
            vector(qr + "a2.b"), vector(qr + "norm"), matrix(qr + "o"), tau=r.tau, **sizes)
        return get_part("mixer", "parallel")(left, right, left_scale=0.5, right_scale=0.5,
                                             out_norms=(vector(ql + "out"), vector(qr + "out"), eps))

    def feed_forward_of(ml, p):
        if ml is None:
            return None
        if ml.kind == "dense":
            return get_part("feed_forward", "gated_mlp")(matrix(p + "gate"), matrix(p + "up"), matrix(p + "down"), activation="silu")

        def stack(what):
            return torch.stack([matrix(p + f"e{e}.{what}") for e in range(ml.experts)]).contiguous()
        shared = None
        if ml.shared_ff:
            shared = (matrix(p + "shared.gate"), matrix(p + "shared.up"), matrix(p + "shared.down"), None)
        return get_part("feed_forward", "routed_experts")(matrix(p + "router"), None, stack("gate"), stack("up"), stack("down"), top=ml.top,
                                                          shared=shared, scoring="sigmoid", weights_on="input")

    norm_cls, block_cls = get_part("norm", "group_rmsnorm"), get_part("block", "parallel_sublayers")
    layers = [block_cls(norm_cls(vector(f"l{i}.norm1"), eps, cfg.norm_groups), mixer_of(m, f"l{i}.mix."), feed_forward_of(ml, f"l{i}.mlp."))
              for i, (m, ml) in enumerate(zip(cfg.mixers, cfg.mlps))]
    embedding = TokenEmbedding(matrix("embed"), get_part("position", "sinusoidal")(cfg.width, dev))
    return DecoderModel(config=cfg, embedding=embedding, layers=layers, schedule=[LayerCall(i) for i in range(len(layers))],
                        final_norm=norm_cls(vector("final.norm"), eps, cfg.norm_groups), head=LMHead(matrix("head"), cfg.logit_softcap),
                        options=options, max_seq_len=MAX_POSITIONS)


PELENEX = register_architecture(Architecture(
    name="Pelenex", config_cls=PelenexConfig, weight_spec=weight_spec, random_weights=random_weights, build=build))
