"""Lagelorn as data: its tensor names, its random initialisation, and its ModelSpec.

A decoder whose norms come AFTER the sums (parts/block.py: `post_norm`): x <- norm1(alpha x + mixer(x)), then
x <- norm2(alpha x + feed_forward(x)), RMS norms with a gain per coordinate; the sublayers read the stream itself. The stream starts
as the token's row plus the position's row of a learned table. A layer's mixer is the gated delta rule behind short
convolutions (parts/recurrent.py: `delta`), or two mixers side by side whose scaled outputs are summed (`side_by_side_sum`): attention
by chunks with norms over whole query and key rows, a learned bias by distance, a learned sink per head and values that are the
keys before their norm (parts/attention.py: `distance_bias_attention`), and time mixing with a decay per channel (`time_mix`). The
feed-forward, where a layer has one, is a gated gelu unit with biases. At its end every layer adds what it makes from the stream and
from the token's own row of a side table (parts/token_side.py: `gated_rows`). The head is a table of its own behind one more norm; its
logits are capped.

Tensor names (matrices stored [out, in]): `embed`, `pos`, `head`, `final.norm`, `side.embed` (the layers' columns side by side), and for
layer i `l<i>.norm1`, with a feed-forward `l<i>.norm2`, `l<i>.side.{gate proj norm}`, the mixer's under `l<i>.mix.` and the
feed-forward's under `l<i>.mlp.`:
  delta     q k v (each with .conv) b a A_log dt_bias norm g o
  parallel  left.{q q.b q.norm k k.b k.norm rel sink o}, right.{mu.r mu.k mu.v mu.g mu.w r k v g w1 w2 w0 u norm o}
  dense     gate gate.b up up.b down down.b
"""

from __future__ import annotations

import torch

from ..config.lagelorn import NAME, DeltaMixer, LagelornConfig
from ..config.registry import Architecture, register_architecture
from ..parts import LayerSpec, PartSpec, Runtime
from ..weights.loader import TensorSpec, WeightSpec
from .decoder import DecoderModel, ModelSpec

# A constant that the design fixes: queries and keys of the delta rule are divided by sqrt(sum of squares + UNIT_EPS).
UNIT_EPS = 1e-6


def _mixer_names(layer, i: int, width: int) -> dict[str, tuple[str, tuple]]:
    """The mixer part's weight name -> (tensor name, shape). The rows of a bias table and the decays' inner width are the
    checkpoint's own sizes, a name per layer stands for them."""
    def entry(name, *shape):
        return (f"l{i}.mix.{name}", tuple(shape))

    m = layer.mixer
    if isinstance(m, DeltaMixer):
        qk, v = m.kv_heads * m.dim, m.heads * m.vdim
        return {"w_q": entry("q", qk, width), "conv_q": entry("q.conv", qk, m.conv), "w_k": entry("k", qk, width), "conv_k": entry("k.conv", qk, m.conv),
                "w_v": entry("v", v, width), "conv_v": entry("v.conv", v, m.conv), "w_b": entry("b", m.heads, width), "a_log": entry("A_log", m.heads),
                "norm": entry("norm", m.vdim), "w_a": entry("a", m.heads, width), "dt_bias": entry("dt_bias", m.heads),
                "w_gate": entry("g", v, width), "w_out": entry("o", width, v)}
    a, t = m.left, m.right
    q, k, n = a.heads * a.dim, a.kv_heads * a.dim, t.heads * t.dim
    buckets, rank = f"l{i} bias rows", f"l{i} decay rank"
    out = {"left.w_q": entry("left.q", q, width), "left.b_q": entry("left.q.b", q), "left.w_k": entry("left.k", k, width), "left.b_k": entry("left.k.b", k),
           "left.q_norm": entry("left.q.norm", q), "left.k_norm": entry("left.k.norm", k), "left.rel": entry("left.rel", buckets, a.heads),
           "left.sink": entry("left.sink", a.heads), "left.w_out": entry("left.o", width, q)}
    out.update({f"right.mu_{s}": entry(f"right.mu.{s}", width) for s in "rkvgw"})
    out.update({f"right.{own}": entry(f"right.{stored}", n, width) for own, stored in (("w_r", "r"), ("w_k", "k"), ("w_v", "v"), ("w_gate", "g"))})
    out.update({"right.w1": entry("right.w1", rank, width), "right.w2": entry("right.w2", n, rank), "right.w0": entry("right.w0", n),
                "right.bonus": entry("right.u", t.heads, t.dim), "right.norm": entry("right.norm", n), "right.w_out": entry("right.o", width, n)})
    return out


def _mlp_names(layer, i: int, width: int) -> dict[str, tuple[str, tuple]]:
    ff, p = layer.mlp.ff, f"l{i}.mlp."
    return {"w_gate": (p + "gate", (ff, width)), "b_gate": (p + "gate.b", (ff,)), "w_up": (p + "up", (ff, width)), "b_up": (p + "up.b", (ff,)),
            "w_down": (p + "down", (width, ff)), "b_down": (p + "down.b", (width,))}


def weight_spec(cfg: LagelornConfig) -> WeightSpec:
    d = cfg.width
    tensors = [TensorSpec("embed", (cfg.vocab_size, d)), TensorSpec("pos", (cfg.max_positions, d))]
    if cfg.side_dim:
        tensors.append(TensorSpec("side.embed", (cfg.vocab_size, len(cfg.layers) * cfg.side_dim)))
    for i, layer in enumerate(cfg.layers):
        tensors += [TensorSpec(f"l{i}.{name}", (d,)) for name in (("norm1", "norm2") if layer.mlp is not None else ("norm1",))]
        tensors += [TensorSpec(name, shape) for name, shape in _mixer_names(layer, i, d).values()]
        if layer.mlp is not None:
            tensors += [TensorSpec(name, shape) for name, shape in _mlp_names(layer, i, d).values()]
        if cfg.side_dim:
            tensors += [TensorSpec(f"l{i}.side.gate", (cfg.side_dim, d)), TensorSpec(f"l{i}.side.proj", (d, cfg.side_dim)), TensorSpec(f"l{i}.side.norm", (d,))]
    tensors += [TensorSpec("final.norm", (d,)), TensorSpec("head", (cfg.vocab_size, d))]
    return WeightSpec(tensors=tuple(tensors))


def random_weights(cfg: LagelornConfig, seed: int, std: float = 0.05, norm_std: float = 0.1, bias_rows: int = 16, decay_rank: int = 16) -> dict[str, torch.Tensor]:
    """Float32 draws from ONE CPU generator, in the order of `weight_spec`: matrices N(0, std), those over fewer inputs than the
    model's width by their input's size; tables N(0, 1); gains 1 + N(0, norm_std) (the side norms' a third of it); biases, sinks, bias
    tables and bonuses N(0, 1) times a size that lets them show; shares of the row before in (0, 1); decays spread over a decade.
    `bias_rows` and `decay_rank` are the sizes that a configuration leaves to the checkpoint."""
    gen = torch.Generator(device="cpu")
    gen.manual_seed(seed)
    sizes = {"bias rows": bias_rows, "decay rank": decay_rank}
    out: dict[str, torch.Tensor] = {}
    for ts in weight_spec(cfg).tensors:
        shape = tuple(sizes[d.split(" ", 1)[1]] if isinstance(d, str) else d for d in ts.shape)
        draw = torch.randn(shape, generator=gen, dtype=torch.float32)
        name, last = ts.name, ts.name.rsplit(".", 1)[-1]
        if name in ("embed", "pos", "side.embed"):
            out[name] = draw * (0.5 if name == "pos" else 1.0)
        elif last == "conv":
            out[name] = 0.4 * draw
        elif last == "rel" or last == "u":
            out[name] = 0.7 * draw
        elif name.rsplit(".", 2)[-2:-1] == ["mu"]:
            out[name] = torch.sigmoid(draw)
        elif len(shape) == 2:
            out[name] = (std if shape[1] >= cfg.width else shape[1] ** -0.5) * draw
        elif last in ("norm", "norm1", "norm2"):
            out[name] = (1.0 + norm_std * draw) * (0.3 if name.endswith("side.norm") else 1.0)
        elif last == "w0":
            out[name] = 1.0 * draw - 1.5
        elif last == "A_log":
            out[name] = 0.8 * draw - 0.5
        elif last == "sink":
            out[name] = draw
        else:
            out[name] = 0.3 * draw      # biases of projections and step sizes
    return out


def model_spec(cfg: LagelornConfig) -> ModelSpec:
    eps, d = cfg.norm_eps, cfg.width
    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        weights = {own: name for own, (name, _) in _mixer_names(layer, i, d).items()}
        if isinstance(m, DeltaMixer):
            mixer = PartSpec("delta", {"n_heads": m.heads, "n_groups": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "conv_taps": m.conv,
                                       "unit_eps": UNIT_EPS, "norm_eps": eps}, weights)
        else:
            a, t = m.left, m.right
            left = {"kind": "distance_bias_attention", "params": {
                "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "v_head_dim": a.dim, "scale": a.scale, "chunk": a.chunk,
                "bias_max": a.bias_max, "qk_norm_eps": eps}}
            right = {"kind": "time_mix", "params": {"n_heads": t.heads, "head_dim": t.dim, "norm_eps": eps}}
            mixer = PartSpec("side_by_side_sum", {"left": left, "right": right, "left_scale": m.left_scale, "right_scale": m.right_scale}, weights)
        feed_forward = norm_2 = side = None
        if layer.mlp is not None:
            feed_forward = PartSpec("gated_mlp", {"activation": "gelu_tanh"}, {own: name for own, (name, _) in _mlp_names(layer, i, d).items()})
            norm_2 = PartSpec("rms_norm", {"eps": eps}, {"weight": f"l{i}.norm2"})
        if cfg.side_dim:
            side = PartSpec("gated_rows", {"column": i * cfg.side_dim, "dim": cfg.side_dim, "eps": eps},
                            {"table": "side.embed", "gate": f"l{i}.side.gate", "proj": f"l{i}.side.proj", "norm": f"l{i}.side.norm"})
        layers.append(LayerSpec(block="post_norm", mixer=mixer, feed_forward=feed_forward,
                                norm_1=PartSpec("rms_norm", {"eps": eps}, {"weight": f"l{i}.norm1"}), norm_2=norm_2, token_side=side,
                                block_params={"alpha": cfg.alpha}))
    return ModelSpec(
        vocab_size=cfg.vocab_size, hidden=d, max_seq_len=cfg.max_positions, eos_token=None, embedding="embed", head="head",
        positions=PartSpec("learned", {"n_positions": cfg.max_positions}, {"table": "pos"}), layers=tuple(layers),
        final_norm=PartSpec("rms_norm", {"eps": eps}, {"weight": "final.norm"}), logit_softcap=cfg.logit_softcap)


def build(cfg: LagelornConfig, tensors: dict[str, torch.Tensor], rt: Runtime) -> DecoderModel:
    return DecoderModel(model_spec(cfg), tensors, rt, config=cfg)


LAGELORN = register_architecture(Architecture(
    name=NAME, parse_config=LagelornConfig.from_json, weight_spec=weight_spec, random_weights=random_weights,
    build=build, config_to_json=LagelornConfig.to_json,
))
