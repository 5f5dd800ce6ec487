"""Tagulix as data: its tensor names, its random initialisation, and its ModelSpec.

A pre-norm decoder whose residual stream runs in several copies side by side (parts/block.py: `streams`): a sublayer reads a weighted sum
of them through an RMS norm, and its output, times a constant, joins each of them by a weight of its own while a small matrix mixes
them; the head reads their sum. A layer's mixer is grouped attention inside a sliding window with rotated, then normed
queries and keys and biases on every projection (parts/attention.py: `rotary_window_attention`), or two mixers side by side whose scaled
outputs are summed (`side_by_side_sum`): attention with a learned bias by distance, a learned sink per head and queries
that grow with the position (`distance_bias_attention`), and linear attention with a fixed decay per head and silu on queries, keys and
values (parts/recurrent.py: `decay_attention`). The feed-forward, where a layer has one, is a mixture of gelu experts chosen by corrected
softmax scores inside the best groups; some of the router's outputs stand for no expert but for the input itself (parts/mlp.py:
`routed_experts`). A layer may run with an earlier or later layer's tensors and a cache and state of its own.

Tensor names (matrices stored [out, in]): `embed`, `head`, `final.norm`, and for every layer i with tensors of its own `l<i>.norm1`,
`l<i>.hc1.{in out mix}`, with a feed-forward `l<i>.norm2` and `l<i>.hc2.{in out mix}`, the mixer's under `l<i>.mix.` and the
feed-forward's under `l<i>.mlp.`:
  attention  q q.b k k.b v v.b o o.b
  parallel   left.{q k v q.norm k.norm rel sink o}, right.{q k v g o norm}
  moe        e<j>.{up down}, router, correction
"""

from __future__ import annotations

import torch

from ..config.registry import Architecture, register_architecture
from ..config.tagulix import NAME, TagulixConfig, WindowAttention
from ..parts import LayerSpec, PartSpec, Runtime
from ..weights.loader import TensorSpec, WeightSpec
from .decoder import DecoderModel, ModelSpec, ScheduleEntry

# No mixer limits a sequence's length: the engine's options bound it.
UNBOUNDED_SEQ_LEN = 1 << 30


def _mixer_names(layer, i: int, width: int) -> dict[str, tuple[str, tuple]]:
    """The mixer part's weight name -> (tensor name, shape). The rows of a bias table are the checkpoint's own: a name per
    layer stands for them."""
    def entry(name, *shape):
        return (f"l{i}.mix.{name}", tuple(shape))

    m = layer.mixer
    if isinstance(m, WindowAttention):
        out = {}
        for name, n in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
            out.update({f"w_{name}": entry(name, n, width), f"b_{name}": entry(f"{name}.b", n)})
        out.update({"w_out": entry("o", width, m.heads * m.vdim), "b_out": entry("o.b", width)})
        return out
    a, r = m.left, m.right
    return {"left.w_q": entry("left.q", a.heads * a.dim, width), "left.w_k": entry("left.k", a.kv_heads * a.dim, width),
            "left.w_v": entry("left.v", a.kv_heads * a.vdim, width), "left.q_norm": entry("left.q.norm", a.dim),
            "left.k_norm": entry("left.k.norm", a.dim), "left.rel": entry("left.rel", f"l{i} bias rows", a.heads),
            "left.sink": entry("left.sink", a.heads), "left.w_out": entry("left.o", width, a.heads * a.vdim),
            "right.w_q": entry("right.q", r.heads * r.dim, width), "right.w_k": entry("right.k", r.heads * r.dim, width),
            "right.w_v": entry("right.v", r.heads * r.vdim, width), "right.w_gate": entry("right.g", r.heads * r.vdim, width),
            "right.w_out": entry("right.o", width, r.heads * r.vdim), "right.norm": entry("right.norm", r.heads * r.vdim)}


def _mlp_names(layer, i: int, width: int) -> dict[str, tuple[str, tuple]]:
    e, p, out = layer.mlp, f"l{i}.mlp.", {}
    for j in range(e.experts):
        out.update({f"e{j}.w_up": (f"{p}e{j}.up", (e.ff, width)), f"e{j}.w_down": (f"{p}e{j}.down", (width, e.ff))})
    out.update({"router": (p + "router", (e.experts + e.identity, width)), "correction": (p + "correction", (e.experts + e.identity,))})
    return out


def _stream_names(cfg: TagulixConfig, layer, i: int) -> dict[str, tuple[str, tuple]]:
    s, out = cfg.streams, {}
    for q in (1, 2) if s and layer.mlp is not None else (1,) if s else ():
        out.update({f"in_{q}": (f"l{i}.hc{q}.in", (s,)), f"out_{q}": (f"l{i}.hc{q}.out", (s,)), f"mix_{q}": (f"l{i}.hc{q}.mix", (s, s))})
    return out


def weight_spec(cfg: TagulixConfig) -> WeightSpec:
    d = cfg.width
    tensors = [TensorSpec("embed", (cfg.vocab_size, d))]
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is not None:
            continue
        tensors += [TensorSpec(f"l{i}.{name}", (d,)) for name in (("norm1", "norm2") if layer.mlp is not None else ("norm1",))]
        names = {**_mixer_names(layer, i, d), **(_mlp_names(layer, i, d) if layer.mlp is not None else {}), **_stream_names(cfg, layer, i)}
        tensors += [TensorSpec(name, shape) for name, shape in names.values()]
    tensors += [TensorSpec("final.norm", (d,)), TensorSpec("head", (cfg.vocab_size, d))]
    return WeightSpec(tensors=tuple(tensors))


def random_weights(cfg: TagulixConfig, seed: int, std: float = 0.05, norm_std: float = 0.1, bias_rows: int = 16,
                   correction_std: float | None = None) -> dict[str, torch.Tensor]:
    """Float32 draws from ONE CPU generator, in the order of `weight_spec`: matrices N(0, std), those over fewer inputs than the
    model's width by their input's size; the token table N(0, 1); gains 1 + N(0, norm_std); biases, sinks and bias tables N(0, 1) times a
    size that lets them show; corrections N(0, correction_std) (default: a tenth of a score); streams read by weights that sum to about one, joined by weights
    around one and mixed by a matrix near the identity. `bias_rows` is the size that a configuration leaves to the checkpoint."""
    gen = torch.Generator(device="cpu")
    gen.manual_seed(seed)
    out: dict[str, torch.Tensor] = {}
    for ts in weight_spec(cfg).tensors:
        shape = tuple(bias_rows if isinstance(n, str) else n for n in ts.shape)
        draw = torch.randn(shape, generator=gen, dtype=torch.float32)
        name, last = ts.name, ts.name.rsplit(".", 1)[-1]
        if name == "embed":
            out[name] = draw
        elif ".hc" in name:
            s = cfg.streams
            out[name] = torch.eye(s) + 0.2 * draw / s ** 0.5 if last == "mix" else (1.0 + 0.3 * draw) / (s if last == "in" else 1)
        elif last == "router":
            out[name] = shape[1] ** -0.5 * draw
        elif last == "correction":
            out[name] = (0.1 / shape[0] if correction_std is None else correction_std) * draw
        elif last == "rel" or last == "sink":
            out[name] = 0.7 * draw
        elif len(shape) == 2:
            out[name] = (std if shape[1] >= cfg.width else shape[1] ** -0.5) * draw
        elif last in ("norm", "norm1", "norm2"):
            out[name] = 1.0 + norm_std * draw
        else:
            out[name] = 0.3 * draw      # biases of projections
    return out


def _layer_spec(cfg: TagulixConfig, layer, i: int) -> LayerSpec:
    eps, d, m = cfg.norm_eps, cfg.width, layer.mixer
    weights = {own: name for own, (name, _) in _mixer_names(layer, i, d).items()}
    if isinstance(m, WindowAttention):
        mixer = PartSpec("rotary_window_attention", {
            "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "scale": m.scale, "window": m.window,
            "rot_dims": m.rot.dims if m.rot is not None else 0, "rot_base": m.rot.base if m.rot is not None else 1.0, "rot_layout": "interleaved",
            "qk_norm_eps": eps, "exact_weights": True}, weights)
    else:
        a, r = m.left, m.right
        left = {"kind": "distance_bias_attention", "params": {
            "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "v_head_dim": a.vdim, "scale": a.scale, "bias_max": a.bias_max,
            "qk_norm_eps": eps, "qk_norm_over": "head", "q_temp_coef": a.temp_coef, "q_temp_every": a.temp_every}}
        right = {"kind": "decay_attention", "params": {"n_heads": r.heads, "head_dim": r.dim, "v_head_dim": r.vdim, "decay": list(r.decay), "norm_eps": eps}}
        mixer = PartSpec("side_by_side_sum", {"left": left, "right": right, "left_scale": m.left_scale, "right_scale": m.right_scale}, weights)
    feed_forward = norm_2 = None
    if layer.mlp is not None:
        e = layer.mlp
        feed_forward = PartSpec("routed_experts", {
            "n_experts": e.experts, "n_identity": e.identity, "top": e.top, "scoring": "softmax", "n_groups": e.groups, "keep_groups": e.keep_groups,
            "group_mark": "best", "normalise": True, "route_scale": e.scale, "activation": "gelu", "gated": False},
            {own: name for own, (name, _) in _mlp_names(layer, i, d).items()})
        norm_2 = PartSpec("rms_norm", {"eps": eps}, {"weight": f"l{i}.norm2"})
    return LayerSpec(block="streams", mixer=mixer, feed_forward=feed_forward, norm_1=PartSpec("rms_norm", {"eps": eps}, {"weight": f"l{i}.norm1"}),
                     norm_2=norm_2, block_params={"factor": cfg.residual_mult},
                     block_weights={own: name for own, (name, _) in _stream_names(cfg, layer, i).items()})


def model_spec(cfg: TagulixConfig) -> ModelSpec:
    # the parts list holds the layers that own tensors; the schedule runs every configured layer, a borrower as its lender's parts
    # with a cache member and a state member of its own
    index, owned, schedule, n_states = {}, [], [], 0
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is None:
            index[i] = len(owned)
            owned.append(_layer_spec(cfg, layer, i))
    for i, layer in enumerate(cfg.layers):
        state = None
        if layer.type == "parallel":
            state, n_states = n_states, n_states + 1
        schedule.append(ScheduleEntry(layer=index[cfg.owner(i)], cache=i, writes_cache=True, state=state))
    return ModelSpec(
        vocab_size=cfg.vocab_size, hidden=cfg.width, max_seq_len=UNBOUNDED_SEQ_LEN, eos_token=None, embedding="embed", head="head",
        positions=None, layers=tuple(owned), final_norm=PartSpec("rms_norm", {"eps": cfg.norm_eps}, {"weight": "final.norm"}),
        schedule=tuple(schedule))


def build(cfg: TagulixConfig, tensors: dict[str, torch.Tensor], rt: Runtime) -> DecoderModel:
    return DecoderModel(model_spec(cfg), tensors, rt, config=cfg)


TAGULIX = register_architecture(Architecture(
    name=NAME, parse_config=TagulixConfig.from_json, weight_spec=weight_spec, random_weights=random_weights,
    build=build, config_to_json=TagulixConfig.to_json,
))
