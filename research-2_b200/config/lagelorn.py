"""The typed Lagelorn configuration, read from the design's own config.json keys.

A Lagelorn config.json names its model with `"architecture": "Lagelorn"` and lists its layers one by one: every entry of
`layers` gives the layer's `type` (which mixer it has: `delta`, the gated delta rule, or `parallel`, attention by chunks with a
bias by distance beside time mixing with a decay per channel), the mixer's sizes and constants (`mixer`), and its feed-forward
(`mlp`: `kind` `dense`, or null for a layer without one). Beside the layers stand `vocab`, `width`, `max_positions` (the rows of
the table of positions), `norm.eps`, `postln_alpha` (the factor on the stream inside the sum that a layer's norm follows),
`token_side.dim` (the width of a token's own row for one layer) and `logit_softcap`. No size has a default: a size that is missing
is an error that names it. Two sizes are the checkpoint's own: the rows of a bias table and the inner width of the decays. A
mechanism that a file does not mention is not there: no `mask` (or no `mask.size`) is one chunk, no `token_side` no side input, no
`logit_softcap` plain logits; `postln_alpha` left out is one, `kv_heads` and `vdim` left out equal `heads` and `dim`.
"""

from __future__ import annotations

from dataclasses import dataclass

from .pidodra import _number_or_one
from .registry import ConfigError
from .zirunex import _get, _int, _number
from .zudalorn import _optional

NAME = "Lagelorn"
MIXER_TYPES = ("delta", "parallel")
MLP_KINDS = ("dense",)


def _heads(data: dict, where: str) -> tuple[int, int]:
    heads = _int(data, "heads", where)
    kv_heads = _int(data, "kv_heads", where) if "kv_heads" in data else heads
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}'heads' ({heads}) must be a multiple of 'kv_heads' ({kv_heads})")
    return heads, kv_heads


@dataclass(frozen=True)
class DeltaMixer:
    heads: int
    kv_heads: int   # heads of queries and keys; `heads` of values
    dim: int
    vdim: int
    conv: int       # taps of the short convolutions

    @staticmethod
    def from_json(data: dict, where: str) -> "DeltaMixer":
        dim = _int(data, "dim", where)
        heads, kv_heads = _heads(data, where)
        return DeltaMixer(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_int(data, "vdim", where) if "vdim" in data else dim,
                          conv=_int(data, "conv", where))

    def to_json(self) -> dict:
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}


@dataclass(frozen=True)
class ChunkAttention:
    heads: int
    kv_heads: int
    dim: int        # size of a query, key and value head: the values are the keys before their norm
    scale: float    # scores are (q . k) * scale, then the bias
    chunk: int      # mask.size: position i sees the keys of its own chunk; 0: every key up to i
    bias_max: int   # farther keys share the bias table's last row

    @staticmethod
    def from_json(data: dict, where: str) -> "ChunkAttention":
        dim = _int(data, "dim", where)
        heads, kv_heads = _heads(data, where)
        vdim = _int(data, "vdim", where) if "vdim" in data else dim
        if vdim != dim:
            raise ConfigError(f"config.json: {where}'vdim' ({vdim}) must equal 'dim' ({dim}): the values are the keys")
        mask = _optional(data, "mask")
        if mask is not None and not isinstance(mask, dict):
            raise ConfigError(f"config.json: {where}'mask' must be an object, got {mask!r}")
        return ChunkAttention(heads=heads, kv_heads=kv_heads, dim=dim, scale=_number(data, "scale", where),
                              chunk=_int(mask, "size", where + "mask.") if mask and mask.get("size") is not None else 0,
                              bias_max=_int(data, "bias_max", where, minimum=2))

    def to_json(self) -> dict:
        out = {"bias_max": self.bias_max, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.dim}
        if self.chunk:
            out["mask"] = {"size": self.chunk}
        return out


@dataclass(frozen=True)
class TimeMixing:
    heads: int
    dim: int

    @staticmethod
    def from_json(data: dict, where: str) -> "TimeMixing":
        return TimeMixing(heads=_int(data, "heads", where), dim=_int(data, "dim", where))

    def to_json(self) -> dict:
        return {"dim": self.dim, "heads": self.heads}


@dataclass(frozen=True)
class ParallelMixer:
    left: ChunkAttention
    right: TimeMixing
    left_scale: float
    right_scale: float

    @staticmethod
    def from_json(data: dict, where: str) -> "ParallelMixer":
        return ParallelMixer(
            left=ChunkAttention.from_json(_get(data, "left", where), where + "left."), right=TimeMixing.from_json(_get(data, "right", where), where + "right."),
            left_scale=_number(data, "left_scale", where, positive=False), right_scale=_number(data, "right_scale", where, positive=False))

    def to_json(self) -> dict:
        return {"left": self.left.to_json(), "left_scale": self.left_scale, "right": self.right.to_json(), "right_scale": self.right_scale}


@dataclass(frozen=True)
class DenseMlp:
    ff: int

    @staticmethod
    def from_json(data: dict, where: str) -> "DenseMlp":
        kind = _get(data, "kind", where)
        if kind not in MLP_KINDS:
            raise ConfigError(f"config.json: {where}'kind' {kind!r} is not supported (supported: {', '.join(MLP_KINDS)})")
        return DenseMlp(ff=_int(data, "ff", where))

    def to_json(self) -> dict:
        return {"ff": self.ff, "kind": "dense"}


@dataclass(frozen=True)
class LagelornLayer:
    type: str
    mixer: DeltaMixer | ParallelMixer
    mlp: DenseMlp | None


@dataclass(frozen=True)
class LagelornConfig:
    vocab_size: int
    width: int
    max_positions: int
    norm_eps: float
    alpha: float          # a layer's sums are norm(alpha x + sublayer(x))
    side_dim: int         # width of a token's own row for one layer; 0: no side input
    logit_softcap: float  # 0: plain logits
    layers: tuple[LagelornLayer, ...]

    eos_token_id = None  # the design names no end-of-sequence token

    @staticmethod
    def from_json(data: dict) -> "LagelornConfig":
        layers_json = _get(data, "layers", "")
        if not isinstance(layers_json, list) or not layers_json:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(layers_json):
            where = f"layers[{i}]."
            kind = _get(entry, "type", where)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}'type' {kind!r} is not supported (supported: {', '.join(MIXER_TYPES)})")
            mixer = (DeltaMixer if kind == "delta" else ParallelMixer).from_json(_get(entry, "mixer", where), where + "mixer.")
            mlp_json = entry.get("mlp")
            layers.append(LagelornLayer(kind, mixer, None if mlp_json is None else DenseMlp.from_json(mlp_json, where + "mlp.")))
        side = _optional(data, "token_side")
        return LagelornConfig(
            vocab_size=_int(data, "vocab", ""), width=_int(data, "width", ""), max_positions=_int(data, "max_positions", ""),
            norm_eps=_number(_get(data, "norm", ""), "eps", "norm."), alpha=_number_or_one(data, "postln_alpha", ""),
            side_dim=_int(side, "dim", "token_side.") if side is not None else 0,
            logit_softcap=_number(data, "logit_softcap", "") if data.get("logit_softcap") is not None else 0.0, layers=tuple(layers))

    def to_json(self) -> dict:
        out = {"architecture": NAME, "max_positions": self.max_positions, "norm": {"eps": self.norm_eps}, "postln_alpha": self.alpha,
               "vocab": self.vocab_size, "width": self.width,
               "layers": [{"mixer": layer.mixer.to_json(), "mlp": None if layer.mlp is None else layer.mlp.to_json(), "type": layer.type}
                          for layer in self.layers]}
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        return out
