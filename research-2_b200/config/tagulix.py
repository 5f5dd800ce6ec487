"""The typed Tagulix configuration, read from the design's own config.json keys.

A Tagulix config.json names its model with `"architecture": "Tagulix"` and lists its layers one by one: every entry of
`layers` gives the layer's `type` (which mixer it has: `attention`, rotated queries and keys inside a sliding window, or
`parallel`, attention with a learned bias by distance beside linear attention with a fixed decay per head), the mixer's sizes and
constants (`mixer`), its feed-forward (`mlp`: `kind` `moe`, or null for a layer without one), and optionally `weights_of: j` for a
layer that runs with layer j's tensors and a cache and state of its own. Beside the layers stand `vocab`, `width`, `norm.eps`,
`streams` (how many copies of the residual stream run side by side) and `residual_mult`, the factor on what joins them. No size has a
default: a size that is missing is an error that names it. The rows of a bias table are the checkpoint's own. A mechanism that a file
does not mention is not there: no `mask` (or no `mask.size`) is no window, no `rot` no rotation, no `q_temp` queries that do not
depend on the position, no `router.groups` one group of all, no `router.identity` no identity outputs, no `streams` the plain
residual sum; factors left out are one, `kv_heads` and `vdim` left out equal `heads` and `dim`.
"""

from __future__ import annotations

from dataclasses import dataclass, replace

from .lagelorn import _heads
from .registry import ConfigError
from .zirunex import _get, _int, _number
from .zudalorn import Rotation, _optional

NAME = "Tagulix"
MIXER_TYPES = ("attention", "parallel")
MLP_KINDS = ("moe",)


def _value_size(data: dict, dim: int, where: str) -> int:
    return _int(data, "vdim", where) if data.get("vdim") is not None else dim


@dataclass(frozen=True)
class WindowAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float          # scores are (q . k) * scale
    window: int           # mask.size: position i sees j when 0 <= i - j < window; 0: every j <= i
    rot: Rotation | None

    @staticmethod
    def from_json(data: dict, where: str) -> "WindowAttention":
        dim = _int(data, "dim", where)
        heads, kv_heads = _heads(data, where)
        mask, rot = _optional(data, "mask"), _optional(data, "rot")
        return WindowAttention(
            heads=heads, kv_heads=kv_heads, dim=dim, vdim=_value_size(data, dim, where), scale=_number(data, "scale", where),
            window=_int(mask, "size", where + "mask.") if _optional(mask, "size") is not None else 0,
            rot=Rotation.from_json(rot, where + "rot.", dim) if rot is not None else None)

    def to_json(self) -> dict:
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.window:
            out["mask"] = {"size": self.window}
        if self.rot is not None:
            out["rot"] = self.rot.to_json()
        return out


@dataclass(frozen=True)
class BiasedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float       # scores are (q . k) * scale, then the bias
    bias_max: int      # farther keys share the bias table's last row
    temp_coef: float   # queries at position p are multiplied by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1); 0: by one
    temp_every: int

    @staticmethod
    def from_json(data: dict, where: str) -> "BiasedAttention":
        dim = _int(data, "dim", where)
        heads, kv_heads = _heads(data, where)
        temp = _optional(data, "q_temp")
        return BiasedAttention(
            heads=heads, kv_heads=kv_heads, dim=dim, vdim=_value_size(data, dim, where), scale=_number(data, "scale", where),
            bias_max=_int(data, "bias_max", where, minimum=2),
            temp_coef=_number(temp, "coef", where + "q_temp.", positive=False) if temp is not None else 0.0,
            temp_every=_int(temp, "every", where + "q_temp.") if temp is not None else 1)

    def to_json(self) -> dict:
        out = {"bias_max": self.bias_max, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.temp_coef:
            out["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        return out


@dataclass(frozen=True)
class DecayAttention:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]   # one factor per head

    @staticmethod
    def from_json(data: dict, where: str) -> "DecayAttention":
        heads, dim, decay = _int(data, "heads", where), _int(data, "dim", where), _get(data, "decay", where)
        if not isinstance(decay, list) or len(decay) != heads:
            raise ConfigError(f"config.json: {where}'decay' must list one number for each of the {heads} heads")
        return DecayAttention(heads=heads, dim=dim, vdim=_value_size(data, dim, where),
                              decay=tuple(_number({"decay": d}, "decay", where, positive=False) for d in decay))

    def to_json(self) -> dict:
        return {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}


@dataclass(frozen=True)
class ParallelMixer:
    left: BiasedAttention
    right: DecayAttention
    left_scale: float
    right_scale: float

    @staticmethod
    def from_json(data: dict, where: str) -> "ParallelMixer":
        def factor(key):
            return _number(data, key, where, positive=False) if key in data else 1.0

        return ParallelMixer(left=BiasedAttention.from_json(_get(data, "left", where), where + "left."),
                             right=DecayAttention.from_json(_get(data, "right", where), where + "right."),
                             left_scale=factor("left_scale"), right_scale=factor("right_scale"))

    def to_json(self) -> dict:
        return {"left": self.left.to_json(), "left_scale": self.left_scale, "right": self.right.to_json(), "right_scale": self.right_scale}


@dataclass(frozen=True)
class ExpertsMlp:
    experts: int
    identity: int       # router outputs after the experts' that give the input back
    top: int
    ff: int             # inner width of an expert
    groups: int         # experts and identity outputs together form this many equal groups of neighbours ...
    keep_groups: int    # ... and only those of the best keep_groups groups can be chosen
    scale: float        # the chosen ones' weights sum to it

    @staticmethod
    def from_json(data: dict, where: str) -> "ExpertsMlp":
        kind = _get(data, "kind", where)
        if kind not in MLP_KINDS:
            raise ConfigError(f"config.json: {where}'kind' {kind!r} is not supported (supported: {', '.join(MLP_KINDS)})")
        router, expert, at = _get(data, "router", where), _get(data, "expert", where), where + "router."
        experts, top = _int(router, "experts", at), _int(router, "top", at)
        identity = _int(router, "identity", at, minimum=0) if router.get("identity") is not None else 0
        groups_json = _optional(router, "groups")
        groups = _int(groups_json, "count", at + "groups.") if groups_json is not None else 1
        keep = _int(groups_json, "keep", at + "groups.") if groups_json is not None else 1
        total = experts + identity
        if total % groups or keep > groups:
            raise ConfigError(f"config.json: {at}groups: {groups} groups (keep {keep}) do not fit {total} router outputs")
        if top > total // groups * keep:
            raise ConfigError(f"config.json: {at}'top' ({top}) exceeds what can be chosen ({total // groups * keep})")
        return ExpertsMlp(experts=experts, identity=identity, top=top, ff=_int(expert, "ff", where + "expert."), groups=groups, keep_groups=keep,
                          scale=_number(router, "scale", at, positive=False) if "scale" in router else 1.0)

    def to_json(self) -> dict:
        return {"expert": {"ff": self.ff}, "kind": "moe",
                "router": {"experts": self.experts, "groups": {"count": self.groups, "keep": self.keep_groups}, "identity": self.identity,
                           "scale": self.scale, "top": self.top}}


@dataclass(frozen=True)
class TagulixLayer:
    type: str
    mixer: WindowAttention | ParallelMixer
    mlp: ExpertsMlp | None
    weights_of: int | None = None   # the layer whose tensors this one runs with; None: its own


@dataclass(frozen=True)
class TagulixConfig:
    vocab_size: int
    width: int
    norm_eps: float
    residual_mult: float
    streams: int        # copies of the residual stream; 0: the plain residual sum
    layers: tuple[TagulixLayer, ...]

    eos_token_id = None  # the design names no end-of-sequence token

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        j = self.layers[i].weights_of
        return i if j is None else j

    @staticmethod
    def from_json(data: dict) -> "TagulixConfig":
        layers_json = _get(data, "layers", "")
        if not isinstance(layers_json, list) or not layers_json:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: list[TagulixLayer] = []
        for i, entry in enumerate(layers_json):
            where = f"layers[{i}]."
            kind = _get(entry, "type", where)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}'type' {kind!r} is not supported (supported: {', '.join(MIXER_TYPES)})")
            mixer = (WindowAttention if kind == "attention" else ParallelMixer).from_json(_get(entry, "mixer", where), where + "mixer.")
            mlp_json, owner = entry.get("mlp"), entry.get("weights_of")
            if owner is not None and (isinstance(owner, bool) or not isinstance(owner, int) or not 0 <= owner < len(layers_json) or owner == i):
                raise ConfigError(f"config.json: {where}'weights_of' must name another layer, got {owner!r}")
            layers.append(TagulixLayer(kind, mixer, None if mlp_json is None else ExpertsMlp.from_json(mlp_json, where + "mlp."), owner))
        for i, layer in enumerate(layers):
            seen, j = {i}, layer.weights_of
            while j is not None and layers[j].weights_of is not None:   # a lender that borrows itself: follow to the owner
                if j in seen:
                    raise ConfigError(f"config.json: layers[{i}].'weights_of' leads in a circle")
                seen.add(j)
                j = layers[j].weights_of
            if j is None:
                continue
            if replace(layers[j], weights_of=None) != replace(layer, weights_of=None):
                raise ConfigError(f"config.json: layers[{i}] runs with the tensors of layer {j} but describes another layer")
            layers[i] = replace(layer, weights_of=j)
        return TagulixConfig(
            vocab_size=_int(data, "vocab", ""), width=_int(data, "width", ""), norm_eps=_number(_get(data, "norm", ""), "eps", "norm."),
            residual_mult=_number(data, "residual_mult", "", positive=False) if "residual_mult" in data else 1.0,
            streams=_int(data, "streams", "") if data.get("streams") is not None else 0, layers=tuple(layers))

    def to_json(self) -> dict:
        layers = []
        for layer in self.layers:
            entry = {"mixer": layer.mixer.to_json(), "mlp": None if layer.mlp is None else layer.mlp.to_json(), "type": layer.type}
            if layer.weights_of is not None:
                entry["weights_of"] = layer.weights_of
            layers.append(entry)
        out = {"architecture": NAME, "layers": layers, "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
               "vocab": self.vocab_size, "width": self.width}
        if self.streams:
            out["streams"] = self.streams
        return out
