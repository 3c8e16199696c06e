"""Typed view of a Dubarax ``config.json``.

The file lists its layers one by one: ``layers[i] = {"type", "mixer", "mlp"}``.  ``type`` names the mixer (``parallel``,
``attention``, ``mamba2``; a numeric suffix, as in ``attention_2``, marks a further set of sizes of the same kind), ``mixer``
holds its sizes and constants, ``mlp`` the feed-forward or null for a layer without one.

* ``parallel``: ``left`` = ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size`` (the chunk); ``right`` =
  ``heads``, ``dim``, ``vdim``, ``decay`` (one number per head); ``left_scale``, ``right_scale``.
* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap``, ``mask.size`` (the window), ``bias_max``.
* ``mamba2``: ``heads``, ``vdim``, ``state``, ``groups``, ``conv``, ``norm_groups``.
* ``mlp.kind`` ``moe``: ``router.experts``, ``router.top``, ``router.groups.count``, ``router.groups.keep``, ``expert.ff`` and
  optionally ``shared.ff``.

Top level: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``loop`` = ``start``, ``stop``, ``times``: the layers ``start``
to ``stop - 1`` run ``times`` times in a row.  Every size and constant is read from the file; a missing key, a wrong type or
an unknown kind is an error that names the key.  Parts that a file leaves out (``loop``, ``embedding``, ``router.groups``,
``softcap``, ``mlp.shared``) are switched off.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

from .fields import need as _need, positive as _positive
from .model_config import ConfigError

ARCHITECTURE = "Dubarax"


def _heads(d: dict, where: str):
    """(heads, kv_heads, dim, vdim, scale, mask.size)"""
    heads = _positive(_need(d, "heads", int, where), where + ".heads")
    kv = _positive(_need(d, "kv_heads", int, where, default=heads, required=False), where + ".kv_heads")
    if heads % kv:
        raise ConfigError(f"config.json: '{where}.heads' must be a multiple of '{where}.kv_heads'")
    dim = _positive(_need(d, "dim", int, where), where + ".dim")
    vdim = _positive(_need(d, "vdim", int, where, default=dim, required=False), where + ".vdim")
    size = _positive(_need(_need(d, "mask", dict, where), "size", int, where + ".mask"), where + ".mask.size")
    return heads, kv, dim, vdim, _need(d, "scale", float, where), size


@dataclass
class ChunkAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "ChunkAttentionConfig":
        return cls(*_heads(d, where))


@dataclass
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: list                       # one number per head

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "LightningConfig":
        heads = _positive(_need(d, "heads", int, where), where + ".heads")
        dim = _positive(_need(d, "dim", int, where), where + ".dim")
        vdim = _positive(_need(d, "vdim", int, where, default=dim, required=False), where + ".vdim")
        decay = d.get("decay")
        if (not isinstance(decay, list) or len(decay) != heads
                or any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in decay)):
            raise ConfigError(f"config.json: '{where}.decay' must be a list of one number per head ({heads})")
        return cls(heads, dim, vdim, [float(x) for x in decay])


@dataclass
class ParallelConfig:
    left: ChunkAttentionConfig
    right: LightningConfig
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "ParallelConfig":
        return cls(ChunkAttentionConfig.from_dict(_need(d, "left", dict, where), where + ".left"),
                   LightningConfig.from_dict(_need(d, "right", dict, where), where + ".right"),
                   _need(d, "left_scale", float, where), _need(d, "right_scale", float, where))


@dataclass
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    softcap: float                    # 0: scores are not capped
    bias_max: int                     # where the logarithmic scale of the learned distance table ends

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "WindowAttentionConfig":
        cap = _need(d, "softcap", float, where, default=0.0, required=False)
        if cap < 0:
            raise ConfigError(f"config.json: '{where}.softcap' must not be negative")
        return cls(*_heads(d, where), cap, _positive(_need(d, "bias_max", int, where), where + ".bias_max"))


@dataclass
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "StateSpaceConfig":
        out = cls(*(_positive(_need(d, k, int, where), f"{where}.{k}") for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
        if out.heads % out.groups:
            raise ConfigError(f"config.json: '{where}.heads' must be a multiple of '{where}.groups'")
        if (out.heads * out.vdim) % out.norm_groups:
            raise ConfigError(f"config.json: '{where}.norm_groups' must divide heads * vdim")
        return out


@dataclass
class MoeConfig:
    experts: int
    top: int
    ff: int
    groups: Optional[tuple]           # (count, keep)
    shared_ff: int                    # 0: no shared expert

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "MoeConfig":
        kind = _need(d, "kind", str, where)
        if kind != "moe":
            raise ConfigError(f"config.json: '{where}.kind' is {kind!r}; known: moe")
        r, w = _need(d, "router", dict, where), where + ".router"
        experts = _positive(_need(r, "experts", int, w), w + ".experts")
        top = _positive(_need(r, "top", int, w), w + ".top")
        if top > experts:
            raise ConfigError(f"config.json: '{w}.top' must be at most '{w}.experts'")
        groups = None
        if r.get("groups") is not None:
            g, w = _need(r, "groups", dict, w), w + ".groups"
            count, keep = _positive(_need(g, "count", int, w), w + ".count"), _positive(_need(g, "keep", int, w), w + ".keep")
            if experts % count:
                raise ConfigError(f"config.json: '{w}.count' must divide the number of experts")
            if keep > count or keep * (experts // count) < top:
                raise ConfigError(f"config.json: '{w}.keep' must be at most '{w}.count' and leave enough experts to choose from")
            groups = (count, keep)
        ff = _positive(_need(_need(d, "expert", dict, where), "ff", int, where + ".expert"), where + ".expert.ff")
        shared = 0
        if d.get("shared") is not None:
            shared = _positive(_need(_need(d, "shared", dict, where), "ff", int, where + ".shared"), where + ".shared.ff")
        return cls(experts, top, ff, groups, shared)


@dataclass
class LoopConfig:
    start: int
    stop: int
    times: int

    @classmethod
    def from_dict(cls, d: dict, layers: int) -> "LoopConfig":
        out = cls(*(_need(d, k, int, "loop") for k in ("start", "stop", "times")))
        if not 0 <= out.start < out.stop <= layers:
            raise ConfigError(f"config.json: 'loop.start' and 'loop.stop' must name a stretch of the {layers} layers")
        _positive(out.times, "loop.times")
        return out


MIXER_KINDS = {"parallel": ParallelConfig, "attention": WindowAttentionConfig, "mamba2": StateSpaceConfig}


def _kind_of(name: str) -> str:
    if name in MIXER_KINDS:
        return name
    head, sep, tail = name.rpartition("_")
    return head if sep and tail.isdigit() and head else name


@dataclass
class DubaraxLayer:
    type: str
    mixer: object
    mlp: Optional[MoeConfig]


@dataclass
class DubaraxConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    eps: float
    embed_scale: float
    loop: Optional[LoopConfig]
    layers: list = field(default_factory=list)
    raw: dict = field(default_factory=dict)
    eos_token_id: int = -1

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict) -> "DubaraxConfig":
        layers_raw = d.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: key 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(layers_raw):
            where = f"layers[{i}]"
            typ = _need(L, "type", str, where)
            kind = MIXER_KINDS.get(_kind_of(typ))
            if kind is None:
                raise ConfigError(f"config.json: '{where}.type' is {typ!r}; known: {', '.join(sorted(MIXER_KINDS))} "
                                  "(with a numeric suffix for further sets of sizes)")
            mixer = kind.from_dict(_need(L, "mixer", dict, where), where + ".mixer")
            mlp = MoeConfig.from_dict(L["mlp"], where + ".mlp") if L.get("mlp") is not None else None
            layers.append(DubaraxLayer(typ, mixer, mlp))
        scale = 1.0
        if d.get("embedding") is not None:
            scale = _need(d["embedding"], "scale", float, "embedding", default=1.0, required=False)
        loop = LoopConfig.from_dict(_need(d, "loop", dict, ""), len(layers)) if d.get("loop") is not None else None
        eos = d.get("eos_token_id", -1)
        return cls(architecture=d.get("architecture", ARCHITECTURE),
                   vocab_size=_positive(_need(d, "vocab", int, ""), "vocab"),
                   hidden_size=_positive(_need(d, "width", int, ""), "width"),
                   eps=_need(_need(d, "norm", dict, ""), "eps", float, "norm"), embed_scale=scale, loop=loop, layers=layers,
                   raw=dict(d), eos_token_id=int(eos) if isinstance(eos, int) and not isinstance(eos, bool) else -1)

    def to_dict(self) -> dict:
        return dict(self.raw)
