"""Decoders whose layers choose their mixer one by one: configuration and weights.

A :class:`HybridConfig` is a list of layers, each with a mixer (a kind of attention or a
recurrence, with its own sizes and constants) and a feed-forward or none.  A
:class:`HybridLM` holds the weights the way the serving step wants them; the step itself, with the
cache and the recurrent state, is :class:`coeus_b200.infer.hybrid_engine.HybridEngine`.

What a design fixes for all its models is a :class:`Design`; the mixers are open to every design:

* Sapasun: a parallel block (mixer and feed-forward read the same residual stream through two
  norms), chunked attention with short convolutions, sinks, value mixing and head gates, and a
  gated delta rule with per-channel decay.
* Bananex: norms before and after each sublayer, a token shift in front of every mixer, a run of
  layers that is looped with the embedding fed in again, and latent attention under a sliding
  window, Mamba-2 and minGRU layers.
* Rupasun: norms before and after each sublayer, differential attention over the whole context,
  attention under a sliding window with normalised queries and keys, capped scores and an output
  gate, and feed-forwards that are dense or a mixture of experts with a shared one.
* Dogilorn: layer norms in front of each sublayer and layer scales behind it, a short convolution in
  front of every mixer, attention under a sliding window that keeps the first tokens, whose keys and
  values layers can share, and feed-forwards that are a bounded gated unit or a mixture of experts among
  which some pass their input on.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, ClassVar, Dict, List, Mapping, NamedTuple, Optional, Tuple, Union

import torch

from ..foundation.error import ConfigError, ProcessingError

MAX_HEAD_DIM = 256           # the attention and recurrence kernels' limit per head
MAX_LATENT = 640             # and per cached latent row
MAX_TAPS = 17                # and of the convolution kernels
MAX_WIDTH = 16384            # and of the pass between two sublayers
MAX_EXPERTS, MAX_TOP = 256, 16   # and of the routing kernels
DEFAULT_MAX_SEQ_LEN = 8192   # serving default; the designs themselves have no length limit

Shapes = Dict[str, Tuple[int, ...]]


@dataclass(frozen=True)
class Design:
    """The constants of a design."""

    name: str
    mixers: Mapping[str, str]    # type of a layer in a configuration file -> kind of mixer
    parallel: bool           # mixer and feed-forward side by side on one stream, else one by one
    post_norms: bool         # sublayer results are normalised before they are added
    scalar_norms: bool       # the gain of a norm of the stream is one number
    embed_norm: bool
    token_shift: bool
    act: str                 # of the dense feed-forward
    mlp_bias: bool
    mlps: Mapping[str, str] = field(default_factory=lambda: _same("dense"))   # name in a file -> kind
    scaled_logits: bool = False
    layer_norms: bool = False     # norms of the stream subtract the mean and have a bias
    layer_scale: bool = False     # sublayer results times a vector
    input_conv: bool = False      # a mixer reads h + conv(h)
    scaled_embed: bool = False
    tied_head: bool = False       # the logits' matrix is the embedding table


def _same(*kinds: str) -> Dict[str, str]:
    return {k: k for k in kinds}


DESIGNS = {d.name: d for d in (
    Design("Sapasun", _same("attention", "channel_delta"), parallel=True, post_norms=False,
           scalar_norms=False, embed_norm=True, token_shift=False, act="relu2", mlp_bias=False),
    Design("Bananex", _same("latent_attention", "mamba2", "mingru"), parallel=False, post_norms=True,
           scalar_norms=True, embed_norm=False, token_shift=True, act="gelu_erf", mlp_bias=True,
           scaled_logits=True),
    Design("Rupasun", {"attention": "diff_attention", "attention_2": "capped_attention"}, parallel=False,
           post_norms=True, scalar_norms=False, embed_norm=False, token_shift=False, act="relu2",
           mlp_bias=False, mlps=_same("dense", "moe")),
    Design("Dogilorn", {"attention": "kept_window_attention"}, parallel=False, post_norms=False,
           scalar_norms=False, embed_norm=False, token_shift=False, act="none", mlp_bias=True,
           mlps={"dense": "glu", "moe": "softmax_moe"}, layer_norms=True, layer_scale=True, input_conv=True,
           scaled_embed=True, tied_head=True),
)}
ARCHITECTURES = tuple(DESIGNS)


def _refuse(where: str, value, why: str) -> None:
    raise ConfigError.invalid(where, value, why)


def _heads_ok(where: str, *dims: int) -> None:
    if not all(1 <= d <= MAX_HEAD_DIM for d in dims):
        _refuse(where, "/".join(map(str, dims)), f"Head sizes must lie in 1..{MAX_HEAD_DIM}")


def _taps_ok(where: str, taps: int) -> None:
    if not 1 <= taps <= MAX_TAPS:
        _refuse(where, taps, f"A convolution has 1 to {MAX_TAPS} taps")


@dataclass(frozen=True)
class AttentionSpec:
    kind: ClassVar[str] = "attention"
    heads: int
    kv_heads: int
    dim: int                 # per-head query/key size
    vdim: int                # per-head value size
    conv: int                # taps of the short convolution on q, k and v
    scale: float
    chunk: Optional[int]     # positions of one chunk see each other, none outside
    rot_dims: int
    rot_base: float
    v_mix: bool

    @classmethod
    def read(cls, m: Mapping[str, Any], shapes: Mapping[str, Any], p: str) -> "AttentionSpec":
        rot, mask = m.get("rot"), m.get("mask")
        return cls(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                   vdim=int(m["vdim"]), conv=int(m["conv"]), scale=float(m["scale"]),
                   chunk=int(mask["size"]) if mask else None,
                   rot_dims=int(rot["dims"]) if rot else 0,
                   rot_base=float(rot["base"]) if rot else 1.0, v_mix=bool(m.get("v_mix", False)))

    def to_json(self) -> Dict[str, Any]:
        out: Dict[str, Any] = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim,
                                   vdim=self.vdim, conv=self.conv, scale=self.scale, v_mix=self.v_mix)
        if self.chunk is not None:
            out["mask"] = {"size": self.chunk}
        if self.rot_dims:
            out["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return out

    def check(self, where: str) -> None:
        if self.kv_heads < 1 or self.heads < 1 or self.heads % self.kv_heads:
            _refuse(where, f"{self.heads}/{self.kv_heads}",
                    "Key/value heads must divide the number of heads")
        _heads_ok(where, self.dim, self.vdim)
        _taps_ok(where, self.conv)
        if self.rot_dims % 2 or not 0 <= self.rot_dims <= self.dim:
            _refuse(where, self.rot_dims, "Rotated dimensions must be even and fit the head")
        if self.chunk is not None and self.chunk < 1:
            _refuse(where, self.chunk, "A chunk has at least one position")

    def tensors(self, W: int) -> Shapes:
        rows = {"q": self.heads * self.dim, "k": self.kv_heads * self.dim,
                "v": self.kv_heads * self.vdim}
        out: Shapes = {"sink": (self.heads,), "g": (self.heads, W)}
        if self.v_mix:
            out["vmix"] = ()
        for n, r in rows.items():
            out[n], out[n + ".conv"] = (r, W), (r, self.conv)
        return out

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class ChannelDeltaSpec:
    kind: ClassVar[str] = "channel_delta"
    heads: int               # value heads
    kv_heads: int            # query/key heads
    dim: int
    vdim: int
    conv: int
    decay_rank: int          # width between the two factors of the decay projection
    gate_rank: int           # and of the output-gate projection

    @classmethod
    def read(cls, m: Mapping[str, Any], shapes: Mapping[str, Any], p: str) -> "ChannelDeltaSpec":
        return cls(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                   vdim=int(m["vdim"]), conv=int(m["conv"]), decay_rank=_rank(shapes, p + "a1"),
                   gate_rank=_rank(shapes, p + "g1"))

    def to_json(self) -> Dict[str, Any]:
        return dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim,
                    conv=self.conv)

    def check(self, where: str) -> None:
        if self.kv_heads < 1 or self.heads < 1 or self.heads % self.kv_heads:
            _refuse(where, f"{self.heads}/{self.kv_heads}",
                    "Key/value heads must divide the number of heads")
        _heads_ok(where, self.dim, self.vdim)
        _taps_ok(where, self.conv)

    def tensors(self, W: int) -> Shapes:
        H, qk, v = self.heads, self.kv_heads * self.dim, self.heads * self.vdim
        out: Shapes = {"b": (H, W), "A_log": (H,), "norm": (self.vdim,), "a1": (self.decay_rank, W),
                       "a2": (H * self.dim, self.decay_rank), "dt_bias": (H * self.dim,),
                       "g1": (self.gate_rank, W), "g2": (v, self.gate_rank)}
        for n, r in (("q", qk), ("k", qk), ("v", v)):
            out[n], out[n + ".conv"] = (r, W), (r, self.conv)
        return out

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class LatentAttentionSpec:
    kind: ClassVar[str] = "latent_attention"
    heads: int
    dim: int                 # unrotated query/key size per head
    rot_dim: int             # rotated query/key size per head; the key's is shared by all heads
    vdim: int
    kv_rank: int             # numbers per token that keys and values are made from
    scale: float
    window: Optional[int]    # a position sees itself and window - 1 before it
    rot_base: float

    @classmethod
    def read(cls, m: Mapping[str, Any], shapes: Mapping[str, Any], p: str) -> "LatentAttentionSpec":
        rot, mask = m.get("rot"), m.get("mask")
        if rot and int(rot.get("dims", m["rot_dim"])) != int(m["rot_dim"]):
            _refuse(p + "rot", rot["dims"], "The rotated part is rotated as a whole")
        return cls(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]),
                   vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                   window=int(mask["size"]) if mask else None,
                   rot_base=float(rot["base"]) if rot else 1.0)

    def to_json(self) -> Dict[str, Any]:
        out: Dict[str, Any] = dict(heads=self.heads, dim=self.dim, rot_dim=self.rot_dim,
                                   vdim=self.vdim, kv_rank=self.kv_rank, scale=self.scale,
                                   rot={"base": self.rot_base, "dims": self.rot_dim})
        if self.window is not None:
            out["mask"] = {"size": self.window}
        return out

    def check(self, where: str) -> None:
        if self.heads < 1:
            _refuse(where, self.heads, "Attention needs a head")
        _heads_ok(where, self.dim + self.rot_dim, self.dim, self.vdim)
        if self.rot_dim % 2 or self.rot_dim < 2:
            _refuse(where, self.rot_dim, "Rotated dimensions must be even")
        if self.kv_rank < 1 or self.latent > MAX_LATENT:
            _refuse(where, self.kv_rank, f"A cached row holds 1 to {MAX_LATENT} numbers")
        if self.window is not None and self.window < 1:
            _refuse(where, self.window, "A window has at least one position")

    def tensors(self, W: int) -> Shapes:
        H, r = self.heads, self.kv_rank
        return {"q": (H * (self.dim + self.rot_dim), W), "dkv": (r + self.rot_dim, W), "dkv.norm": (r,),
                "uk": (H * self.dim, r), "uv": (H * self.vdim, r), "g": (H * self.vdim, W)}

    @property
    def latent(self) -> int:
        return self.kv_rank + self.rot_dim

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class Mamba2Spec:
    kind: ClassVar[str] = "mamba2"
    heads: int
    vdim: int
    state: int
    groups: int              # of heads that share B and C
    conv: int
    norm_groups: int         # equal parts of the output norm

    @classmethod
    def read(cls, m: Mapping[str, Any], shapes: Mapping[str, Any], p: str) -> "Mamba2Spec":
        return cls(**{k: int(m[k]) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")})

    def to_json(self) -> Dict[str, Any]:
        return dict(heads=self.heads, vdim=self.vdim, state=self.state, groups=self.groups,
                    conv=self.conv, norm_groups=self.norm_groups)

    def check(self, where: str) -> None:
        if self.heads < 1 or self.groups < 1 or self.heads % self.groups:
            _refuse(where, f"{self.heads}/{self.groups}", "Groups must divide the number of heads")
        if self.norm_groups < 1 or self.out_dim % self.norm_groups:
            _refuse(where, self.norm_groups, "The parts of the output norm must be equal")
        if self.vdim < 1:
            _refuse(where, self.vdim, "Heads have at least one column")
        _heads_ok(where, self.state)
        _taps_ok(where, self.conv)

    @property
    def channels(self) -> int:
        return self.out_dim + 2 * self.groups * self.state

    def tensors(self, W: int) -> Shapes:
        H, c = self.heads, self.channels
        return {"in": (self.out_dim + c + H, W), "conv": (c, self.conv), "conv.b": (c,),
                "dt_bias": (H,), "A_log": (H,), "D": (H,), "norm": (self.out_dim,)}

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class MinGruSpec:
    kind: ClassVar[str] = "mingru"
    width: int

    @classmethod
    def read(cls, m: Mapping[str, Any], shapes: Mapping[str, Any], p: str) -> "MinGruSpec":
        return cls(width=int(m["width"]))

    def to_json(self) -> Dict[str, Any]:
        return dict(width=self.width)

    def check(self, where: str) -> None:
        if self.width < 1:
            _refuse(where, self.width, "A recurrence has at least one channel")

    def tensors(self, W: int) -> Shapes:
        n = self.width
        return {"z": (n, W), "z.b": (n,), "x": (n, W), "x.b": (n,), "g": (n, W)}

    @property
    def out_dim(self) -> int:
        return self.width


@dataclass(frozen=True)
class HeadAttentionSpec:
    """Softmax attention of rotated heads straight from the projections.  What a kind fixes are class
    attributes, what its models choose are fields."""

    kind: ClassVar[str]
    maps: ClassVar[int] = 1             # attention maps per head, over the same values
    interleaved: ClassVar[bool] = False  # rotated pairs are neighbours, else half a rotation apart
    unit_qk: ClassVar[bool] = False     # rotated queries and keys are divided by their root mean square
    gated: ClassVar[bool] = False       # the output times the sigmoid of a projection, number by number
    row_norms: ClassVar[bool] = False   # RMS norms of q and of k over all heads at once, before the rotation
    unit_v: ClassVar[bool] = False      # each head's value is divided by its root mean square
    tempered: ClassVar[bool] = False    # a head's scores times a number of its own
    beside_one: ClassVar[bool] = False  # one more term exp(0) in the softmax's denominator

    heads: int
    kv_heads: int
    dim: int                 # query/key size per head and map
    vdim: int
    scale: float
    rot_dims: int
    rot_base: float
    window: Optional[int] = None        # a position sees itself and window - 1 before it
    softcap: Optional[float] = None     # scores s become softcap * tanh(s / softcap)
    diff: Optional[float] = None        # two maps: what their weights add to
    keep_first: int = 0                 # positions that stay visible when the window has passed them
    kv_from: Optional[int] = None       # the layer whose keys and values this one uses

    @classmethod
    def read(cls, m: Mapping[str, Any], shapes: Mapping[str, Any], p: str) -> "HeadAttentionSpec":
        rot, mask, cap = m.get("rot"), m.get("mask"), m.get("softcap")
        return cls(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                   vdim=int(m["vdim"]), scale=float(m["scale"]), rot_dims=int(rot["dims"]) if rot else 0,
                   rot_base=float(rot["base"]) if rot else 1.0,
                   window=int(mask["size"]) if mask else None,
                   softcap=None if cap is None else float(cap),
                   diff=float(m["diff"]) if cls.maps == 2 else None,
                   keep_first=int(mask.get("keep_first") or 0) if mask else 0,
                   kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))

    def to_json(self) -> Dict[str, Any]:
        out: Dict[str, Any] = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim,
                                   vdim=self.vdim, scale=self.scale)
        if self.rot_dims:
            out["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        if self.window is not None:
            out["mask"] = {"size": self.window}
            if self.keep_first:
                out["mask"]["keep_first"] = self.keep_first
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        if self.softcap is not None:
            out["softcap"] = self.softcap
        if self.diff is not None:
            out["diff"] = self.diff
        return out

    def check(self, where: str) -> None:
        if self.kv_heads < 1 or self.heads < 1 or self.heads % self.kv_heads:
            _refuse(where, f"{self.heads}/{self.kv_heads}",
                    "Key/value heads must divide the number of heads")
        _heads_ok(where, self.dim, self.vdim)
        if self.rot_dims % 2 or not 0 <= self.rot_dims <= self.dim:
            _refuse(where, self.rot_dims, "Rotated dimensions must be even and fit the head")
        if self.window is not None and self.window < 1:
            _refuse(where, self.window, "A window has at least one position")
        if self.keep_first < 0 or (self.keep_first and self.window is None):
            _refuse(where, self.keep_first, "Only a window keeps first positions")
        if self.softcap is not None and not self.softcap > 0:
            _refuse(where, self.softcap, "A cap of scores is positive")
        if (self.diff is not None) != (self.maps == 2):
            _refuse(where, self.diff, "Two maps, and only two, need the constant of their difference")

    def tensors(self, W: int) -> Shapes:
        out: Shapes = {"q": (self.heads * self.maps * self.dim, W)}
        if self.kv_from is None:
            out.update({"k": (self.kv_heads * self.maps * self.dim, W), "v": (self.kv_heads * self.vdim, W)})
        if self.row_norms:
            out.update({n + ".norm": out[n][:1] for n in "qk" if n in out})
        if self.tempered:
            out["temp"] = (self.heads,)
        if self.maps == 2:
            out.update({n: (self.dim,) for n in MAP_VECTORS})
        if self.gated:
            out["g"] = (self.out_dim, W)
        return out

    @property
    def score_max(self) -> float:
        """A bound on scores before the cap, with room for the rounding of q and k to bf16; 0: none."""
        return 1.02 * self.dim * abs(self.scale) if self.unit_qk else 0.0

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim


MAP_VECTORS = ("lq1", "lk1", "lq2", "lk2")    # exp(lq1 . lk1) - exp(lq2 . lk2) + diff weighs the second map


@dataclass(frozen=True)
class DiffAttentionSpec(HeadAttentionSpec):
    """Two maps over the same values; the head is their weighted difference, divided by its root mean
    square, times ``1 - diff``."""

    kind: ClassVar[str] = "diff_attention"
    maps: ClassVar[int] = 2


@dataclass(frozen=True)
class CappedAttentionSpec(HeadAttentionSpec):
    kind: ClassVar[str] = "capped_attention"
    interleaved: ClassVar[bool] = True
    unit_qk: ClassVar[bool] = True
    gated: ClassVar[bool] = True


@dataclass(frozen=True)
class KeptWindowAttentionSpec(HeadAttentionSpec):
    """A sliding window beside which the first positions stay visible."""

    kind: ClassVar[str] = "kept_window_attention"
    interleaved: ClassVar[bool] = True
    row_norms: ClassVar[bool] = True
    unit_v: ClassVar[bool] = True
    tempered: ClassVar[bool] = True
    beside_one: ClassVar[bool] = True


MixerSpec = Union[AttentionSpec, ChannelDeltaSpec, LatentAttentionSpec, Mamba2Spec, MinGruSpec,
                  HeadAttentionSpec]
MIXERS = {c.kind: c for c in (AttentionSpec, ChannelDeltaSpec, LatentAttentionSpec, Mamba2Spec,
                              MinGruSpec, DiffAttentionSpec, CappedAttentionSpec, KeptWindowAttentionSpec)}
# mixers that look back through the paged cache
CACHED = (AttentionSpec, LatentAttentionSpec, HeadAttentionSpec)


@dataclass(frozen=True)
class MlpSpec:
    """down(act(up))."""

    kind: ClassVar[str] = "dense"
    ff: int

    @classmethod
    def read(cls, m: Mapping[str, Any]) -> "MlpSpec":
        return cls(ff=int(m["ff"]))

    def to_json(self) -> Dict[str, Any]:
        return dict(ff=self.ff)

    def check(self, where: str) -> None:
        if self.ff < 1:
            _refuse(where, self.ff, "A feed-forward has at least one channel")

    def tensors(self, W: int, bias: bool) -> Shapes:
        out: Shapes = {"up": (self.ff, W), "down": (W, self.ff)}
        if bias:
            out.update({"up.b": (self.ff,), "down.b": (W,)})
        return out


@dataclass(frozen=True)
class GluMlpSpec:
    """``down(g * sigmoid(slope * g) * (u + shift))``, ``g`` (of ``gate``) bounded by ``limit`` above and ``u``
    (of ``up``) on both sides."""

    kind: ClassVar[str] = "glu"
    slope: ClassVar[float] = 1.702
    shift: ClassVar[float] = 1.0
    ff: int
    limit: float

    @classmethod
    def read(cls, m: Mapping[str, Any]) -> "GluMlpSpec":
        return cls(ff=int(m["ff"]), limit=float(m["limit"]))

    def to_json(self) -> Dict[str, Any]:
        return dict(ff=self.ff, limit=self.limit)

    def check(self, where: str) -> None:
        if self.ff < 1 or not self.limit > 0:
            _refuse(where, f"{self.ff}/{self.limit}", "A feed-forward has a channel and a positive limit")

    def tensors(self, W: int, bias: bool) -> Shapes:
        out: Shapes = {"gate": (self.ff, W), "up": (self.ff, W), "down": (W, self.ff)}
        if bias:
            out.update({n + ".b": out[n][:1] for n in ("gate", "up", "down")})
        return out


@dataclass(frozen=True)
class GluSpec:
    """An expert: the same unit without biases, bounded or (``limit`` infinite) not."""

    ff: int
    limit: float = math.inf

    @classmethod
    def read(cls, m: Mapping[str, Any], bounded: bool = True) -> "GluSpec":
        return cls(ff=int(m["ff"]), limit=float(m["limit"]) if bounded else math.inf)

    def to_json(self) -> Dict[str, Any]:
        return dict(ff=self.ff) if math.isinf(self.limit) else dict(ff=self.ff, limit=self.limit)

    def tensors(self, W: int, p: str) -> Shapes:
        return {p + "gate": (self.ff, W), p + "up": (self.ff, W), p + "down": (W, self.ff)}


@dataclass(frozen=True)
class MoeSpec:
    """Every token uses the ``top`` of ``experts`` with the largest scores among the ``keep`` best of
    ``groups`` equal groups of neighbours, weighted by their scores times ``scale``; and the shared expert,
    if there is one.  Class attributes are what a kind fixes."""

    kind: ClassVar[str] = "moe"
    softmax: ClassVar[bool] = False      # scores are a softmax over all experts, else sigmoids
    corrected: ClassVar[bool] = False    # a number per expert is added to its score for the choice only
    group_best: ClassVar[int] = 2        # a group counts the sum of so many of its largest scores
    normalised: ClassVar[bool] = True    # weights are divided by their sum
    shared_gate: ClassVar[bool] = False  # the shared expert times the sigmoid of a projection
    slope: ClassVar[float] = 1.702       # of the experts' gated unit
    shift: ClassVar[float] = 1.0
    bounded: ClassVar[bool] = True

    experts: int
    top: int
    expert: GluSpec
    scale: float = 1.0
    groups: int = 1
    keep: int = 1
    shared: Optional[GluSpec] = None
    identity: int = 0                    # experts behind the others whose result is their input

    @classmethod
    def read(cls, m: Mapping[str, Any]) -> "MoeSpec":
        r = m["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}
        return cls(experts=int(r["experts"]), top=int(r["top"]), expert=GluSpec.read(m["expert"], cls.bounded),
                   scale=float(r.get("scale", 1.0)), groups=int(groups["count"]), keep=int(groups["keep"]),
                   shared=GluSpec.read(m["shared"], cls.bounded) if m.get("shared") else None,
                   identity=int(r.get("identity") or 0))

    def to_json(self) -> Dict[str, Any]:
        router: Dict[str, Any] = dict(experts=self.experts, top=self.top,
                                      groups=dict(count=self.groups, keep=self.keep))
        if self.normalised or self.scale != 1.0:
            router["scale"] = self.scale
        if self.identity:
            router["identity"] = self.identity
        out: Dict[str, Any] = dict(expert=self.expert.to_json(), router=router)
        if self.shared is not None:
            out["shared"] = self.shared.to_json()
        return out

    def check(self, where: str) -> None:
        if self.experts < 1 or self.identity < 0 or self.outputs > MAX_EXPERTS or not 1 <= self.top <= MAX_TOP:
            _refuse(where, f"{self.top} of {self.outputs}",
                    f"Up to {MAX_TOP} of up to {MAX_EXPERTS} experts are chosen")
        if self.groups < 1 or self.outputs % self.groups or not 1 <= self.keep <= self.groups:
            _refuse(where, f"{self.keep} of {self.groups}", "Groups must be equal, and one of them kept")
        if self.top > self.keep * (self.outputs // self.groups):
            _refuse(where, self.top, "The kept groups must hold enough experts")
        for g in (self.expert, self.shared):
            if g is not None and (g.ff < 1 or not g.limit > 0):
                _refuse(where, f"{g.ff}/{g.limit}", "An expert has a channel and a positive limit")

    @property
    def outputs(self) -> int:
        """Of the router."""
        return self.experts + self.identity

    def routing(self):
        from ..ops.experts import Routing
        return Routing(self.experts, self.top, self.groups, self.keep, self.scale, self.identity, self.softmax,
                       self.group_best, self.normalised, self.shared_gate and self.shared is not None)

    def tensors(self, W: int, bias: bool) -> Shapes:
        out: Shapes = {"router": (self.outputs, W)}
        if self.corrected:
            out["correction"] = (self.outputs,)
        for e in range(self.experts):
            out.update(self.expert.tensors(W, f"e{e}."))
        if self.shared is not None:
            out.update(self.shared.tensors(W, "shared."))
            if self.shared_gate:
                out["shared.sg"] = (1, W)
        return out


@dataclass(frozen=True)
class SoftmaxMoeSpec(MoeSpec):
    kind: ClassVar[str] = "softmax_moe"
    softmax: ClassVar[bool] = True
    corrected: ClassVar[bool] = True
    group_best: ClassVar[int] = 1
    normalised: ClassVar[bool] = False
    shared_gate: ClassVar[bool] = True
    slope: ClassVar[float] = 1.0
    shift: ClassVar[float] = 0.0
    bounded: ClassVar[bool] = False


FeedForwardSpec = Union[MlpSpec, GluMlpSpec, MoeSpec]
MLPS = {c.kind: c for c in (MlpSpec, GluMlpSpec, MoeSpec, SoftmaxMoeSpec)}


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    mlp: Optional[FeedForwardSpec]


@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start .. stop - 1`` run ``times`` times in a row with the same weights."""

    start: int
    stop: int
    times: int


class Run(NamedTuple):
    """One run of a layer; every run has its own cache or state."""

    layer: int
    starts: Optional[int]    # the number of the pass this run begins, if it begins one


@dataclass(frozen=True)
class HybridConfig:
    vocab_size: int
    hidden_dim: int
    layers: Tuple[LayerSpec, ...]
    norm_eps: float
    logit_softcap: Optional[float] = None
    architecture: str = "Sapasun"
    max_seq_len: int = DEFAULT_MAX_SEQ_LEN
    logit_scale: float = 1.0
    loop: Optional[LoopSpec] = None
    embed_scale: float = 1.0
    conv_taps: int = 0       # of the convolution in front of the mixers
    pos: str = field(default="rope", init=False)   # positions need no table of trained rows

    @property
    def design(self) -> Design:
        return DESIGNS[self.architecture]

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def width_padded(self) -> int:
        return _up8(self.hidden_dim)

    @property
    def vocab_padded(self) -> int:
        return _up8(self.vocab_size)

    def runs(self) -> List[Run]:
        """The layers in the order they run."""
        a, b, n = (self.loop.start, self.loop.stop, self.loop.times) if self.loop else (0, 0, 0)
        return [Run(i, None) for i in range(a)] + \
            [Run(i, t if i == a else None) for t in range(n) for i in range(a, b)] + \
            [Run(i, None) for i in range(b, self.num_layers)]

    def validate(self) -> None:
        if self.architecture not in DESIGNS:
            _refuse("architecture", self.architecture, f"Known designs: {', '.join(DESIGNS)}")
        if self.vocab_size < 1 or self.hidden_dim < 1 or not self.layers:
            _refuse("layers", self.num_layers, "A model needs a vocabulary, a width and layers")
        if self.hidden_dim > MAX_WIDTH:
            _refuse("width", self.hidden_dim, f"The width must not exceed {MAX_WIDTH}")
        mixing = None
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            where = f"layers[{i}].mixer"
            if m.kind not in self.design.mixers.values():
                _refuse(where, m.kind, f"{self.architecture} has {', '.join(self.design.mixers.values())}")
            m.check(where)
            if getattr(m, "v_mix", False):
                size = m.kv_heads * m.vdim
                if mixing not in (None, size):
                    _refuse(where, size, "Layers that mix values must agree in their size")
                mixing = size
            if layer.mlp is not None:
                if layer.mlp.kind not in self.design.mlps.values():
                    _refuse(f"layers[{i}].mlp", layer.mlp.kind,
                            f"Feed-forwards of {self.architecture}: {', '.join(self.design.mlps.values())}")
                layer.mlp.check(f"layers[{i}].mlp")
            if getattr(m, "kv_from", None) is not None:
                self._check_shared(i, m)
        if self.design.input_conv:
            _taps_ok("conv_taps", self.conv_taps)
        if self.loop is not None:
            lo = self.loop
            if self.design.parallel:
                _refuse("loop", lo, f"{self.architecture} has no loop")
            if not 0 <= lo.start < lo.stop <= self.num_layers or lo.times < 1:
                _refuse("loop", f"{lo.start}..{lo.stop} x {lo.times}", "The loop must be a run of layers")

    def _check_shared(self, i: int, m: "HeadAttentionSpec") -> None:
        where = f"layers[{i}].mixer.kv_from"
        if not 0 <= m.kv_from < i or self.loop is not None:
            _refuse(where, m.kv_from, "Keys and values come from an earlier layer")
        s = self.layers[m.kv_from].mixer
        if s.kind != m.kind or s.kv_from is not None:
            _refuse(where, m.kv_from, "Keys and values come from a layer that makes them")
        if (s.kv_heads, s.dim, s.vdim) != (m.kv_heads, m.dim, m.vdim):
            _refuse(where, m.kv_from, "Layers that share keys and values have the same key/value heads")

    def to_dict(self) -> Dict[str, Any]:
        return config_to_json(self)


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


def _rank(shapes: Mapping[str, Any], name: str) -> int:
    if name not in shapes:
        raise ProcessingError.invalid_input(f"missing tensor '{name}'")
    return int(shapes[name][0])


def config_from_json(config: Mapping[str, Any], shapes: Mapping[str, Any]) -> HybridConfig:
    """``config``: the parsed ``config.json``; ``shapes``: tensor name -> shape, which gives the
    sizes the file does not name (the inner widths of the factored projections)."""
    layers = []
    architecture = str(config.get("architecture", "Sapasun"))
    if architecture not in DESIGNS:
        raise ProcessingError.unsupported(f"architecture '{architecture}'", ", ".join(DESIGNS))
    design = DESIGNS[architecture]
    kinds = design.mixers
    for i, entry in enumerate(config["layers"]):
        if entry["type"] not in kinds:
            raise ProcessingError.unsupported(f"mixer type '{entry['type']}'", ", ".join(kinds))
        mixer = MIXERS[kinds[entry["type"]]].read(entry["mixer"], shapes, f"l{i}.mix.")
        mlp = entry.get("mlp")
        if mlp and mlp["kind"] not in design.mlps:
            raise ProcessingError.unsupported(f"feed-forward '{mlp['kind']}'", ", ".join(design.mlps))
        layers.append(LayerSpec(mixer, MLPS[design.mlps[mlp["kind"]]].read(mlp) if mlp else None))
    cap, loop = config.get("logit_softcap"), config.get("loop")
    cfg = HybridConfig(
        vocab_size=int(config["vocab"]), hidden_dim=int(config["width"]), layers=tuple(layers),
        norm_eps=float(config["norm"]["eps"]), logit_softcap=None if cap is None else float(cap),
        architecture=architecture,
        logit_scale=float(config.get("logit_scale", 1.0)) if design.scaled_logits else 1.0,
        embed_scale=float(config["embedding"]["scale"]) if design.scaled_embed else 1.0,
        conv_taps=int(config["canon"]["taps"]) if design.input_conv else 0,
        loop=None if not loop else LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"])))
    cfg.validate()
    return cfg


def config_to_json(cfg: HybridConfig) -> Dict[str, Any]:
    types = {kind: name for name, kind in cfg.design.mixers.items()}
    mlps = {kind: name for name, kind in cfg.design.mlps.items()}
    layers = [{"type": types[layer.mixer.kind], "mixer": layer.mixer.to_json(),
               "mlp": None if layer.mlp is None else dict(kind=mlps[layer.mlp.kind], **layer.mlp.to_json())}
              for layer in cfg.layers]
    out = {"architecture": cfg.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_dim,
           "norm": {"eps": cfg.norm_eps}, "layers": layers}
    if cfg.design.parallel:
        out["logit_softcap"] = cfg.logit_softcap
    elif cfg.design.scaled_logits:
        out["logit_scale"] = cfg.logit_scale
    if cfg.design.scaled_embed:
        out["embedding"] = {"scale": cfg.embed_scale}
    if cfg.design.input_conv:
        out["canon"] = {"taps": cfg.conv_taps}
    if cfg.loop is not None:
        out["loop"] = {"start": cfg.loop.start, "stop": cfg.loop.stop, "times": cfg.loop.times}
    return out


def tensor_shapes(cfg: HybridConfig) -> Shapes:
    """Every tensor of a checkpoint and its shape (linear weights ``[out, in]``)."""
    W, V, d = cfg.hidden_dim, cfg.vocab_size, cfg.design
    norm: Tuple[int, ...] = () if d.scalar_norms else (W,)
    out: Shapes = {"embed": (V, W)}
    if d.embed_norm:
        out["embed.norm"] = norm
    if cfg.loop is not None:
        out.update({"loop.in": (W, 2 * W), "loop.step": (cfg.loop.times, W)})
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        for n in ("norm1", "norm2")[:1 if layer.mlp is None else 2]:
            out[p + n] = norm
            if d.post_norms:
                out[p + n + "b"] = norm
            if d.layer_norms:
                out[p + n + ".b"] = norm
            if d.layer_scale:
                out[p + "ls" + n[4:]] = (W,)
        if d.token_shift:
            out[p + "shift"] = (W,)
        if d.input_conv:
            out[p + "canon1"] = (W, cfg.conv_taps)
        out.update({f"{p}mix.{n}": s for n, s in layer.mixer.tensors(W).items()})
        out[p + "mix.o"] = (W, layer.mixer.out_dim)
        if layer.mlp is not None:
            out.update({f"{p}mlp.{n}": s for n, s in layer.mlp.tensors(W, d.mlp_bias).items()})
    out["final.norm"] = norm
    if d.layer_norms:
        out["final.norm.b"] = norm
    if not d.tied_head:
        out["head"] = (V, W)
    return out


def random_state(cfg: HybridConfig, seed: int = 0, device="cpu",
                 dtype: torch.dtype = torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random weights of a configuration, scaled so that activations stay of order one."""
    gen = torch.Generator(device=device)
    gen.manual_seed(seed)

    def normal(shape, std):
        return torch.randn(shape, generator=gen, device=device) * std
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf.startswith("norm") or leaf in ("ls1", "ls2", "temp"):
            t = 1.0 + normal(shape, 0.1)
        elif leaf == "canon1":
            t = normal(shape, 0.3)
        elif leaf == "embed" and cfg.design.tied_head:
            t = normal(shape, shape[-1] ** -0.5)
        elif leaf == "correction":
            t = normal(shape, 0.1)
        elif leaf == "conv":
            t = normal(shape, 0.3)
            t[:, -1] += 1.0
        elif leaf in ("embed", "D"):
            t = normal(shape, 1.0)
        elif leaf in ("sink", "vmix", "A_log", "dt_bias"):
            t = normal(shape, 0.5)
        elif leaf in MAP_VECTORS or leaf == "step" or (leaf == "b" and len(shape) == 1):
            t = normal(shape, 0.2)
        elif leaf == "shift":
            t = torch.sigmoid(normal(shape, 1.0))
        else:
            t = normal(shape, shape[-1] ** -0.5)
        out[name] = t.to(dtype)
    return out


def _pad(t: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    out = torch.zeros((rows, cols), dtype=t.dtype, device=t.device)
    out[:t.shape[0], :t.shape[1]] = t
    return out


def _alternate(a: torch.Tensor, b: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    """Rows of ``a`` and ``b`` in turn, each padded to ``rows x cols``."""
    return torch.stack([_pad(a, rows, cols), _pad(b, rows, cols)], 1).view(2 * rows, cols)


class Experts:
    """Device weights of a mixture of experts.  Rows of gate and up alternate (``w_in [experts, 2 ff, W]``),
    so that a tile of the product has both numbers of a channel; ``w_down [experts, W, ff]``; the shared
    expert's ``s_in`` and ``s_down`` likewise."""

    def __init__(self, spec: MoeSpec, mat, vec, wp: int) -> None:
        self.spec, self.wp = spec, wp
        self.slope, self.shift = spec.slope, spec.shift
        self.routing = spec.routing()
        router = mat("mlp.router")
        if self.routing.shared_gate:          # one more output of the same product
            router = torch.cat([router, mat("mlp.shared.sg")])
        self.router = _pad(router, _up8(router.shape[0]), wp)
        self.correction = vec("mlp.correction") if spec.corrected else None

        def pair(p: str, g: GluSpec):
            return _alternate(mat(p + "gate"), mat(p + "up"), _up8(g.ff), wp), _pad(mat(p + "down"), wp, _up8(g.ff))
        ws = [pair(f"mlp.e{e}.", spec.expert) for e in range(spec.experts)]
        self.w_in, self.w_down = (torch.stack(t).contiguous() for t in zip(*ws))
        self.s_in, self.s_down = pair("mlp.shared.", spec.shared) if spec.shared else (None, None)

    def tensors(self, W: int) -> Dict[str, torch.Tensor]:
        s = self.spec
        out = {"router": self.router[:s.outputs, :W]}
        if self.correction is not None:
            out["correction"] = self.correction
        if self.routing.shared_gate:
            out["shared.sg"] = self.router[s.outputs:s.outputs + 1, :W]

        def apart(p: str, w_in: torch.Tensor, down: torch.Tensor, ff: int) -> None:
            out.update({p + "gate": w_in[0:2 * ff:2, :W], p + "up": w_in[1:2 * ff:2, :W],
                        p + "down": down[:W, :ff]})
        for e in range(s.experts):
            apart(f"e{e}.", self.w_in[e], self.w_down[e], s.expert.ff)
        if s.shared is not None:
            apart("shared.", self.s_in, self.s_down, s.shared.ff)
        return out


class HybridLayer:
    """Device weights of one layer.  ``w_in`` stacks every projection of the mixer's input (each
    segment starts at a multiple of eight rows, ``seg[name]`` is its first output column; ``b_in``
    the biases, where a segment has one).  In a parallel block ``w_out`` puts the mixer's output
    projection and the feed-forward's down projection side by side: both are added to the same
    stream, so they are one product over ``[mixer output | activation]``, the activation starting at
    column ``act_off``.  Otherwise ``w_out`` is the mixer's output projection and ``w_down`` the
    feed-forward's.  A feed-forward with a gated unit has the rows of its gate and up projections in
    turn in ``w_up`` (and their biases in ``b_up``)."""

    def __init__(self, spec: LayerSpec, design: Design, w_get, width: int, dtype: torch.dtype) -> None:
        self.spec, self.dtype = spec, dtype
        self._get = w_get
        self.wp = _up8(width)
        self.norm1 = self._gain("norm1", design)
        self.norm1b = self._gain("norm1b", design) if design.post_norms else None
        self.center1 = self._vec("norm1.b", self.wp) if design.layer_norms else None
        self.scale1 = self._vec("ls1", self.wp) if design.layer_scale else None
        self.center2 = self.scale2 = self.taps = None
        if design.input_conv:         # taps-major
            t = w_get("canon1").float()
            self.taps = _pad(t.t(), t.shape[1], self.wp)
        self.shift = self._vec("shift", self.wp) if design.token_shift else None
        self.seg: Dict[str, int] = {}
        {"attention": self._attention, "channel_delta": self._channel_delta,
         "latent_attention": self._latent, "mamba2": self._mamba2, "mingru": self._mingru,
         "diff_attention": self._heads, "capped_attention": self._heads,
         "kept_window_attention": self._heads}[spec.mixer.kind](spec.mixer)
        self.out_dim = spec.mixer.out_dim
        self.act_off = _up8(self.out_dim)
        outs = [_pad(self._mat("mix.o"), self.wp, self.act_off)]
        self.norm2 = self.norm2b = self.w_up = self.b_up = self.w_down = self.b_down = None
        self.ff = self.ff_padded = 0
        self.experts: Optional[Experts] = None
        if spec.mlp is not None:
            self.norm2 = self._gain("norm2", design)
            self.norm2b = self._gain("norm2b", design) if design.post_norms else None
            self.center2 = self._vec("norm2.b", self.wp) if design.layer_norms else None
            self.scale2 = self._vec("ls2", self.wp) if design.layer_scale else None
        self.glu: Optional[Tuple[float, float, float]] = None
        if isinstance(spec.mlp, MoeSpec):
            self.experts = Experts(spec.mlp, self._mat, self._vec, self.wp)
        elif spec.mlp is not None:
            self.ff, self.ff_padded = spec.mlp.ff, _up8(spec.mlp.ff)
            if isinstance(spec.mlp, GluMlpSpec):
                self.glu = (spec.mlp.slope, spec.mlp.limit, spec.mlp.shift)
                self.w_up = _alternate(self._mat("mlp.gate"), self._mat("mlp.up"), self.ff_padded, self.wp)
            else:
                self.w_up = _pad(self._mat("mlp.up"), self.ff_padded, self.wp)
            down = _pad(self._mat("mlp.down"), self.wp, self.ff_padded)
            if design.parallel:
                outs.append(down)
            else:
                self.w_down = down
            if design.mlp_bias:
                self.b_up = self._vec("mlp.up.b", self.ff_padded).to(dtype)
                if self.glu is not None:
                    self.b_up = torch.stack([self._vec("mlp.gate.b", self.ff_padded).to(dtype), self.b_up],
                                            1).flatten()
                self.b_down = self._vec("mlp.down.b", self.wp)
        self.w_out = torch.cat(outs, 1).contiguous()
        del self._get

    def _mat(self, name: str) -> torch.Tensor:
        return self._get(name).to(self.dtype)

    def _vec(self, name: str, pad: int = 0) -> torch.Tensor:
        t = self._get(name).float()
        return torch.nn.functional.pad(t, (0, pad - t.numel())).contiguous() if pad else t.contiguous()

    def _gain(self, name: str, design: Design) -> torch.Tensor:
        return self._vec(name).reshape(1) if design.scalar_norms else self._vec(name, self.wp)

    def _stack(self, parts: Mapping[str, torch.Tensor], biases: Optional[Mapping[str, torch.Tensor]] = None
               ) -> None:
        blocks, at = [], 0
        for n, t in parts.items():
            self.seg[n] = at
            blocks.append(_pad(t, _up8(t.shape[0]), self.wp))
            at += blocks[-1].shape[0]
        self.w_in = torch.cat(blocks).contiguous()
        self.b_in = None
        if biases:
            self.b_in = torch.zeros(at, dtype=self.dtype, device=self.w_in.device)
            for n, b in biases.items():
                self.b_in[self.seg[n]:self.seg[n] + b.numel()] = b.to(self.dtype)

    def _conv_qkv(self) -> None:      # taps-major, channels q | k | v
        self.conv = torch.cat([self._get(f"mix.{n}.conv").float() for n in "qkv"]).t().contiguous()
        self.channels = self.conv.shape[1]

    def _attention(self, m: AttentionSpec) -> None:
        self._stack({n: self._mat("mix." + n) for n in ("q", "k", "v", "g")})
        self._conv_qkv()
        self.sink = self._vec("mix.sink")
        self.mix = self._vec("mix.vmix").reshape(1) if m.v_mix else None
        self.rope_key = (m.rot_base, m.rot_dims) if m.rot_dims else None

    def _channel_delta(self, m: ChannelDeltaSpec) -> None:
        self._stack({n: self._mat("mix." + n) for n in ("q", "k", "v", "b", "a1", "g1")})
        self._conv_qkv()
        self.A_log, self.dt_bias = self._vec("mix.A_log"), self._vec("mix.dt_bias")
        self.head_norm = self._vec("mix.norm")
        self.w_a2 = _pad(self._mat("mix.a2"), _up8(m.heads * m.dim), _up8(m.decay_rank))
        self.w_g2 = _pad(self._mat("mix.g2"), _up8(m.heads * m.vdim), _up8(m.gate_rank))

    def _latent(self, m: LatentAttentionSpec) -> None:
        """``w_kv [2, heads, P, latent]`` makes every head's key (its rotated part copied from the
        cached row by unit rows) and value from cached rows; ``w_absorb [heads, latent, P]`` is its
        key part transposed, which brings a query to the cached rows instead."""
        from ..ops.latent import head_pitch
        self._stack({n: self._mat("mix." + n) for n in ("q", "dkv", "g")})
        self.latent_norm = self._vec("mix.dkv.norm")
        self.rope_key = (m.rot_base, m.rot_dim)
        H, r, P = m.heads, m.kv_rank, head_pitch(m.dim + m.rot_dim, m.vdim)
        w = torch.zeros((2, H, P, _up8(m.latent)), dtype=self.dtype, device=self.w_in.device)
        w[0, :, :m.dim, :r] = self._mat("mix.uk").view(H, m.dim, r)
        for i in range(m.rot_dim):
            w[0, :, m.dim + i, r + i] = 1.0
        w[1, :, :m.vdim, :r] = self._mat("mix.uv").view(H, m.vdim, r)
        self.w_kv = w
        self.w_absorb = w[0].transpose(1, 2).contiguous()
        self.w_value = w[1, :, :m.vdim].contiguous()

    def _mamba2(self, m: Mamba2Spec) -> None:
        """The convolved channels are ``x | B | C``, each starting at a multiple of eight."""
        bc = m.groups * m.state
        sizes = dict(z=m.out_dim, x=m.out_dim, B=bc, C=bc, dt=m.heads)
        self._stack(dict(zip(sizes, torch.split(self._mat("mix.in"), list(sizes.values())))))
        pads = [(n, _up8(sizes[n])) for n in ("x", "B", "C")]
        self.boff, self.coff = pads[0][1], pads[0][1] + pads[1][1]
        self.channels = sum(p for _, p in pads)

        def spread(t: torch.Tensor) -> torch.Tensor:
            parts = torch.split(t, [sizes[n] for n, _ in pads])
            return torch.cat([_pad(x, p, t.shape[1]) for x, (_, p) in zip(parts, pads)])
        self.conv = spread(self._get("mix.conv").float()).t().contiguous()
        self.conv_b = spread(self._vec("mix.conv.b")[:, None])[:, 0].contiguous()
        self.dt_bias, self.A_log, self.D = (self._vec("mix." + n) for n in ("dt_bias", "A_log", "D"))
        self.out_norm = self._vec("mix.norm")

    def _mingru(self, m: MinGruSpec) -> None:
        self._stack({n: self._mat("mix." + n) for n in ("z", "x", "g")},
                    {n: self._get(f"mix.{n}.b") for n in ("z", "x")})

    def _heads(self, m: HeadAttentionSpec) -> None:
        shapes = m.tensors(self.wp)
        self._stack({n: self._mat("mix." + n) for n in "qkvg" if n in shapes})
        self.q_norm, self.k_norm = (self._vec(f"mix.{n}.norm") if n + ".norm" in shapes else None for n in "qk")
        self.temp = self._vec("mix.temp") if m.tempered else None
        # a term exp(0) in the softmax's denominator is a sink of score 0
        self.sink = torch.zeros(m.heads, device=self.w_in.device) if m.beside_one else None
        self.rope_key = (m.rot_base, m.rot_dims) if m.rot_dims else None
        self.map_vectors = self.map_weight = None
        if m.maps == 2:
            self.map_vectors = {n: self._vec("mix." + n) for n in MAP_VECTORS}
            a, b, c, d = (self.map_vectors[n].double() for n in MAP_VECTORS)
            self.map_weight = ((a * b).sum().exp() - (c * d).sum().exp() + m.diff).float().reshape(1)

    # ------------------------------------------------------------------ taken apart again
    def tensors(self, width: int) -> Dict[str, torch.Tensor]:
        """The layer's tensors under their names in a checkpoint (without the layer's prefix)."""
        m, W = self.spec.mixer, width
        shapes = m.tensors(W)
        out = {"norm1": self.norm1, "mix.o": self.w_out[:W, :self.out_dim]}

        def stacked(names):
            for n in names:
                out["mix." + n] = self.w_in[self.seg[n]:self.seg[n] + shapes[n][0], :W]
        if isinstance(m, (AttentionSpec, ChannelDeltaSpec)):
            c = 0
            for n in "qkv":
                r = shapes[n][0]
                out[f"mix.{n}.conv"] = self.conv[:, c:c + r].t()
                c += r
        if isinstance(m, AttentionSpec):
            stacked(("q", "k", "v", "g"))
            out["mix.sink"] = self.sink
            if self.mix is not None:
                out["mix.vmix"] = self.mix
        elif isinstance(m, ChannelDeltaSpec):
            stacked(("q", "k", "v", "b", "a1", "g1"))
            out.update({"mix.A_log": self.A_log, "mix.dt_bias": self.dt_bias, "mix.norm": self.head_norm})
            for n, t in (("a2", self.w_a2), ("g2", self.w_g2)):
                out["mix." + n] = t[:shapes[n][0], :shapes[n][1]]
        elif isinstance(m, LatentAttentionSpec):
            stacked(("q", "dkv", "g"))
            out["mix.dkv.norm"] = self.latent_norm
            out["mix.uk"] = self.w_kv[0, :, :m.dim, :m.kv_rank].reshape(shapes["uk"])
            out["mix.uv"] = self.w_kv[1, :, :m.vdim, :m.kv_rank].reshape(shapes["uv"])
        elif isinstance(m, Mamba2Spec):
            bc = m.groups * m.state
            sizes = dict(z=m.out_dim, x=m.out_dim, B=bc, C=bc, dt=m.heads)
            out["mix.in"] = torch.cat([self.w_in[self.seg[n]:self.seg[n] + r, :W] for n, r in sizes.items()])
            at = {"x": 0, "B": self.boff, "C": self.coff}
            idx = torch.cat([torch.arange(at[n], at[n] + sizes[n]) for n in at]).to(self.conv.device)
            out.update({"mix.conv": self.conv[:, idx].t(), "mix.conv.b": self.conv_b[idx],
                        "mix.dt_bias": self.dt_bias, "mix.A_log": self.A_log, "mix.D": self.D,
                        "mix.norm": self.out_norm})
        elif isinstance(m, HeadAttentionSpec):
            stacked(n for n in ("q", "k", "v", "g") if n in shapes)
            out.update({"mix." + n: t for n, t in (("q.norm", self.q_norm), ("k.norm", self.k_norm),
                                                   ("temp", self.temp)) if t is not None})
            out.update({"mix." + n: t for n, t in (self.map_vectors or {}).items()})
        else:
            stacked(("z", "x", "g"))
            for n in ("z", "x"):
                out[f"mix.{n}.b"] = self.b_in[self.seg[n]:self.seg[n] + m.width]
        for n, t in (("norm1b", self.norm1b), ("norm2", self.norm2), ("norm2b", self.norm2b), ("shift", self.shift),
                     ("norm1.b", self.center1), ("norm2.b", self.center2), ("ls1", self.scale1), ("ls2", self.scale2)):
            if t is not None:
                out[n] = t
        if self.taps is not None:
            out["canon1"] = self.taps[:, :W].t()
        if self.experts is not None:
            out.update({"mlp." + n: t for n, t in self.experts.tensors(W).items()})
        if self.w_up is not None:
            out["mlp.up"] = self.w_up[:self.ff, :W]
            if self.glu is not None:
                out["mlp.gate"], out["mlp.up"] = (self.w_up[i:2 * self.ff:2, :W] for i in (0, 1))
            out["mlp.down"] = self.w_out[:W, self.act_off:self.act_off + self.ff] \
                if self.w_down is None else self.w_down[:W, :self.ff]
            if self.b_up is not None:
                out["mlp.up.b"], out["mlp.down.b"] = self.b_up[:self.ff], self.b_down[:W]
                if self.glu is not None:
                    out["mlp.gate.b"], out["mlp.up.b"] = (self.b_up[i:2 * self.ff:2] for i in (0, 1))
        return out


class HybridLM:
    """Weights of a hybrid decoder on one device, in bf16 (the serving precision) or fp32."""

    def __init__(self, cfg: HybridConfig, state: Mapping[str, torch.Tensor], device="cuda",
                 dtype: Optional[torch.dtype] = None) -> None:
        cfg.validate()
        self.cfg = cfg
        self.device = torch.device(device)
        self.dtype = dtype or (torch.bfloat16 if self.device.type == "cuda" else torch.float32)
        if self.dtype not in (torch.bfloat16, torch.float32):
            raise ProcessingError.unsupported(f"working dtype {self.dtype}", "bf16 and fp32")
        shapes = tensor_shapes(cfg)

        def get(name: str) -> torch.Tensor:
            if name not in state:
                raise ProcessingError.invalid_input(f"missing tensor '{name}'")
            t = state[name]
            if tuple(t.shape) != shapes[name]:
                raise ProcessingError.invalid_input(
                    f"tensor '{name}' has shape {tuple(t.shape)}, expected {shapes[name]}")
            return t.to(self.device)
        W, wp, design = cfg.hidden_dim, cfg.width_padded, cfg.design

        def gain(name):
            t = get(name).float()
            return t.reshape(1) if design.scalar_norms else \
                torch.nn.functional.pad(t, (0, wp - W)).contiguous()
        self.embed = _pad(get("embed").to(self.dtype), cfg.vocab_padded if design.tied_head else cfg.vocab_size, wp)
        self.embed_norm = gain("embed.norm") if design.embed_norm else None
        self.loop_in = self.loop_step = None
        if cfg.loop is not None:       # [W, 2 W] with the padding of each half behind it
            a, b = get("loop.in").to(self.dtype).split(W, 1)
            self.loop_in = torch.cat([_pad(a, wp, wp), _pad(b, wp, wp)], 1).contiguous()
            self.loop_step = _pad(get("loop.step").float(), cfg.loop.times, wp)
        self.layers = [HybridLayer(spec, design, lambda n, i=i: get(f"l{i}.{n}"), W, self.dtype)
                       for i, spec in enumerate(cfg.layers)]
        self.final_norm = gain("final.norm")
        # the logits' factor rides on the last norm's gain
        self.final_gain = self.final_norm * cfg.logit_scale
        self.final_center = gain("final.norm.b") * cfg.logit_scale if design.layer_norms else None
        self.head = self.embed if design.tied_head else _pad(get("head").to(self.dtype), cfg.vocab_padded, wp)
        # rotary frequencies base^(-2i/dims), one table per distinct (base, dims)
        self.inv_freq: Dict[Tuple[float, int], torch.Tensor] = {}
        for layer in self.layers:
            key = getattr(layer, "rope_key", None)
            if key is not None and key not in self.inv_freq:
                base, dims = key
                f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
                self.inv_freq[key] = torch.tensor(f, dtype=torch.float32, device=self.device)
        self._shapes = shapes

    @classmethod
    def random(cls, cfg: HybridConfig, device="cuda", seed: int = 0,
               dtype: Optional[torch.dtype] = None) -> "HybridLM":
        return cls(cfg, random_state(cfg, seed, device), device, dtype)

    def num_parameters(self) -> int:
        return sum(_size(shape) for shape in self._shapes.values())

    def make_engine(self, **kw):
        from ..infer.hybrid_engine import HybridEngine
        return HybridEngine(self, **kw)

    def state_dict(self) -> Dict[str, torch.Tensor]:
        """The checkpoint's tensors, taken apart again."""
        cfg, W = self.cfg, self.cfg.hidden_dim
        out = {"embed": self.embed[:cfg.vocab_size, :W], "final.norm": self.final_norm[:W]}
        if not cfg.design.tied_head:
            out["head"] = self.head[:cfg.vocab_size, :W]
        if self.final_center is not None:
            out["final.norm.b"] = self.final_center[:W] / cfg.logit_scale
        if self.embed_norm is not None:
            out["embed.norm"] = self.embed_norm[:W]
        if self.loop_in is not None:
            wp = cfg.width_padded
            out["loop.in"] = torch.cat([self.loop_in[:W, :W], self.loop_in[:W, wp:wp + W]], 1)
            out["loop.step"] = self.loop_step[:, :W]
        for i, layer in enumerate(self.layers):
            out.update({f"l{i}.{n}": t for n, t in layer.tensors(W).items()})
        return {n: t.detach().flatten()[:_size(self._shapes[n])].reshape(self._shapes[n]).cpu()
                .contiguous().clone() if t.dim() < 2 else t.detach().cpu().contiguous().clone()
                for n, t in out.items()}


def _size(shape: Tuple[int, ...]) -> int:
    n = 1
    for s in shape:
        n *= s
    return n


def load_hybrid(state: Mapping[str, torch.Tensor], config: Mapping[str, Any], device="cuda",
                training: bool = False, dtype: Optional[torch.dtype] = None) -> HybridLM:
    if training:
        raise ProcessingError.unsupported(f"training a {config.get('architecture')} model",
                                          "the hybrid decoders are served only")
    cfg = config_from_json(config, {n: tuple(t.shape) for n, t in state.items()})
    return HybridLM(cfg, state, device, dtype)


def export_hybrid(lm: HybridLM):
    return {n: t.to(torch.bfloat16) for n, t in lm.state_dict().items()}, config_to_json(lm.cfg)
