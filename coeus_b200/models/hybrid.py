"""Decoders whose layers choose their mixer one by one: configuration and weights.

A :class:`HybridConfig` is a list of layers, each with a mixer (a kind of attention or a
recurrence, with its own sizes and constants) and a feed-forward or none.  A
:class:`HybridLM` holds the weights the way the serving step wants them; the step itself, with the
cache and the recurrent state, is :class:`coeus_b200.infer.hybrid_engine.HybridEngine`.

The design served this way is Sapasun: a parallel block (mixer and feed-forward read the same
residual stream through two norms), chunked attention with short convolutions, sinks, value mixing
and head gates, and a gated delta rule with per-channel decay.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Mapping, Optional, Tuple, Union

import torch

from ..foundation.error import ConfigError, ProcessingError

ARCHITECTURES = ("Sapasun",)
MAX_HEAD_DIM = 256           # the attention and recurrence kernels' limit per head
MAX_TAPS = 17                # and of the convolution kernels
DEFAULT_MAX_SEQ_LEN = 8192   # serving default; the design itself has no length limit


@dataclass(frozen=True)
class AttentionSpec:
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


@dataclass(frozen=True)
class ChannelDeltaSpec:
    heads: int               # value heads
    kv_heads: int            # query/key heads
    dim: int
    vdim: int
    conv: int
    decay_rank: int          # width between the two factors of the decay projection
    gate_rank: int           # and of the output-gate projection


@dataclass(frozen=True)
class MlpSpec:
    ff: int
    kind: str = "dense"      # down(relu(up)^2)


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, ChannelDeltaSpec]
    mlp: Optional[MlpSpec]


@dataclass(frozen=True)
class HybridConfig:
    vocab_size: int
    hidden_dim: int
    layers: Tuple[LayerSpec, ...]
    norm_eps: float
    logit_softcap: Optional[float]
    architecture: str = "Sapasun"
    max_seq_len: int = DEFAULT_MAX_SEQ_LEN
    pos: str = field(default="rope", init=False)   # positions need no table of trained rows

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def width_padded(self) -> int:
        return _up8(self.hidden_dim)

    @property
    def vocab_padded(self) -> int:
        return _up8(self.vocab_size)

    def attention_layers(self) -> List[int]:
        return [i for i, l in enumerate(self.layers) if isinstance(l.mixer, AttentionSpec)]

    def first_v_mix(self) -> Optional[int]:
        return next((i for i in self.attention_layers() if self.layers[i].mixer.v_mix), None)

    def validate(self) -> None:
        if self.vocab_size < 1 or self.hidden_dim < 1 or not self.layers:
            raise ConfigError.invalid("layers", self.num_layers,
                                      "A model needs a vocabulary, a width and layers")
        mixing = None
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            where = f"layers[{i}].mixer"
            if m.kv_heads < 1 or m.heads < 1 or m.heads % m.kv_heads:
                raise ConfigError.invalid(where, f"{m.heads}/{m.kv_heads}",
                                          "Key/value heads must divide the number of heads")
            if not (1 <= m.dim <= MAX_HEAD_DIM and 1 <= m.vdim <= MAX_HEAD_DIM):
                raise ConfigError.invalid(where, f"{m.dim}/{m.vdim}",
                                          f"Head sizes must lie in 1..{MAX_HEAD_DIM}")
            if not 1 <= m.conv <= MAX_TAPS:
                raise ConfigError.invalid(where, m.conv, f"A convolution has 1 to {MAX_TAPS} taps")
            if isinstance(m, AttentionSpec):
                if m.rot_dims % 2 or not 0 <= m.rot_dims <= m.dim:
                    raise ConfigError.invalid(where, m.rot_dims,
                                              "Rotated dimensions must be even and fit the head")
                if m.chunk is not None and m.chunk < 1:
                    raise ConfigError.invalid(where, m.chunk, "A chunk has at least one position")
                if m.v_mix:
                    size = m.kv_heads * m.vdim
                    if mixing not in (None, size):
                        raise ConfigError.invalid(where, size,
                                                  "Layers that mix values must agree in their size")
                    mixing = size
            if layer.mlp is not None and layer.mlp.kind != "dense":
                raise ConfigError.invalid(f"layers[{i}].mlp", layer.mlp.kind,
                                          "Feed-forward kind must be 'dense'")

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
    for i, entry in enumerate(config["layers"]):
        m, p = entry["mixer"], f"l{i}.mix."
        if entry["type"] == "attention":
            rot, mask = m.get("rot"), m.get("mask")
            mixer = AttentionSpec(
                heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                vdim=int(m["vdim"]), conv=int(m["conv"]), scale=float(m["scale"]),
                chunk=int(mask["size"]) if mask else None,
                rot_dims=int(rot["dims"]) if rot else 0,
                rot_base=float(rot["base"]) if rot else 1.0, v_mix=bool(m.get("v_mix", False)))
        elif entry["type"] == "channel_delta":
            mixer = ChannelDeltaSpec(
                heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                vdim=int(m["vdim"]), conv=int(m["conv"]), decay_rank=_rank(shapes, p + "a1"),
                gate_rank=_rank(shapes, p + "g1"))
        else:
            raise ProcessingError.unsupported(f"mixer type '{entry['type']}'",
                                              "attention and channel_delta")
        mlp = entry.get("mlp")
        layers.append(LayerSpec(mixer, None if mlp is None else
                                MlpSpec(ff=int(mlp["ff"]), kind=str(mlp["kind"]))))
    cap = config.get("logit_softcap")
    cfg = HybridConfig(
        vocab_size=int(config["vocab"]), hidden_dim=int(config["width"]), layers=tuple(layers),
        norm_eps=float(config["norm"]["eps"]), logit_softcap=None if cap is None else float(cap),
        architecture=str(config.get("architecture", "Sapasun")))
    cfg.validate()
    return cfg


def config_to_json(cfg: HybridConfig) -> Dict[str, Any]:
    layers = []
    for layer in cfg.layers:
        m = layer.mixer
        mixer: Dict[str, Any] = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim,
                                     conv=m.conv)
        if isinstance(m, AttentionSpec):
            kind = "attention"
            mixer.update(scale=m.scale, v_mix=m.v_mix)
            if m.chunk is not None:
                mixer["mask"] = {"size": m.chunk}
            if m.rot_dims:
                mixer["rot"] = {"base": m.rot_base, "dims": m.rot_dims}
        else:
            kind = "channel_delta"
        layers.append({"type": kind, "mixer": mixer, "mlp": None if layer.mlp is None else
                       {"kind": layer.mlp.kind, "ff": layer.mlp.ff}})
    return {"architecture": cfg.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_dim,
            "norm": {"eps": cfg.norm_eps}, "logit_softcap": cfg.logit_softcap, "layers": layers}


def tensor_shapes(cfg: HybridConfig) -> Dict[str, Tuple[int, ...]]:
    """Every tensor of a checkpoint and its shape (linear weights ``[out, in]``)."""
    W, V = cfg.hidden_dim, cfg.vocab_size
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, W), "embed.norm": (W,)}
    for i, layer in enumerate(cfg.layers):
        m, p = layer.mixer, f"l{i}."
        out[p + "norm1"] = (W,)
        if layer.mlp is not None:
            out[p + "norm2"] = (W,)
        x = p + "mix."
        if isinstance(m, AttentionSpec):
            rows = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
            out.update({x + "sink": (m.heads,), x + "g": (m.heads, W)})
            if m.v_mix:
                out[x + "vmix"] = ()
        else:
            rows = {"q": m.kv_heads * m.dim, "k": m.kv_heads * m.dim, "v": m.heads * m.vdim}
            out.update({x + "b": (m.heads, W), x + "A_log": (m.heads,), x + "norm": (m.vdim,),
                        x + "a1": (m.decay_rank, W), x + "a2": (m.heads * m.dim, m.decay_rank),
                        x + "dt_bias": (m.heads * m.dim,), x + "g1": (m.gate_rank, W),
                        x + "g2": (m.heads * m.vdim, m.gate_rank)})
        for n, r in rows.items():
            out[x + n] = (r, W)
            out[x + n + ".conv"] = (r, m.conv)
        out[x + "o"] = (W, m.heads * m.vdim)
        if layer.mlp is not None:
            out[p + "mlp.up"] = (layer.mlp.ff, W)
            out[p + "mlp.down"] = (W, layer.mlp.ff)
    out.update({"final.norm": (W,), "head": (V, W)})
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
        if leaf.startswith("norm"):
            t = 1.0 + normal(shape, 0.1)
        elif leaf == "conv":
            t = normal(shape, 0.3)
            t[:, -1] += 1.0
        elif leaf == "embed":
            t = normal(shape, 1.0)
        elif leaf in ("sink", "vmix", "A_log", "dt_bias"):
            t = normal(shape, 0.5)
        else:
            t = normal(shape, shape[-1] ** -0.5)
        out[name] = t.to(dtype)
    return out


def _pad(t: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    out = torch.zeros((rows, cols), dtype=t.dtype, device=t.device)
    out[:t.shape[0], :t.shape[1]] = t
    return out


class HybridLayer:
    """Device weights of one layer.  ``w_in`` stacks every projection of the normalised stream
    (each segment starts at a multiple of eight rows, ``seg[name]`` is its first output column),
    ``w_out`` puts the mixer's output projection and the feed-forward's down projection side by
    side: both are added to the same stream, so they are one product over
    ``[mixer output | activation]``, the activation starting at column ``act_off``."""

    def __init__(self, spec: LayerSpec, w_get, width: int, dtype: torch.dtype) -> None:
        self.spec = spec
        m = spec.mixer
        attn = isinstance(m, AttentionSpec)
        wp = _up8(width)

        def mat(name):
            return w_get(name).to(dtype)

        def vec(name, pad=0):
            t = w_get(name).float()
            return torch.nn.functional.pad(t, (0, pad - t.numel())).contiguous() if pad \
                else t.contiguous()
        self.norm1 = vec("norm1", wp)
        parts = ["q", "k", "v", "g"] if attn else ["q", "k", "v", "b", "a1", "g1"]
        self.seg: Dict[str, int] = {}
        blocks, at = [], 0
        for n in parts:
            t = mat("mix." + n)
            self.seg[n] = at
            blocks.append(_pad(t, _up8(t.shape[0]), wp))
            at += blocks[-1].shape[0]
        self.w_in = torch.cat(blocks).contiguous()
        # taps-major, channels q | k | v
        self.conv = torch.cat([w_get(f"mix.{n}.conv").float() for n in "qkv"]).t().contiguous()
        self.channels = self.conv.shape[1]
        if attn:
            self.sink = vec("mix.sink")
            self.mix = vec("mix.vmix").reshape(1) if m.v_mix else None
            half = m.rot_dims // 2
            self.rope_key = (m.rot_base, m.rot_dims) if half else None
        else:
            self.A_log, self.dt_bias = vec("mix.A_log"), vec("mix.dt_bias")
            self.head_norm = vec("mix.norm")
            self.w_a2 = _pad(mat("mix.a2"), _up8(m.heads * m.dim), _up8(m.decay_rank))
            self.w_g2 = _pad(mat("mix.g2"), _up8(m.heads * m.vdim), _up8(m.gate_rank))
        self.out_dim = m.heads * m.vdim
        self.act_off = _up8(self.out_dim)
        outs = [_pad(mat("mix.o"), wp, self.act_off)]
        self.norm2 = self.w_up = None
        self.ff = self.ff_padded = 0
        if spec.mlp is not None:
            self.norm2 = vec("norm2", wp)
            self.ff, self.ff_padded = spec.mlp.ff, _up8(spec.mlp.ff)
            self.w_up = _pad(mat("mlp.up"), self.ff_padded, wp)
            outs.append(_pad(mat("mlp.down"), wp, self.ff_padded))
        self.w_out = torch.cat(outs, 1).contiguous()


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
        W, wp = cfg.hidden_dim, cfg.width_padded

        def vec(name):
            return torch.nn.functional.pad(get(name).float(), (0, wp - W)).contiguous()
        self.embed = _pad(get("embed").to(self.dtype), cfg.vocab_size, wp)
        self.embed_norm = vec("embed.norm")
        self.layers = [HybridLayer(spec, lambda n, i=i: get(f"l{i}.{n}"), W, self.dtype)
                       for i, spec in enumerate(cfg.layers)]
        self.final_norm = vec("final.norm")
        self.head = _pad(get("head").to(self.dtype), cfg.vocab_padded, wp)
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
        n = 0
        for shape in self._shapes.values():
            k = 1
            for s in shape:
                k *= s
            n += k
        return n

    def make_engine(self, **kw):
        from ..infer.hybrid_engine import HybridEngine
        return HybridEngine(self, **kw)

    def state_dict(self) -> Dict[str, torch.Tensor]:
        """The checkpoint's tensors, taken apart again."""
        cfg, W = self.cfg, self.cfg.hidden_dim
        out = {"embed": self.embed[:, :W], "embed.norm": self.embed_norm[:W],
               "final.norm": self.final_norm[:W], "head": self.head[:cfg.vocab_size, :W]}
        for i, (layer, spec) in enumerate(zip(self.layers, cfg.layers)):
            p, x = f"l{i}.", f"l{i}.mix."
            out[p + "norm1"] = layer.norm1[:W]
            c = 0
            for n, at in layer.seg.items():
                rows = self._shapes[x + n][0]
                out[x + n] = layer.w_in[at:at + rows, :W]
                if n in "qkv":
                    out[f"{x}{n}.conv"] = layer.conv[:, c:c + rows].t()
                    c += rows
            if isinstance(spec.mixer, AttentionSpec):
                out[x + "sink"] = layer.sink
                if layer.mix is not None:
                    out[x + "vmix"] = layer.mix.reshape(())
            else:
                out.update({x + "A_log": layer.A_log, x + "dt_bias": layer.dt_bias,
                            x + "norm": layer.head_norm})
                for n, t in (("a2", layer.w_a2), ("g2", layer.w_g2)):
                    r, k = self._shapes[x + n]
                    out[x + n] = t[:r, :k]
            out[x + "o"] = layer.w_out[:W, :layer.out_dim]
            if layer.w_up is not None:
                out[p + "norm2"] = layer.norm2[:W]
                out[p + "mlp.up"] = layer.w_up[:layer.ff, :W]
                out[p + "mlp.down"] = layer.w_out[:W, layer.act_off:layer.act_off + layer.ff]
        return {n: t.detach().cpu().contiguous().clone() for n, t in out.items()}


def load_hybrid(state: Mapping[str, torch.Tensor], config: Mapping[str, Any], device="cuda",
                training: bool = False, dtype: Optional[torch.dtype] = None) -> HybridLM:
    if training:
        raise ProcessingError.unsupported(f"training a {config.get('architecture')} model",
                                          "the hybrid decoders are served only")
    cfg = config_from_json(config, {n: tuple(t.shape) for n, t in state.items()})
    return HybridLM(cfg, state, device, dtype)


def export_hybrid(lm: HybridLM):
    return {n: t.to(torch.bfloat16) for n, t in lm.state_dict().items()}, config_to_json(lm.cfg)
