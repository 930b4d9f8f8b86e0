"""Bolonex: a decoder-only model of parallel blocks whose mixers are grouped-query attention behind short convolutions
or mamba2 layers, on the same sessions as ``Gpt`` (``GptDecoder`` over ``libtnsr_b200.so``).

The model is handed to the library as a list of layers (``tnsr_b200_decoder_create_stack``); sizes, constants, the order
of layers and tensor sharing all come from its config.json.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, Optional, Tuple

from . import _native
from .described import DEFAULT_CONTEXT, DescribedModel
from .nn import TnsrError


@dataclass(frozen=True)
class RotaryConfig:
    dims: int
    base: float
    factor: float = 0.0          # 0: no frequency scaling
    low: float = 0.0
    high: float = 0.0
    original: float = 0.0


@dataclass(frozen=True)
class LayerConfig:
    mixer: str                   # "attention" or "mamba2"
    heads: int
    vdim: int
    conv: int
    feed_forward: int = 0        # 0: no feed-forward
    weights_of: Optional[int] = None
    # attention
    kv_heads: int = 0
    dim: int = 0
    rotary: Optional[RotaryConfig] = None
    scale: float = 0.0
    softcap: float = 0.0         # 0: scores are not capped
    # mamba2
    state: int = 0
    groups: int = 0
    norm_groups: int = 0

    def shape(self):
        """Everything that two layers sharing tensors must have in common."""
        return (self.mixer, self.heads, self.vdim, self.conv, self.feed_forward, self.kv_heads, self.dim, self.state, self.groups)


def _rotary(entry) -> Optional[RotaryConfig]:
    if not entry:
        return None
    scaling = entry.get("scaling") or {}
    return RotaryConfig(int(entry["dims"]), float(entry["base"]), float(scaling.get("factor", 0.0)), float(scaling.get("low", 0.0)),
                        float(scaling.get("high", 0.0)), float(scaling.get("original", 0.0)))


def _layer(entry: dict, index: int) -> LayerConfig:
    mixer, kind = entry["mixer"], entry["type"]
    mlp = entry.get("mlp")
    if mlp and mlp.get("kind") != "dense":
        raise TnsrError(f"layer {index}: unknown feed-forward {mlp.get('kind')!r}")
    common = dict(mixer=kind, heads=int(mixer["heads"]), vdim=int(mixer["vdim"]), conv=int(mixer["conv"]),
                  feed_forward=int(mlp["ff"]) if mlp else 0,
                  weights_of=None if entry.get("weights_of") is None else int(entry["weights_of"]))
    if kind == "attention":
        return LayerConfig(**common, kv_heads=int(mixer["kv_heads"]), dim=int(mixer["dim"]), rotary=_rotary(mixer.get("rot")),
                           scale=float(mixer["scale"]), softcap=float(mixer.get("softcap") or 0.0))
    if kind == "mamba2":
        return LayerConfig(**common, state=int(mixer["state"]), groups=int(mixer["groups"]), norm_groups=int(mixer["norm_groups"]))
    raise TnsrError(f"layer {index}: unknown mixer {kind!r}")


@dataclass
class BolonexConfig:
    vocab_size: int
    embed_dim: int
    layers: Tuple[LayerConfig, ...]
    embedding_scale: float = 1.0
    layer_norm_epsilon: float = 1e-5      # of every norm
    weight_dtype: str = "bf16"
    max_sequence_length: int = DEFAULT_CONTEXT
    architecture: str = field(default="Bolonex", init=False)

    @classmethod
    def from_dict(cls, config: dict, weight_dtype: str = "bf16", max_sequence_length: int = DEFAULT_CONTEXT) -> "BolonexConfig":
        """From a parsed config.json."""
        try:
            return cls(vocab_size=int(config["vocab"]), embed_dim=int(config["width"]),
                       layers=tuple(_layer(entry, i) for i, entry in enumerate(config["layers"])),
                       embedding_scale=float(config["embedding"]["scale"]), layer_norm_epsilon=float(config["norm"]["eps"]),
                       weight_dtype=weight_dtype, max_sequence_length=max_sequence_length)
        except (KeyError, TypeError) as e:
            raise TnsrError(f"Bolonex configuration: missing or malformed entry {e}")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def owner(self, index: int) -> int:
        """The layer whose tensors layer ``index`` uses."""
        seen = set()
        while self.layers[index].weights_of is not None:
            if index in seen:
                raise TnsrError("weights_of forms a loop")
            seen.add(index)
            target = self.layers[index].weights_of
            if not 0 <= target < len(self.layers) or self.layers[target].shape() != self.layers[index].shape():
                raise TnsrError(f"layer {index}: weights_of {target} is not a layer of the same sizes")
            index = target
        return index

    def stack(self) -> _native.StackDesc:
        """The description the library builds its session from."""
        array = (_native.LayerDesc * len(self.layers))()
        for out, l in zip(array, self.layers):
            out.mixer = _native.MIXER[l.mixer]
            out.weights_of = -1 if l.weights_of is None else l.weights_of
            out.heads, out.vdim, out.conv_taps, out.feed_forward = l.heads, l.vdim, l.conv, l.feed_forward
            out.kv_heads, out.dim = l.kv_heads, l.dim
            if l.rotary is not None:
                r = l.rotary
                out.rotary_dims, out.rotary_base = r.dims, r.base
                out.rotary_factor, out.rotary_low, out.rotary_high, out.rotary_original = r.factor, r.low, r.high, r.original
            out.score_scale, out.score_softcap = l.scale, l.softcap
            out.state, out.groups, out.norm_groups = l.state, l.groups, l.norm_groups
        return _native.StackDesc(self.embedding_scale, 1.0, array, len(self.layers))

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Tensor names and shapes in the order of the library's parameter table."""
        d = self.embed_dim
        shapes: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab_size, d), "head": (self.vocab_size, d), "final.norm": (d,)}
        for i, l in enumerate(self.layers):
            if self.owner(i) != i:
                continue
            p = f"l{i}."
            shapes[p + "norm1"] = (d,)
            m = p + "mix."
            if l.mixer == "attention":
                sizes = {"q": l.heads * l.dim, "k": l.kv_heads * l.dim, "v": l.kv_heads * l.vdim}
                for name, n in sizes.items():
                    shapes[m + name], shapes[m + name + ".b"] = (n, d), (n,)
                shapes[m + "q.norm"], shapes[m + "k.norm"] = (l.dim,), (l.dim,)
                for name, n in sizes.items():
                    shapes[m + name + ".conv"] = (n, l.conv)
                shapes[m + "g"] = (l.heads, d)
            else:
                inner, gn = l.heads * l.vdim, l.groups * l.state
                shapes[m + "in"] = (2 * inner + 2 * gn + l.heads, d)
                shapes[m + "conv"], shapes[m + "conv.b"] = (inner + 2 * gn, l.conv), (inner + 2 * gn,)
                shapes[m + "dt_bias"], shapes[m + "A_log"], shapes[m + "D"] = (l.heads,), (l.heads,), (l.heads,)
                shapes[m + "norm"] = (inner,)
            shapes[m + "o"] = (d, l.heads * l.vdim)
            if l.feed_forward:
                shapes[p + "mlp.up"], shapes[p + "mlp.down"] = (l.feed_forward, d), (d, l.feed_forward)
        return shapes


class Bolonex(DescribedModel):
    def __init__(self, config: BolonexConfig, tensors):
        super().__init__(config, tensors)
