"""Ganupel: a decoder-only model of sequential pre-norm blocks with layer scales.  A block's mixer is either windowed
attention with sigmoid weights beside HGRN2 linear attention, or a real-gated linear recurrent unit (RG-LRU); its
feed-forward a dense one with PolyNorm, a mixture of relu^2 experts with identity experts, or none.

Served by the sessions of ``Gpt`` through ``tnsr_b200_decoder_create_stack``; sizes, constants and the order of layers all
come from its config.json.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple, Union

from . import _native
from .described import DEFAULT_CONTEXT, DescribedModel
from .nn import TnsrError


@dataclass(frozen=True)
class WindowedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int                  # 0: every earlier position is visible
    rotary_dims: int = 0
    rotary_base: float = 1.0


@dataclass(frozen=True)
class Hgrn2:
    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class ParallelMixer:
    left: WindowedAttention
    right: Hgrn2
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class RgLru:
    width: int
    blocks: int
    conv: int


@dataclass(frozen=True)
class Dense:
    feed_forward: int


@dataclass(frozen=True)
class Experts:
    feed_forward: int            # of one expert
    experts: int
    identity: int
    top: int
    scale: float


@dataclass(frozen=True)
class LayerConfig:
    mixer: Union[ParallelMixer, RgLru]
    mlp: Union[Dense, Experts, None] = None


def _mixer(kind: str, m: dict, index: int):
    if kind == "parallel":
        left, right, rot, mask = m["left"], m["right"], m["left"].get("rot") or {}, m["left"].get("mask") or {}
        return ParallelMixer(
            WindowedAttention(int(left["heads"]), int(left["kv_heads"]), int(left["dim"]), int(left["vdim"]), float(left["scale"]),
                              int(mask.get("size", 0)), int(rot.get("dims", 0)), float(rot.get("base", 1.0))),
            Hgrn2(int(right["heads"]), int(right["dim"]), int(right["vdim"])), float(m["left_scale"]), float(m["right_scale"]))
    if kind == "rglru":
        return RgLru(int(m["width"]), int(m["blocks"]), int(m["conv"]))
    raise TnsrError(f"layer {index}: unknown mixer {kind!r}")


def _mlp(m: Optional[dict], index: int):
    if not m:
        return None
    if m["kind"] == "dense":
        return Dense(int(m["ff"]))
    if m["kind"] == "moe":
        router = m["router"]
        return Experts(int(m["expert"]["ff"]), int(router["experts"]), int(router.get("identity") or 0), int(router["top"]), float(router["scale"]))
    raise TnsrError(f"layer {index}: unknown feed-forward {m['kind']!r}")


@dataclass
class GanupelConfig:
    vocab_size: int
    embed_dim: int
    layers: Tuple[LayerConfig, ...]
    layer_norm_epsilon: float = 1e-5      # of every norm
    weight_dtype: str = "bf16"
    max_sequence_length: int = DEFAULT_CONTEXT
    architecture: str = field(default="Ganupel", init=False)

    @classmethod
    def from_dict(cls, config: dict, weight_dtype: str = "bf16", max_sequence_length: int = DEFAULT_CONTEXT) -> "GanupelConfig":
        """From a parsed config.json."""
        try:
            return cls(vocab_size=int(config["vocab"]), embed_dim=int(config["width"]),
                       layers=tuple(LayerConfig(_mixer(entry["type"], entry["mixer"], i), _mlp(entry.get("mlp"), i)) for i, entry in enumerate(config["layers"])),
                       layer_norm_epsilon=float(config["norm"]["eps"]), weight_dtype=weight_dtype, max_sequence_length=max_sequence_length)
        except (KeyError, TypeError, AttributeError) as e:
            raise TnsrError(f"Ganupel configuration: missing or malformed entry {e}")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def stack(self) -> _native.StackDesc:
        """The description the library builds its session from."""
        array = (_native.LayerDesc * len(self.layers))()
        for out, layer in zip(array, self.layers):
            out.weights_of, out.block_form = -1, _native.BLOCK["sequential"]
            m, f = layer.mixer, layer.mlp
            if isinstance(m, ParallelMixer):
                a, r = m.left, m.right
                out.mixer = _native.MIXER["attention+hgrn2"]
                out.heads, out.kv_heads, out.dim, out.vdim = a.heads, a.kv_heads, a.dim, a.vdim
                out.rotary_dims, out.rotary_base, out.rotary_layout = a.rotary_dims, a.rotary_base, _native.ROTARY["halves"]
                out.score_scale, out.score_kind, out.window = a.scale, _native.SCORE["sigmoid"], a.window
                out.rec_heads, out.rec_dim, out.rec_vdim = r.heads, r.dim, r.vdim
                out.attention_gain, out.recurrent_gain = m.left_scale, m.right_scale
            else:
                out.mixer = _native.MIXER["rglru"]
                out.width, out.blocks, out.conv_taps = m.width, m.blocks, m.conv
            if f is not None:
                out.feed_forward = f.feed_forward
                out.feed_forward_kind = _native.FEED_FORWARD["experts" if isinstance(f, Experts) else "polynorm"]
            if isinstance(f, Experts):
                out.experts, out.identity_experts, out.top, out.router_scale = f.experts, f.identity, f.top, f.scale
        return _native.StackDesc(1.0, 1.0, array, len(self.layers))

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Tensor names and shapes in the order of the library's parameter table."""
        d = self.embed_dim
        shapes: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab_size, d), "head": (self.vocab_size, d), "final.norm": (d,)}
        for i, layer in enumerate(self.layers):
            p, mix = f"l{i}.", f"l{i}.mix."
            m, f = layer.mixer, layer.mlp
            shapes[p + "norm1"] = (d,)
            if isinstance(m, ParallelMixer):
                a, r = m.left, m.right
                shapes.update({mix + "left.q": (a.heads * a.dim, d), mix + "left.k": (a.kv_heads * a.dim, d), mix + "left.v": (a.kv_heads * a.vdim, d),
                               mix + "left.pb": (a.heads,), mix + "left.o": (d, a.heads * a.vdim)})
                k = r.heads * r.dim
                shapes.update({mix + "right.q": (k, d), mix + "right.f": (k, d), mix + "right.f.b": (k,), mix + "right.lower": (k,),
                               mix + "right.v": (r.heads * r.vdim, d), mix + "right.norm": (r.vdim,), mix + "right.o": (d, r.heads * r.vdim)})
            else:
                n = m.width // max(1, m.blocks)
                shapes.update({mix + "y": (m.width, d), mix + "y.b": (m.width,), mix + "x": (m.width, d), mix + "x.b": (m.width,),
                               mix + "conv": (m.width, m.conv), mix + "conv.b": (m.width,), mix + "ra": (m.blocks, n, n), mix + "ra.b": (m.blocks, n),
                               mix + "ri": (m.blocks, n, n), mix + "ri.b": (m.blocks, n), mix + "lam": (m.width,), mix + "o": (d, m.width)})
            shapes[p + "ls1"] = (d,)
            if f is None:
                continue
            shapes[p + "norm2"] = (d,)
            if isinstance(f, Experts):
                for e in range(f.experts):
                    shapes[p + f"mlp.e{e}.up"], shapes[p + f"mlp.e{e}.down"] = (f.feed_forward, d), (d, f.feed_forward)
                total = f.experts + f.identity
                shapes[p + "mlp.router"], shapes[p + "mlp.correction"] = (total, d), (total,)
            else:
                shapes[p + "mlp.up"], shapes[p + "mlp.down"], shapes[p + "mlp.act"] = (f.feed_forward, d), (d, f.feed_forward), (4,)
            shapes[p + "ls2"] = (d,)
        return shapes

    def unused_tensors(self) -> List[str]:
        """Norm and scale of a feed-forward that a layer does not have."""
        return [f"l{i}.{name}" for i, layer in enumerate(self.layers) if layer.mlp is None for name in ("norm2", "ls2")]


class Ganupel(DescribedModel):
    def __init__(self, config: GanupelConfig, tensors):
        super().__init__(config, tensors, config.unused_tensors())
