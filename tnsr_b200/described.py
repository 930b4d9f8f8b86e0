"""What models described layer by layer have in common: a checked table of named tensors on the sessions of ``Gpt``
(``GptDecoder`` over ``tnsr_b200_decoder_create_stack``).

A configuration of such a model offers ``tensor_shapes()`` (names and shapes in the order of the library's parameter table),
``stack()`` (the description the library builds a session from), ``vocab_size``, ``embed_dim``, ``num_layers``,
``layer_norm_epsilon``, ``weight_dtype`` and ``max_sequence_length``.
"""
from __future__ import annotations

from typing import Dict, Iterable, List

import numpy as np

from .nn import CachedModel, MAX_EXACT_F32_INTEGER, Parameter, TnsrError

# Longest context unless the caller says otherwise: rotary positions have no table to run out of, but a session's
# positions stay exact f32 integers.
DEFAULT_CONTEXT = 1 << 20


class DescribedModel(CachedModel):
    def __init__(self, config, tensors: Dict[str, np.ndarray], unused: Iterable[str] = ()):
        """``unused``: names that a weight file may hold although the configuration has no use for them."""
        assert 0 < config.vocab_size <= MAX_EXACT_F32_INTEGER and config.embed_dim > 0 and config.layers
        assert 0 < config.max_sequence_length <= MAX_EXACT_F32_INTEGER
        assert config.weight_dtype in ("f32", "bf16")
        self._config = config
        shapes = config.tensor_shapes()
        missing, unexpected = sorted(set(shapes) - set(tensors)), sorted(set(tensors) - set(shapes) - set(unused))
        if missing or unexpected:
            raise TnsrError(f"parameter keys mismatch; missing: {missing}; unexpected: {unexpected}")
        self._parameters = {}
        for name, shape in shapes.items():
            if tuple(tensors[name].shape) != shape:
                raise TnsrError(f"{name}: expected shape {list(shape)}, got {list(tensors[name].shape)}")
            self._parameters[name] = Parameter(tensors[name], shape)

    def config(self):
        return self._config

    def parameters(self) -> List[Parameter]:
        return list(self._parameters.values())

    def named(self) -> Dict[str, Parameter]:
        return dict(self._parameters)

    def _generation_capacity(self, needed: int) -> int:
        return min(needed, self._config.max_sequence_length)
