"""How a sublayer reads from, and writes to, a residual of several parallel streams.

A residual of S streams x_1 .. x_S is one [T, S, H] buffer.  A sublayer reads sum_s in[s] x_s; its result y is written as
x_t <- sum_s mix[s, t] x_s + mult out[t] y, all streams at once from the old ones (``mix`` is indexed [from, to]).  Both run in the
kernel of the norm behind the sublayer (``kernels.streams_norm``); this part holds the weights, in float, ``mult`` folded into ``out``.

Parameters: ``streams``, ``mult`` (a constant factor on what is added), ``learned`` (False: no tensors, every stream is read with 1,
kept as it is and written with 1: with one stream the plain residual sum times ``mult``) and the tensor-name pieces ``in``, ``out``, ``mix``.
"""
from __future__ import annotations

import torch

from ..weights.tensors import TensorSpec
from .base import Runtime, to_device


class HyperConnection:
    graph_safe = True

    def __init__(self, params, prefix: str, runtime: Runtime) -> None:
        self.prefix, self.runtime, self.params = prefix, runtime, params
        self.streams = int(params["streams"])
        self.mult = float(params.get("mult", 1.0))
        self.learned = bool(params.get("learned", True))
        self.read = self.mix = self.out = None

    @staticmethod
    def _names(params, prefix: str) -> tuple[str, str, str]:
        return tuple(f"{prefix}.{params.get(key, key)}" for key in ("in", "mix", "out"))

    @classmethod
    def expected_tensors(cls, params, prefix: str) -> dict[str, TensorSpec]:
        if not params.get("learned", True):
            return {}
        count = int(params["streams"])
        read, mix, out = cls._names(params, prefix)
        return {read: TensorSpec((count,), role="vector", init_std=0.3, init_mean=1.0 / count),
                mix: TensorSpec((count, count), role="vector", init_std=0.3, init_mean=1.0 / count),
                out: TensorSpec((count,), role="vector", init_std=0.3, init_mean=1.0)}

    def load(self, source) -> None:
        device = self.runtime.device
        if self.learned:
            read, mix, out = (to_device(source(name), torch.float32, device) for name in self._names(self.params, self.prefix))
        else:
            read, mix, out = torch.ones(self.streams), torch.eye(self.streams), torch.ones(self.streams)
            read, mix, out = (to_device(tensor, torch.float32, device) for tensor in (read, mix, out))
        self.read, self.mix, self.out = read, mix, out * self.mult
