"""Maps of the residual stream between layers.

``linear_of_concat``: x <- W [x; x0] with x0 the embedding's output, before the first layer of a pass of a looped range.  The
stream's rows (with what is pending on it) and x0 go side by side into the activation type, the stream is set to zero, and the
product with W [H, 2 H] is left pending like any sublayer's: the next norm adds its float sums, or, for few tokens, launches it
with the addition and its own preparation in the product's epilogue.

Parameters: ``hidden_size``, ``name`` (the matrix's tensor), ``init_std``.
"""
from __future__ import annotations

from ..ops import kernels
from ..weights.tensors import TensorSpec
from .base import DeferredProduct, ResidualStream, Runtime, register_stream_map
from .linear import Linear


@register_stream_map("linear_of_concat")
class LinearOfConcat:
    graph_safe = True

    def __init__(self, params, runtime: Runtime) -> None:
        self.hidden = int(params["hidden_size"])
        self.name = str(params["name"])
        self.runtime = runtime
        self.linear = Linear("stream_map.concat", self.hidden, 2 * self.hidden, runtime, float_out=True, role="mlp_out")
        runtime.workspace.declare("stream_map.rows", runtime.max_step_tokens * 2 * self.hidden, runtime.dtype)

    @classmethod
    def expected_tensors(cls, params) -> dict[str, TensorSpec]:
        hidden = int(params["hidden_size"])
        return {str(params["name"]): TensorSpec((hidden, 2 * hidden), init_std=float(params.get("init_std", 0.02)))}

    def load(self, source) -> None:
        self.linear.set_weight(source(self.name))

    def apply(self, stream: ResidualStream) -> None:
        if stream.more or stream.post is not None:
            raise RuntimeError(f"{self.name}: this map folds one plain pending addition")
        tokens = stream.residual.shape[0]
        rows = self.runtime.workspace.view("stream_map.rows", tokens, 2 * self.hidden)
        kernels.stream_concat(stream.residual, stream.pending, stream.start, rows)
        stream.pending = None
        stream.add(DeferredProduct(self.linear, rows) if self.linear.fusable(tokens) else self.linear(rows))
