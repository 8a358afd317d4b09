from __future__ import annotations

import torch

from .. import kernels
from .base import Part, TensorDecl, register_part


@register_part("reentry", "embedding_and_offset")
class EmbeddingAndOffset(Part):
    """What a pass over a repeated run of layers starts with: before pass t (0, 1, ...) the row t of a table of offsets
    [passes, H] is added to every token's stream, and before every pass but the first also the embedding's output as it
    was before the first layer.  The model asks for a copy of that output once a step (`remember`), and for the add where
    an entry of the run order opens a pass (`forward`); the add is left pending and runs in the next norm's pass over the
    stream.  params: hidden_size, passes, tensor (the table's name)."""
    capturable = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden, self.passes = int(spec.params["hidden_size"]), int(spec.params["passes"])
        self.tensor = str(spec.params.get("tensor", "offset"))
        self.offsets = None

    def tensors(self):
        return {self.tensor: TensorDecl((self.passes, self.hidden), use="vector")}

    def load(self, tensors):
        self.offsets = tensors[self.tensor].float().contiguous()

    def remember(self, residual):
        """A copy of the embedding's output (the stream is changed in place by the layers); None when no pass needs it."""
        return residual.clone() if self.passes > 1 else None

    def forward(self, residual, pending, first, t: int):
        from .block import PendingGated, settle
        if not (0 <= t < self.passes):
            raise ValueError(f"pass {t} of {self.passes}")
        if pending is not None:
            if isinstance(pending, PendingGated) and pending.rows_add is None and pending.vec_add is None:
                # the part before it has not joined the stream yet: both adds go into the same pass over the rows
                pending.rows_add, pending.vec_add = (first if t > 0 else None), self.offsets[t]
                return residual, pending
            settle(residual, pending)
        return residual, PendingGated(rows_add=first if t > 0 else None, vec_add=self.offsets[t])


@register_part("reentry", "embedding_projection")
class EmbeddingProjection(Part):
    """What a pass over a repeated run of layers starts with: before every pass t (0, 1, ..., the first too) the stream is
    replaced by  W [x; x0] + s_t,  x0 being the embedding's output as it was before the first layer, W [H, 2 H] one matrix
    for all passes and s_t the row t of a table [passes, H].  Once a step (`remember`) x0 is written, in the activations'
    dtype, into the right half of the product's operand; a pass writes the stream beside it and runs one product whose
    float32 result, the row s_t included as its bias, is the new stream.  params: hidden_size, passes, matrix (W's local
    name), tensor (the table's name)."""
    capturable = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden, self.passes = int(spec.params["hidden_size"]), int(spec.params["passes"])
        self.matrix, self.tensor = str(spec.params.get("matrix", "in")), str(spec.params.get("tensor", "offset"))
        self.weight = self.offsets = None

    def tensors(self):
        return {self.matrix: TensorDecl((self.hidden, 2 * self.hidden)), self.tensor: TensorDecl((self.passes, self.hidden), use="vector")}

    def load(self, tensors):
        self.weight = tensors[self.matrix].contiguous()
        self.offsets = tensors[self.tensor].float().contiguous()

    def remember(self, residual):
        pair = torch.empty((residual.shape[0], 2 * self.hidden), dtype=self.env.dtype, device=residual.device)
        kernels.copy_rows(residual, pair[:, self.hidden:])
        return pair

    def forward(self, residual, pending, first, t: int):
        from .block import settle
        if not (0 <= t < self.passes):
            raise ValueError(f"pass {t} of {self.passes}")
        if pending is not None:
            settle(residual, pending)
        kernels.copy_rows(residual, first[:, :self.hidden])
        return kernels.linear(first, self.weight, self.offsets[t], out_dtype=torch.float32), None
