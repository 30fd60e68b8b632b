"""What a schedule entry may do to the residual stream before its layer runs.

``embedding_mix``: the stream is mixed with the embedding's output x0 and a vector of the pass is added,

    x <- W_in [x; x0] + step[t]

params: ``hidden``, ``passes`` (rows of the table), ``in`` ([hidden, 2 hidden], x first) and ``step`` ([passes, hidden],
float32): full tensor names.  The product takes x and x0 in the model dtype and its float32 result is added to the step's vector
in the stream.

Interface of a part of the stream_entry family: ``tensor_specs()``, ``bind(tensors)``, ``begin(x, at_once) -> held`` (called
with the embedding's output before the first layer; ``at_once``: the first ``apply`` follows with the same x), and
``apply(x, held, t)``, which changes x in place.  A schedule entry names the part and t (``LayerCall.entry``).
"""
from __future__ import annotations

import torch

from .. import kernels
from .spec import BuildEnv, PartSpec, TensorSpec, register_part


class EmbeddingMix:
    def __init__(self, spec: PartSpec, env: BuildEnv):
        p = spec.params
        self.hidden, self.passes = int(p["hidden"]), int(p["passes"])
        self.in_name, self.step_name = p["in"], p["step"]
        self.dtype = env.dtype

    def tensor_specs(self):
        return [TensorSpec(self.in_name, (self.hidden, 2 * self.hidden)),
                TensorSpec(self.step_name, (self.passes, self.hidden), store="float32")]

    def bind(self, tensors):
        self.w_in, self.step = tensors[self.in_name], tensors[self.step_name].contiguous()

    def begin(self, x, at_once):
        cat = torch.empty((x.shape[0], 2 * self.hidden), dtype=self.dtype, device=x.device)
        if not at_once:
            kernels.unary(x, "copy", self.dtype, out=cat[:, self.hidden:])
        return {"cat": cat, "fresh": at_once}

    def apply(self, x, held, t):
        kernels.stream_entry(held["cat"], x, self.step[t], held["fresh"])
        held["fresh"] = False
        kernels.linear_into(x, held["cat"], self.w_in)


register_part("stream_entry", "embedding_mix", EmbeddingMix)
