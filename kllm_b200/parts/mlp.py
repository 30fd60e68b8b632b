"""Gated feed-forward (SwiGLU): down( act(x Wg^T) * (x Wu^T) ).

params: ``hidden``, ``intermediate``, ``activation`` ("silu"; "gelu_tanh": the tanh form of the gelu; "clamped" with
``limit`` L and ``alpha`` a: g sigmoid(a g) (u + 1) with g = min(x Wg^T, L) and u = clamp(x Wu^T, -L, L), no biases), optional
``tensors`` (gate, up, down -> full names), ``bias`` (True: all three projections have float32 biases,
``<weight name>.b``).  Tensors:
``<prefix>.{gate,up}_proj.weight`` [f, d] and ``<prefix>.down_proj.weight`` [d, f],
no bias by default (reference backend/model.cu:1112-1115, activation :477-483).  Gate and up
are stacked into one [2f, d] matrix at bind time so both are one product.

Optional ``forward_residual(x, norm, ctx) -> bool``: as for mixers, the part reads
the float32 residual stream, applies ``norm`` inside its first kernel and adds its
result into x, or returns False.  Here, for steps of a few tokens, the gate/up
product carries the norm as prologue and the activation as epilogue, the down
product adds into x (csrc/skinny_gemm.cu).  Large portions in bfloat16 run gate, up
and the activation as one tensor-core kernel (csrc/gemm_tcgen05.cu) where its tiles
fill the GPU; everything else uses the library product and the activation kernel.

``forward_add(x, h, ctx)``: x += ff(h) for a normed input h that another sublayer reads too (the ``parallel`` block).

Interface of a feed-forward part: ``forward(xn, ctx) -> [n, hidden]`` in float32 or
the model dtype.
"""
from __future__ import annotations

import torch

from .. import kernels
from .spec import BuildEnv, PartSpec, TensorSpec, register_part


class GatedMLP:
    def __init__(self, spec: PartSpec, env: BuildEnv):
        p = spec.params
        self.hidden = int(p["hidden"])
        self.inter = int(p["intermediate"])
        self.activation = p.get("activation", "silu")
        if self.activation not in ("silu", "gelu_tanh", "clamped"):
            raise ValueError(f"gated feed-forward: activation {self.activation!r} has no kernel (silu, gelu_tanh, clamped)")
        self.has_bias = bool(p.get("bias", False))
        self.limit, self.alpha = float(p.get("limit") or 0.0), float(p.get("alpha", 1.0))
        if self.activation == "clamped" and (self.has_bias or not self.limit > 0):
            raise ValueError("gated feed-forward: the clamped activation needs a positive limit and goes without biases")
        self.plain = self.activation == "silu" and not self.has_bias
        self.b_gate = self.b_up = self.b_down = None
        self.prefix = spec.prefix
        names = dict(p.get("tensors") or {})
        self.names = {k: names.get(k) or f"{self.prefix}.{k}_proj.weight" for k in ("gate", "up", "down")}
        self.dtype = env.dtype
        self.w_gate_up = None
        self.w_down = None
        self._after = []           # weights streamed right after this part (see set_prefetch_targets)

    def tensor_specs(self):
        out = [TensorSpec(self.names["gate"], (self.inter, self.hidden)),
               TensorSpec(self.names["up"], (self.inter, self.hidden)),
               TensorSpec(self.names["down"], (self.hidden, self.inter))]
        if self.has_bias:
            out += [TensorSpec(self.names[k] + ".b", (size,), store="float32")
                    for k, size in (("gate", self.inter), ("up", self.inter), ("down", self.hidden))]
        return out

    def bind(self, tensors):
        self.w_gate_up = torch.cat([tensors[self.names["gate"]], tensors[self.names["up"]]], dim=0).contiguous()
        self.w_down = tensors[self.names["down"]]
        if self.has_bias:
            self.b_gate, self.b_up, self.b_down = (tensors[self.names[k] + ".b"].contiguous() for k in ("gate", "up", "down"))

    def streamed_weights(self):
        """The matrices this part streams in a small step, in kernel order."""
        return [self.w_gate_up, self.w_down]

    def set_prefetch_targets(self, weights):
        """What the kernels after this part stream first (the next layer's mixer's
        ``streamed_weights``): in a small step this part's two kernels ask for them
        to be brought into L2 while they run."""
        self._after = list(weights)

    def _target(self, i):
        return self._after[i] if i < len(self._after) else None

    def _activation(self, xn):
        """silu(gate) * up as a matrix of the model dtype."""
        n = xn.shape[0]
        act = torch.empty((n, self.inter), dtype=self.dtype, device=xn.device)
        w_gate, w_up = self.w_gate_up[:self.inter], self.w_gate_up[self.inter:]
        if (kernels.skinny_fits(n, self.hidden, self.dtype) and xn.is_contiguous() and xn.data_ptr() % 16 == 0
                and w_gate.data_ptr() % 16 == 0 and w_up.data_ptr() % 16 == 0):
            # a step of a few rows: the weights streamed once, biases and activation in the product's epilogue
            return kernels.skinny_gemm(w_gate, weight_up=w_up, x=xn, epilogue="swiglu", prefetch=self._target(0),
                                       bias=self.b_gate, bias_up=self.b_up, activation=self.activation, limit=self.limit,
                                       alpha=self.alpha)
        epilogue = "clamped" if self.activation == "clamped" else "swiglu" if self.plain else None
        if (epilogue and self.dtype == torch.bfloat16 and kernels.gemm_pays(n, self.inter, epilogue)
                and kernels.gemm_fits(xn, w_gate, act, epilogue, w_up)):
            # large portions: both products and the activation in one tcgen05 kernel
            kernels.gemm(xn, w_gate, weight_up=w_up, epilogue=epilogue, out=act, limit=self.limit, alpha=self.alpha)
        else:
            gu = kernels.linear(xn, self.w_gate_up, out_dtype=torch.float32)
            if self.activation == "clamped":
                kernels.clamped_glu(act, gu[:, :self.inter], gu[:, self.inter:], self.limit, self.alpha)
            elif self.plain:
                kernels.silu_mul(act, gu[:, :self.inter], gu[:, self.inter:])
            else:
                kernels.biased_glu(act, gu[:, :self.inter], gu[:, self.inter:], self.b_gate, self.b_up, self.activation)
        return act

    def forward_add(self, x, h, ctx):
        kernels.linear_into(x, self._activation(h), self.w_down, bias=self.b_down, prefetch=self._target(1))

    def forward(self, xn, ctx):
        # gate and up stay float32 until the activation has been applied; the down
        # projection's float32 result goes into the residual stream unrounded
        n = xn.shape[0]
        if self.activation == "clamped":
            return kernels.linear(self._activation(xn), self.w_down, out_dtype=torch.float32, small_ok=True)
        if not self.plain:
            y = torch.zeros((n, self.hidden), dtype=torch.float32, device=xn.device)
            self.forward_add(y, xn, ctx)
            return y
        if (kernels.skinny_fits(n, self.hidden, self.dtype) and kernels.skinny_fits(n, self.inter, self.dtype)
                and xn.is_contiguous()):
            # a step of a few rows: both products stream their weights once, the activation in the first one's epilogue
            act = kernels.skinny_gemm(self.w_gate_up[:self.inter], weight_up=self.w_gate_up[self.inter:], x=xn,
                                      epilogue="swiglu", prefetch=self._target(0))
            return kernels.skinny_gemm(self.w_down, x=act, epilogue="f32", prefetch=self._target(1))
        act = self._activation(xn)
        return kernels.linear(act, self.w_down, out_dtype=torch.float32)

    def forward_residual(self, x, norm, ctx):
        n = x.shape[0]
        if not self.plain:
            self.forward_add(x, norm.forward(x, None), ctx)
            return True
        if not (getattr(norm, "fusable_rmsnorm", False) and kernels.skinny_fits(n, self.hidden, self.dtype)
                and kernels.skinny_fits(n, self.inter, self.dtype, sliced=True)):
            # larger steps: the down product adds into the residual stream
            kernels.linear_add(x, self._activation(norm.forward(x, None)), self.w_down)
            return True
        act = kernels.skinny_gemm(self.w_gate_up[:self.inter], weight_up=self.w_gate_up[self.inter:], x_f32=x,
                                  gain=norm.gain, eps=norm.eps, epilogue="swiglu", prefetch=self._target(0))
        kernels.skinny_gemm(self.w_down, x=act, epilogue="add", out=x, prefetch=self._target(1))
        return True


class PlainMLP:
    """Feed-forward without a gate: down(act(up x)).  params: ``hidden``, ``intermediate``,
    ``activation`` ("relu2": the square of relu; "gelu": with the error function; "gelu_tanh": its tanh form), optional ``tensors`` (up/down -> full
    names; default ``<prefix>.up`` and ``<prefix>.down``).  The up product's float32 result
    meets the activation unrounded; the result is float32 [n, hidden]."""

    def __init__(self, spec: PartSpec, env: BuildEnv):
        p = spec.params
        self.hidden = int(p["hidden"])
        self.inter = int(p["intermediate"])
        self.activation = p.get("activation", "relu2")
        if self.activation not in ("relu2", "gelu", "gelu_tanh"):
            raise ValueError(f"plain feed-forward: activation {self.activation!r} has no kernel (relu2, gelu, gelu_tanh)")
        names = dict(p.get("tensors") or {})
        self.up_name = names.get("up") or f"{spec.prefix}.up"
        self.down_name = names.get("down") or f"{spec.prefix}.down"
        self.dtype = env.dtype

    def tensor_specs(self):
        return [TensorSpec(self.up_name, (self.inter, self.hidden)), TensorSpec(self.down_name, (self.hidden, self.inter))]

    def bind(self, tensors):
        self.w_up, self.w_down = tensors[self.up_name], tensors[self.down_name]

    def forward(self, xn, ctx):
        act = kernels.unary(kernels.linear(xn, self.w_up, out_dtype=torch.float32, small_ok=True), self.activation,
                            self.dtype)
        return kernels.linear(act, self.w_down, out_dtype=torch.float32, small_ok=True)


register_part("feed_forward", "gated_mlp", GatedMLP)
register_part("feed_forward", "plain_mlp", PlainMLP)
