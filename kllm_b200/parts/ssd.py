"""A state-space recurrence with one decay per head and token behind a short convolution (Mamba-2): a recurrent mixer on
the kernels of csrc/ssd.cu.

With h the mixer's input, H heads of dv values, G groups of N state channels (head i uses group i // (H / G)):

    [z | x | B | C | dt] = W_in h                       [H dv | H dv | G N | G N | H]
    x, B, C <- silu(causal convolution of each channel over its last ``taps`` inputs + bias)
    dt      <- softplus(dt + dt_bias)
    S_t     = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T        y_t = S_t^T C_t + D x_t        S [N, dv] per head
    out     = W_o (partnorm(y * silu(z)) * gain)

partnorm divides each of ``norm_parts`` equal pieces of the row by its own root mean square.

params: ``hidden``, ``heads``, ``head_dim`` (dv), ``state`` (N), ``groups``, ``taps``, ``norm_parts``, ``eps``, optional ``tensors``
(in, conv, conv_bias, dt_bias, a_log, d, norm, o -> full names; default ``<prefix>.{in,conv,conv.b,dt_bias,A_log,D,norm,o}``).

State (``StateNeed``), float32, zero when a request opens: S as [heads][N][dv], and under the name "conv" the convolution's
inputs of the last ``taps`` positions, position p in row p mod taps.  The projections are one product whose float32
result feeds the kernels; convolution, decays, state, sums, gate and norm are float32 in both dtypes; in bfloat16 portions round
x, B and C behind silu where their products run on the tensor cores.  The mixer has the split form (``gla.SplitMixer``).
"""
from __future__ import annotations

import torch

from .. import kernels
from .gla import SplitMixer, stack_rows
from .spec import BuildEnv, PartSpec, StateNeed, TensorSpec, register_part


class StateSpaceMixer(SplitMixer):
    def __init__(self, spec: PartSpec, env: BuildEnv):
        p = spec.params
        self.hidden, self.heads, self.dv = int(p["hidden"]), int(p["heads"]), int(p["head_dim"])
        self.N, self.groups, self.taps = int(p["state"]), int(p["groups"]), int(p["taps"])
        self.parts, self.eps = int(p["norm_parts"]), float(p["eps"])
        self.inner = self.heads * self.dv
        if self.heads % self.groups or self.inner % self.parts:
            raise ValueError(f"ssd: {self.heads} heads in {self.groups} groups, {self.inner} channels in {self.parts} parts of the norm")
        if not (1 <= self.taps <= 64):
            raise ValueError(f"ssd: a convolution of {self.taps} taps (the kernels hold up to 64)")
        self.channels = self.inner + 2 * self.groups * self.N
        self.out_dim = self.inner
        self.dtype = env.dtype
        given = dict(p.get("tensors") or {})
        names = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "a_log": "A_log", "d": "D", "norm": "norm",
                 "o": "o"}
        self.n = {k: given.get(k) or f"{spec.prefix}.{v}" for k, v in names.items()}

    def tensor_specs(self):
        n, f32 = self.n, "float32"
        return [TensorSpec(n["in"], (self.inner + self.channels + self.heads, self.hidden)),
                TensorSpec(n["conv"], (self.channels, self.taps), store=f32, init="uniform:-0.5:0.5"),
                TensorSpec(n["conv_bias"], (self.channels,), store=f32, init="zeros"),
                TensorSpec(n["dt_bias"], (self.heads,), store=f32, init="uniform:-6:-2"),
                TensorSpec(n["a_log"], (self.heads,), store=f32, init="uniform:0:2.7"),
                TensorSpec(n["d"], (self.heads,), store=f32, init="gain"),
                TensorSpec(n["norm"], (self.inner,), store=f32, init="gain"),
                TensorSpec(n["o"], (self.hidden, self.inner))]

    def bind(self, tensors):
        n = self.n
        self.w_in = stack_rows([tensors[n["in"]]])
        self.conv, self.conv_bias, self.dt_bias, self.a_log, self.d, self.gain = (
            tensors[n[k]].contiguous() for k in ("conv", "conv_bias", "dt_bias", "a_log", "d", "norm"))
        self.w_out = tensors[n["o"]]

    def cache_need(self):
        row = -(-self.channels // 4) * 4                    # whole 16-byte units
        return [StateNeed((self.heads * self.N * self.dv,), "float32"), StateNeed((self.taps * row,), "float32", name="conv")]

    def core(self, proj, ctx, cache, y):
        g = kernels.ssd(proj, self.conv, self.conv_bias, self.dt_bias, self.a_log, self.d, cache.state, cache.states["conv"], ctx,
                        self.heads, self.groups, self.N, self.dv, early=True, dtype=self.dtype)
        kernels.part_norm(y, g, self.gain, self.parts, self.eps)


register_part("mixer", "ssd", StateSpaceMixer)
