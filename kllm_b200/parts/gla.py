"""Linear attention whose state decays: two recurrent mixers on one kernel (csrc/gla.cu).

Per head, with dk key channels and dv value channels, a state S [dk, dv] that starts at zero and h the mixer's input:

    S_t = diag(alpha_t) S_(t-1) + k_t v_t^T            o_t = S_t^T q_t
    y   = W_o (o / rms(o over the head) * gain * silu(W_g h))

``gated_linear_attention`` (``GatedLinearAttention``): q = dk^(-1/2) W_q h, k = W_k h, v = W_v h and a decay per key
channel, alpha = sigmoid(W_a2 W_a1 h + b)^(1 / tau); the heads share one gain [dv].  params: ``hidden``, ``heads``,
``head_dim``, ``v_head_dim``, ``tau``, ``eps``, ``decay_rank`` (rows of W_a1 for random weights; a file's own rank is taken from
its tensor), optional ``tensors`` (q, k, v, g, o, norm, a1, a2, a2_bias -> full names; default ``<prefix>.<name>``,
``<prefix>.a2.b``).

``retention`` (``Retention``): a fixed decay per head, alpha = decay_h; the first ``rotary_dim`` values of every query and
key head are rotated (pair (i, i + rotary_dim / 2), angle position * theta^(-2i / rotary_dim) formed in double precision
on the device), k is multiplied by dk^(-1/2); no gain.  params: ``hidden``, ``heads``, ``head_dim``, ``v_head_dim``,
``decay`` (a list), ``eps``, ``rotary_dim``, ``theta``, optional ``scaling`` (as in ``rotary.rotary_frequencies``) and
``tensors`` (q, k, v, g, o).

Both: ``out_factor`` (default 1) multiplies y's rows before W_o.

State (``StateNeed``): per request one float32 vector [heads][dk][dv], zero when the request opens.  The projections
are one stacked product whose float32 result feeds the kernel; decay, state, sums, norm and gate are float32 in both dtypes.

Split form of a mixer, which these and the paged attention offer: ``w_in`` (the stacked projections, rows padded to a
multiple of 8), ``w_out``, ``out_dim`` and ``core(proj, ctx, cache, y)``, which takes the float32 result of the stacked
product (dense rows at any stride) and fills y [n, out_dim] (model dtype, dense rows at any stride).  A mixer in this form may
run beside another one on one stacked product (``side_by_side``).
"""
from __future__ import annotations

import torch

from .. import kernels
from .rotary import rotary_frequencies
from .spec import BuildEnv, PartSpec, StateNeed, TensorSpec, register_part


def stack_rows(tensors):
    """The matrices one under the other, with rows of zeros up to a multiple of 8 (every column of the product's
    result then starts on a 16-byte boundary wherever the matrices' own sizes allow)."""
    rows = sum(t.shape[0] for t in tensors)
    if rows % 8:
        tensors = list(tensors) + [tensors[0].new_zeros((8 - rows % 8, tensors[0].shape[1]))]
    return torch.cat(list(tensors), dim=0).contiguous()


class SplitMixer:
    """What the split form gives: both routes of a mixer from ``w_in``, ``core`` and ``w_out``."""

    def _rows(self, xn, ctx, cache):
        proj = kernels.linear(xn, self.w_in, out_dtype=torch.float32, small_ok=True)
        y = torch.empty((xn.shape[0], self.out_dim), dtype=self.dtype, device=xn.device)
        self.core(proj, ctx, cache, y)
        return y

    def forward(self, xn, ctx, cache):
        return kernels.linear(self._rows(xn, ctx, cache), self.w_out, out_dtype=torch.float32, small_ok=True)

    def forward_add(self, x, h, ctx, cache):
        """x += mixer(h), x the float32 residual stream."""
        kernels.linear_into(x, self._rows(h, ctx, cache), self.w_out)


class _DecayedAttention(SplitMixer):
    def __init__(self, spec: PartSpec, env: BuildEnv, names):
        p = spec.params
        self.hidden, self.heads = int(p["hidden"]), int(p["heads"])
        self.dk, self.dv = int(p["head_dim"]), int(p["v_head_dim"])
        if not (0 < self.dk <= 256):
            raise ValueError(f"{spec.kind}: a head of {self.dk} key channels (the recurrence kernel holds up to 256)")
        self.eps = float(p["eps"])
        self.factor = float(p.get("out_factor", 1.0))
        self.A, self.B = self.heads * self.dk, self.heads * self.dv
        self.out_dim = self.B
        self.dtype, self.device = env.dtype, env.device
        given = dict(p.get("tensors") or {})
        self.n = {k: given.get(k) or f"{spec.prefix}.{v}" for k, v in names.items()}

    def tensor_specs(self):
        n, d = self.n, self.hidden
        return [TensorSpec(n["q"], (self.A, d)), TensorSpec(n["k"], (self.A, d)), TensorSpec(n["v"], (self.B, d)),
                TensorSpec(n["g"], (self.B, d)), TensorSpec(n["o"], (d, self.B))]

    def cache_need(self):
        return StateNeed((self.heads * self.dk * self.dv,), "float32")

    def _columns(self, proj):
        A, B = self.A, self.B
        return proj[:, :A], proj[:, A:2 * A], proj[:, 2 * A:2 * A + B], proj[:, 2 * A + B:2 * (A + B)]


class GatedLinearAttention(_DecayedAttention):
    def __init__(self, spec: PartSpec, env: BuildEnv):
        super().__init__(spec, env, {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm", "a1": "a1",
                                     "a2": "a2", "a2_bias": "a2.b"})
        self.tau = float(spec.params["tau"])
        if not self.tau > 0:
            raise ValueError(f"gated linear attention: tau {self.tau} must be positive")
        self.rank = int(spec.params.get("decay_rank") or 16)

    def tensor_specs(self):
        n = self.n
        return super().tensor_specs() + [
            TensorSpec(n["norm"], (self.dv,), store="float32", init="gain"),
            TensorSpec(n["a1"], (self.rank, self.hidden), free=(0,)), TensorSpec(n["a2"], (self.A, self.rank), free=(1,)),
            TensorSpec(n["a2_bias"], (self.A,), store="float32", init="uniform:2:6")]

    def bind(self, tensors):
        n = self.n
        self.w2 = tensors[n["a2"]].contiguous()
        if tensors[n["a1"]].shape[0] != self.w2.shape[1]:
            raise ValueError(f"gated linear attention: the decay's two matrices disagree on its rank "
                             f"({tuple(tensors[n['a1']].shape)}, {tuple(self.w2.shape)})")
        self.w2_bias = tensors[n["a2_bias"]].contiguous()
        self.w_in = stack_rows([tensors[n[s]] for s in ("q", "k", "v", "g", "a1")])
        self.gain = (tensors[n["norm"]] * self.factor).repeat(self.heads).contiguous()
        self.w_out = tensors[n["o"]]

    def core(self, proj, ctx, cache, y):
        q, k, v, g = self._columns(proj)
        off = 2 * (self.A + self.B)
        kernels.gla(y, q, k, v, g, cache.state, ctx, self.heads, self.dk, self.dv, self.gain, self.eps,
                    low=proj[:, off:off + self.w2.shape[1]], w2=self.w2, w2_bias=self.w2_bias, tau=self.tau,
                    q_scale=self.dk ** -0.5, early=True)


class Retention(_DecayedAttention):
    def __init__(self, spec: PartSpec, env: BuildEnv):
        super().__init__(spec, env, {k: k for k in "qkvgo"})
        p = spec.params
        decay = [float(v) for v in p["decay"]]
        if len(decay) != self.heads or not all(0.0 < v <= 1.0 for v in decay):
            raise ValueError(f"retention: {len(decay)} decays for {self.heads} heads, each in (0, 1]")
        self.decay = torch.tensor(decay, dtype=torch.float32, device=env.device)
        rot = int(p.get("rotary_dim") or 0)
        if rot % 2 or rot > self.dk:
            raise ValueError(f"rotary_dim {rot} must be even and within head_dim {self.dk}")
        self.freq, self.amplitude = None, 1.0
        if rot:
            freq, self.amplitude = rotary_frequencies(rot, float(p["theta"]), p.get("scaling"))
            self.freq = freq.to(env.device)

    def bind(self, tensors):
        n = self.n
        self.w_in = stack_rows([tensors[n[s]] for s in "qkvg"])
        self.gain = torch.full((self.B,), self.factor, dtype=torch.float32, device=self.device)
        self.w_out = tensors[n["o"]]

    def core(self, proj, ctx, cache, y):
        q, k, v, g = self._columns(proj)
        kernels.gla(y, q, k, v, g, cache.state, ctx, self.heads, self.dk, self.dv, self.gain, self.eps, decay=self.decay,
                    freq=self.freq, amplitude=self.amplitude, k_scale=self.dk ** -0.5, early=True)


register_part("mixer", "gated_linear_attention", GatedLinearAttention)
register_part("mixer", "retention", Retention)
