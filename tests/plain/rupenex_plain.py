"""Plain, slow Rupenex forward pass in numpy float64: the yardstick of its tests.

Whole sequences, no cache, no paging, no batches; one function per mechanism.
Nothing here is imported by the product package and nothing of the product
package is imported here.  Weights arrive as a dict of tensor name -> numpy
array and are widened to float64; ``cfg`` is the dict of a config.json.

Notation: T tokens, d the model width, H heads, G key/value heads (attention) or groups (recurrence), dk the
per-head query/key size, dv the per-head value size, N the state size.
"""
from __future__ import annotations

import math

import numpy as np


def f64(a):
    return np.asarray(a, dtype=np.float64)


def sigmoid(z):
    z = f64(z)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, f64(z))


def unit_rms(x, eps):
    x = f64(x)
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def layer_norm(x, w, eps):
    """(x - mean) / sqrt(variance + eps) * w, no bias."""
    x = f64(x)
    c = x - x.mean(axis=-1, keepdims=True)
    return c / np.sqrt((c * c).mean(axis=-1, keepdims=True) + eps) * f64(w)


# ---- attention --------------------------------------------------------------------------

def frequencies(rot):
    """Angles per position [dims / 2] of a rotation {dims, base, scaling {factor} or none}."""
    f = float(rot["base"]) ** (-2.0 * np.arange(rot["dims"] // 2, dtype=np.float64) / rot["dims"])
    return f / float(rot["scaling"]["factor"]) if rot.get("scaling") else f


def rotate(x, positions, rot):
    """x [T, heads, size]: the pairs (i, i + dims / 2) of the first rot.dims values of every head are turned."""
    x = f64(x).copy()
    if not rot:
        return x
    half = rot["dims"] // 2
    a = f64(positions)[:, None, None] * frequencies(rot)
    u, v = x[..., :half].copy(), x[..., half:2 * half].copy()
    x[..., :half] = u * np.cos(a) - v * np.sin(a)
    x[..., half:2 * half] = v * np.cos(a) + u * np.sin(a)
    return x


def visible(positions, mask):
    """[T, T]: whether query i sees key j: no later key, and one of the last mask.size (its own included) or one of
    the first mask.keep_first of the sequence."""
    i, j = np.asarray(positions)[:, None], np.asarray(positions)[None, :]
    see = j <= i
    if mask:
        see &= (i - j < mask["size"]) | (j < (mask.get("keep_first") or 0))
    return see


def sink_attention(q, k, v, scale, see, sinks):
    """q [T, H, dk] over k [S, G, dk], v [S, G, dv]: softmax over the keys that see [T, S] names, with one more term
    exp(sinks[h]) in head h's denominator (sinks None: without)."""
    q, k, v = f64(q), f64(k), f64(v)
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for hd in range(H):
        s = np.where(see, q[:, hd] @ k[:, hd // per].T * scale, -np.inf)
        top = s.max(axis=1, keepdims=True)
        if sinks is not None:
            top = np.maximum(top, float(sinks[hd]))
        e = np.exp(s - top)
        den = e.sum(axis=1, keepdims=True)
        if sinks is not None:
            den = den + np.exp(float(sinks[hd]) - top)
        out[:, hd] = (e / den) @ v[:, hd // per]
    return out


def attention_mixer(h, w, p, m, eps, positions):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ f64(w[p + ".q"]).T).reshape(T, H, dk), eps) * f64(w[p + ".q.norm"])
    k = unit_rms((h @ f64(w[p + ".k"]).T).reshape(T, G, dk), eps) * f64(w[p + ".k.norm"])
    v = (h @ f64(w[p + ".v"]).T).reshape(T, G, dv)
    q, k = rotate(q, positions, m.get("rot")), rotate(k, positions, m.get("rot"))
    a = sink_attention(q, k, v, m["scale"], visible(positions, m.get("mask")), f64(w[p + ".sink"])).reshape(T, H * dv)
    return (a * sigmoid(h @ f64(w[p + ".g"]).T)) @ f64(w[p + ".o"]).T


# ---- the recurrence -----------------------------------------------------------------------

def short_conv(u, kernel, bias, before=None):
    """u [T, channels]: out_t = bias + sum over taps i of kernel[:, i] u_(t - taps + 1 + i); ``before`` holds the
    taps - 1 rows in front of the first one (zeros at the start of a sequence)."""
    u, kernel = f64(u), f64(kernel)
    taps = kernel.shape[1]
    rows = np.concatenate([np.zeros((taps - 1, u.shape[1])) if before is None else f64(before), u])
    return sum(rows[i:i + u.shape[0]] * kernel[:, i] for i in range(taps)) + f64(bias)


def ssd_scan(x, B, C, dt, A_log, D, state=None):
    """x [T, H, dv], B, C [T, G, N], dt [T, H] (after the softplus): S_t = exp(-exp(A_log_h) dt) S_(t-1) + dt B_t x_t^T,
    y_t = S_t^T C_t + D_h x_t, token by token.  Returns (y [T, H, dv], the last state [H, N, dv])."""
    x, B, C, dt = f64(x), f64(B), f64(C), f64(dt)
    T, H, dv = x.shape
    per = H // B.shape[1]
    Bh, Ch = np.repeat(B, per, axis=1), np.repeat(C, per, axis=1)
    S = np.zeros((H, B.shape[2], dv)) if state is None else f64(state).copy()
    y = np.zeros((T, H, dv))
    rate = np.exp(f64(A_log))
    for t in range(T):
        S = np.exp(-rate * dt[t])[:, None, None] * S + (dt[t][:, None] * Bh[t])[:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hne,hn->he", S, Ch[t]) + f64(D)[:, None] * x[t]
    return y, S


def gate_then_norm(y, z, gain, parts, eps):
    """y * silu(z), then each of ``parts`` equal pieces of the row divided by its root mean square, times the gain."""
    g = f64(y) * silu(f64(z))
    T = g.shape[0]
    return unit_rms(g.reshape(T, parts, -1), eps).reshape(T, -1) * f64(gain)


def mamba2_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    proj = h @ f64(w[p + ".in"]).T
    z, u, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    u = silu(short_conv(u, w[p + ".conv"], w[p + ".conv.b"]))
    x = u[:, :inner].reshape(T, H, dv)
    B, C = u[:, inner:inner + G * N].reshape(T, G, N), u[:, inner + G * N:].reshape(T, G, N)
    y, _ = ssd_scan(x, B, C, softplus(dt + f64(w[p + ".dt_bias"])), w[p + ".A_log"], w[p + ".D"])
    return gate_then_norm(y.reshape(T, inner), z, w[p + ".norm"], m["norm_groups"], eps) @ f64(w[p + ".o"]).T


# ---- feed-forwards ----------------------------------------------------------------------

def dense_ff(h, w, p, limit):
    g = np.minimum(h @ f64(w[p + ".gate"]).T, limit)
    u = np.clip(h @ f64(w[p + ".up"]).T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ f64(w[p + ".down"]).T


def relu2_ff(h, w, p):
    return (np.maximum(h @ f64(w[p + ".up"]).T, 0.0) ** 2) @ f64(w[p + ".down"]).T


def route(h, router, correction, top):
    """(experts [T, top], weights [T, top]): chosen by softmax score + correction, weighted by the scores alone over
    their sum."""
    z = f64(h) @ f64(router).T
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s /= s.sum(axis=1, keepdims=True)
    idx = np.argsort(-(s + f64(correction)), axis=1, kind="stable")[:, :top]
    wt = np.take_along_axis(s, idx, axis=1)
    return idx, wt / (wt.sum(axis=1, keepdims=True) + 1e-20)


def routed_ff(h, w, p, m):
    """Experts without a gate, identity experts behind them (their output is the input), and the expert that every
    token runs, if there is one."""
    y = relu2_ff(h, w, p + ".shared") if m.get("shared") else np.zeros_like(f64(h))
    idx, wt = route(h, w[p + ".router"], w[p + ".correction"], m["router"]["top"])
    for t in range(h.shape[0]):
        for e, s in zip(idx[t], wt[t]):
            y[t] += s * (relu2_ff(h[t], w, f"{p}.e{e}") if e < m["router"]["experts"] else h[t])
    return y


# ---- the model --------------------------------------------------------------------------

def forward(w, cfg, ids, return_layers=False):
    """Logits float64 [T, vocab] for the token ids of one sequence, positions 0 .. T-1."""
    eps = float(cfg["norm"]["eps"])
    ids = np.asarray(ids, dtype=np.int64)
    positions = np.arange(len(ids))
    x = layer_norm(f64(w["embed"])[ids], w["embed.norm"], eps)
    layers = []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}"
        if L["type"] == "attention":
            y = attention_mixer(x, w, p + ".mix", L["mixer"], eps, positions)
        elif L["type"] == "mamba2":
            y = mamba2_mixer(x, w, p + ".mix", L["mixer"], eps)
        else:
            raise ValueError(L["type"])
        x = x + layer_norm(y, w[p + ".norm1"], eps) * f64(w[p + ".ls1"])
        mlp = L.get("mlp")
        if mlp:
            y = dense_ff(x, w, p + ".mlp", mlp["limit"]) if mlp["kind"] == "dense" else routed_ff(x, w, p + ".mlp", mlp)
            x = x + layer_norm(y, w[p + ".norm2"], eps) * f64(w[p + ".ls2"])
        layers.append(x.copy())
    z = layer_norm(x, w["final.norm"], eps) @ f64(w["head"]).T * float(cfg["logit_scale"])
    return (z, np.stack(layers)) if return_layers else z


# ---- random models ----------------------------------------------------------------------

def tensor_shapes(cfg):
    d, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, d), "embed.norm": (d,), "final.norm": (d,), "head": (V, d)}
    for i, L in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}", L["mixer"], L.get("mlp")
        q = p + ".mix"
        out.update({p + ".norm1": (d,), p + ".ls1": (d,)})
        if L["type"] == "attention":
            A, K, V_ = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            B = m["heads"] * m["vdim"]
            out.update({q + ".q": (A, d), q + ".k": (K, d), q + ".v": (V_, d), q + ".q.norm": (m["dim"],),
                        q + ".k.norm": (m["dim"],), q + ".sink": (m["heads"],), q + ".g": (B, d), q + ".o": (d, B)})
        else:
            inner, GN, H = m["heads"] * m["vdim"], m["groups"] * m["state"], m["heads"]
            ch = inner + 2 * GN
            out.update({q + ".in": (inner + ch + H, d), q + ".conv": (ch, m["conv"]), q + ".conv.b": (ch,),
                        q + ".dt_bias": (H,), q + ".A_log": (H,), q + ".D": (H,), q + ".norm": (inner,), q + ".o": (d, inner)})
        if not mlp:
            continue
        out.update({p + ".norm2": (d,), p + ".ls2": (d,)})
        if mlp["kind"] == "dense":
            f = mlp["ff"]
            out.update({p + ".mlp.gate": (f, d), p + ".mlp.up": (f, d), p + ".mlp.down": (d, f)})
        else:
            E = mlp["router"]["experts"]
            total = E + (mlp["router"].get("identity") or 0)
            out.update({p + ".mlp.router": (total, d), p + ".mlp.correction": (total,)})
            plain = [(f"e{e}", mlp["expert"]["ff"]) for e in range(E)]
            if mlp.get("shared"):
                plain.append(("shared", mlp["shared"]["ff"]))
            for n, f in plain:
                out.update({f"{p}.mlp.{n}.up": (f, d), f"{p}.mlp.{n}.down": (d, f)})
    return out


def random_weights(cfg, seed, std=0.12, qk_gain=2.0):
    """Weights that make every mechanism count, all of them bfloat16 numbers (both dtypes load the same model):
    matrices N(0, std) scaled by 1 / sqrt(fan-in / 64), norm weights and layer scales around one, decays from quick to
    slow, sinks around the scores' size, routers wide and corrections large enough that the choices differ;
    ``qk_gain`` multiplies the weights of the queries' and the keys' norms, which sharpens the attention."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith((".q.norm", ".k.norm")):
            t = math.sqrt(qk_gain) * (1.0 + 0.2 * rng.standard_normal(shape))
        elif name.endswith(".sink"):
            t = 1.5 * rng.standard_normal(shape)
        elif name.endswith(".A_log"):
            t = rng.uniform(-3.0, 1.0, shape)
        elif name.endswith(".dt_bias"):
            t = rng.uniform(-4.0, 0.5, shape)
        elif name.endswith(".D"):
            t = rng.uniform(1.5, 3.0, shape)       # a head's value D x + S^T C does not cross zero as a whole
        elif name.endswith(".correction"):
            t = rng.uniform(-0.1, 0.1, shape)
        elif name.endswith(".conv"):
            t = 0.5 * rng.standard_normal(shape)
        elif name.endswith(".conv.b"):
            t = 0.3 * rng.standard_normal(shape)
        elif name.endswith((".ls1", ".ls2")):
            t = 0.6 + 0.2 * rng.standard_normal(shape)
        elif len(shape) == 1:
            t = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name == "embed":
            t = rng.standard_normal(shape)
        else:
            t = rng.standard_normal(shape) * std * math.sqrt(64.0 / shape[1])
            if name.endswith(".router"):
                t = t * 2.0
            if name.endswith(".mix.in"):
                t = t * 2.0
        w[name] = round_bf16(t.astype(np.float32))
    return w


def round_bf16(a):
    """float32 array rounded to the nearest bfloat16 (ties to even), as float32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).reshape(np.shape(a))
