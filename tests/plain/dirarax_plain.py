"""Plain, slow Dirarax forward pass in numpy float64: the yardstick of its tests.

Whole sequences, no cache, no paging, no batches; one function per mechanism.
Nothing here is imported by the product package and nothing of the product
package is imported here.  Weights arrive as a dict of tensor name -> numpy
array and are widened to float64; ``cfg`` is the dict of a config.json.

Notation: T tokens, d the model width, H heads, G key/value heads, dk the per-head
query/key size, dv the per-head value size.
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    x = f64(x)
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def norm_one_plus(x, w, eps):
    """x / rms(x) * (1 + w): the weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + f64(w))


def token_shift(h, mu, before=None):
    """h [T, d]: every row moved towards the row before it, channel by channel, by mu [d]; ``before`` is the row
    in front of the first one (zeros at the start of a sequence)."""
    h = f64(h)
    prev = np.concatenate([np.zeros((1, h.shape[1])) if before is None else f64(before)[None], h[:-1]])
    return h + (prev - h) * f64(mu)


# ---- rotation ---------------------------------------------------------------------------

def frequencies(rot):
    """(angles per position [dims / 2], amplitude of cos and sin) of a rotation {dims, base, scaling or none}."""
    dims, base = rot["dims"], float(rot["base"])
    f = base ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(dim_of(sc["fast"])), 0)
    hi = min(math.ceil(dim_of(sc["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot, interleaved):
    """x [T, heads, size]: the first rot.dims values of every head are turned pair by pair: (2i, 2i + 1) when
    ``interleaved``, else (i, i + dims / 2)."""
    x = f64(x).copy()
    if not rot:
        return x
    dims = rot["dims"]
    f, amp = frequencies(rot)
    a = f64(positions)[:, None, None] * f
    c, s = np.cos(a) * amp, np.sin(a) * amp
    first = slice(0, dims, 2) if interleaved else slice(0, dims // 2)
    second = slice(1, dims, 2) if interleaved else slice(dims // 2, dims)
    u, v = x[..., first].copy(), x[..., second].copy()
    x[..., first] = u * c - v * s
    x[..., second] = v * c + u * s
    return x


# ---- mixers -----------------------------------------------------------------------------

def causal_attention(q, k, v, scale):
    """q [T, H, dk] over k [T, G, dk], v [T, G, dv]: softmax over the keys j <= i."""
    q, k, v = f64(q), f64(k), f64(v)
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for hd in range(H):
        s = q[:, hd] @ k[:, hd // per].T * scale
        s[np.triu_indices(T, 1)] = -np.inf
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, hd] = (e / e.sum(axis=1, keepdims=True)) @ v[:, hd // per]
    return out


def decayed_scan(q, k, v, alpha, state=None):
    """q, k, alpha [T, H, dk], v [T, H, dv]: S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, token by
    token.  Returns (o [T, H, dv], the last state [H, dk, dv])."""
    q, k, v, alpha = f64(q), f64(k), f64(v), f64(alpha)
    T, H, dk = q.shape
    S = np.zeros((H, dk, v.shape[2])) if state is None else f64(state).copy()
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hde,hd->he", S, q[t])
    return o, S


def gla_decay(h, w, p, tau, H):
    """alpha [T, H, dk] = sigmoid(W_a2 W_a1 h + b)^(1 / tau)."""
    z = (h @ f64(w[p + ".a1"]).T) @ f64(w[p + ".a2"]).T + f64(w[p + ".a2.b"])
    return sigmoid(z).reshape(h.shape[0], H, -1) ** (1.0 / tau)


def gla_mixer(h, w, p, m, eps):
    """Gated linear attention: a decay per key channel that depends on the token."""
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ f64(w[p + ".q"]).T).reshape(T, H, dk) * dk ** -0.5
    k = (h @ f64(w[p + ".k"]).T).reshape(T, H, dk)
    v = (h @ f64(w[p + ".v"]).T).reshape(T, H, dv)
    o, _ = decayed_scan(q, k, v, gla_decay(h, w, p, m["tau"], H))
    o = unit_rms(o, eps) * f64(w[p + ".norm"])
    return (o.reshape(T, H * dv) * silu(h @ f64(w[p + ".g"]).T)) @ f64(w[p + ".o"]).T


def gated_attention_mixer(h, w, p, m, positions):
    """Grouped causal attention with an interleaved partial rotation and a sigmoid gate on the heads' outputs."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate((h @ f64(w[p + ".q"]).T).reshape(T, H, dk), positions, m.get("rot"), True)
    k = rotate((h @ f64(w[p + ".k"]).T).reshape(T, G, dk), positions, m.get("rot"), True)
    v = (h @ f64(w[p + ".v"]).T).reshape(T, G, dv)
    a = causal_attention(q, k, v, m["scale"]).reshape(T, H * dv)
    return (a * sigmoid(h @ f64(w[p + ".g"]).T)) @ f64(w[p + ".o"]).T


def retention_mixer(h, w, p, m, eps, positions):
    """Linear attention with a fixed decay per head over rotated queries and keys."""
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = rotate((h @ f64(w[p + ".q"]).T).reshape(T, H, dk), positions, m.get("rot"), False)
    k = rotate((h @ f64(w[p + ".k"]).T).reshape(T, H, dk), positions, m.get("rot"), False) * dk ** -0.5
    v = (h @ f64(w[p + ".v"]).T).reshape(T, H, dv)
    alpha = np.broadcast_to(f64(m["decay"])[None, :, None], (T, H, dk))
    o, _ = decayed_scan(q, k, v, alpha)
    return (unit_rms(o, eps).reshape(T, H * dv) * silu(h @ f64(w[p + ".g"]).T)) @ f64(w[p + ".o"]).T


def parallel_mixer(h, w, p, m, eps, positions):
    return (m["left_scale"] * gated_attention_mixer(h, w, p + ".left", m["left"], positions)
            + m["right_scale"] * retention_mixer(h, w, p + ".right", m["right"], eps, positions))


# ---- feed-forwards ----------------------------------------------------------------------

def dense_ff(h, w, p):
    def lin(x, n):
        return x @ f64(w[f"{p}.{n}"]).T + f64(w[f"{p}.{n}.b"])
    return lin(gelu_tanh(lin(h, "gate")) * lin(h, "up"), "down")


def gated_silu(h, w, p):
    return (silu(h @ f64(w[p + ".gate"]).T) * (h @ f64(w[p + ".up"]).T)) @ f64(w[p + ".down"]).T


def routed_ff(h, w, p, m):
    """The ``top`` experts with the largest logits, weighted by the softmax over those logits alone, plus the
    expert that every token runs (if there is one)."""
    z = h @ f64(w[p + ".router"]).T
    y = gated_silu(h, w, p + ".shared") if m.get("shared") else np.zeros_like(h)
    for t in range(h.shape[0]):
        best = np.argsort(-z[t], kind="stable")[:m["router"]["top"]]
        e = np.exp(z[t, best] - z[t, best].max())
        for j, wt in zip(best, e / e.sum()):
            y[t] += wt * gated_silu(h[t], w, f"{p}.e{j}")
    return y


# ---- the model --------------------------------------------------------------------------

def layer_runs(cfg):
    """[(layer, pass or None)] in order; pass t stands at the first layer of the loop's t-th pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    run = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        run += [(i, t if i == a else None) for i in range(a, b)]
    return run + [(i, None) for i in range(b, n)]


def pass_entry(x, x0, w, t):
    """What the stream becomes before the first layer of pass t."""
    return np.concatenate([x, x0], axis=1) @ f64(w["loop.in"]).T + f64(w["loop.step"])[t]


def forward(w, cfg, ids, return_layers=False):
    """Logits float64 [T, vocab] for the token ids of one sequence, positions 0 .. T-1."""
    eps = float(cfg["norm"]["eps"])
    ids = np.asarray(ids, dtype=np.int64)
    positions = np.arange(len(ids))
    x0 = x = f64(w["embed"])[ids]
    layers = []
    for i, t in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}"
        if t is not None:
            x = pass_entry(x, x0, w, t)
        h = norm_one_plus(x, w[p + ".norm1"], eps)
        hs = token_shift(h, w[p + ".shift"])
        if L["type"] == "gla":
            y = gla_mixer(hs, w, p + ".mix", L["mixer"], eps)
        elif L["type"] == "parallel":
            y = parallel_mixer(hs, w, p + ".mix", L["mixer"], eps, positions)
        else:
            raise ValueError(L["type"])
        if L.get("mlp"):
            y = y + (dense_ff(h, w, p + ".mlp") if L["mlp"]["kind"] == "dense" else routed_ff(h, w, p + ".mlp", L["mlp"]))
        x = x + y
        layers.append(x.copy())
    z = norm_one_plus(x, w["final.norm"], eps) @ f64(w["embed"]).T
    return (z, np.stack(layers)) if return_layers else z


# ---- random models ----------------------------------------------------------------------

def tensor_shapes(cfg, rank=5):
    """Names and shapes; ``rank`` is the inner size of the decay's two matrices, which no configuration key names."""
    d, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, d), "final.norm": (d,)}
    if cfg.get("loop"):
        out.update({"loop.in": (d, 2 * d), "loop.step": (cfg["loop"]["times"], d)})
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}", L["mixer"]
        out.update({p + ".norm1": (d,), p + ".shift": (d,)})

        def linear_attention(q, s):
            A, B = s["heads"] * s["dim"], s["heads"] * s["vdim"]
            out.update({q + ".q": (A, d), q + ".k": (A, d), q + ".v": (B, d), q + ".g": (B, d), q + ".o": (d, B)})
        if L["type"] == "gla":
            linear_attention(p + ".mix", m)
            A = m["heads"] * m["dim"]
            out.update({p + ".mix.norm": (m["vdim"],), p + ".mix.a1": (rank, d), p + ".mix.a2": (A, rank),
                        p + ".mix.a2.b": (A,)})
        else:
            a, q = m["left"], p + ".mix.left"
            B = a["heads"] * a["vdim"]
            out.update({q + ".q": (a["heads"] * a["dim"], d), q + ".k": (a["kv_heads"] * a["dim"], d),
                        q + ".v": (a["kv_heads"] * a["vdim"], d), q + ".g": (B, d), q + ".o": (d, B)})
            linear_attention(p + ".mix.right", m["right"])
        mlp = L.get("mlp")
        if mlp and mlp["kind"] == "dense":
            f = mlp["ff"]
            out.update({p + ".mlp.gate": (f, d), p + ".mlp.gate.b": (f,), p + ".mlp.up": (f, d), p + ".mlp.up.b": (f,),
                        p + ".mlp.down": (d, f), p + ".mlp.down.b": (d,)})
        elif mlp:
            out[p + ".mlp.router"] = (mlp["router"]["experts"], d)
            gated = [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            if mlp.get("shared"):
                gated.append(("shared", mlp["shared"]["ff"]))
            for n, f in gated:
                out.update({f"{p}.mlp.{n}.gate": (f, d), f"{p}.mlp.{n}.up": (f, d), f"{p}.mlp.{n}.down": (d, f)})
    return out


def random_weights(cfg, seed, std=0.12, qk_boost=1.0, rank=5):
    """Weights that make every mechanism count, all of them bfloat16 numbers (both dtypes load the same model):
    matrices N(0, std) scaled by 1 / sqrt(fan-in / 64), one-plus weights around zero, plain weights around one,
    shifts in (0, 1), routers wide enough that the choices differ; ``qk_boost`` scales the softmax attention's
    query and key projections, which sharpens it."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        if name.endswith(".norm1") or name == "final.norm":
            t = 0.2 * rng.standard_normal(shape)
        elif name.endswith(".shift"):
            t = rng.uniform(0.0, 1.0, shape)
        elif name.endswith(".mix.norm"):
            t = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name.endswith(".a2.b"):
            t = rng.uniform(-4.0, 4.0, shape)
        elif len(shape) == 1 or name == "loop.step":
            t = 0.3 * rng.standard_normal(shape)
        elif name == "embed":
            t = rng.standard_normal(shape)
        else:
            t = rng.standard_normal(shape) * std * math.sqrt(64.0 / shape[1])
            if name.endswith((".left.q", ".left.k")):
                t = t * qk_boost
            if name.endswith(".router"):
                t = t * 4.0
        w[name] = round_bf16(t.astype(np.float32))
    return w


def round_bf16(a):
    """float32 array rounded to the nearest bfloat16 (ties to even), as float32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).reshape(np.shape(a))
