"""The Rupenex design in the engine against its plain implementation (tests/plain/rupenex_plain.py).

Small configurations of their own, random weights whose values are bfloat16 numbers (so both
dtypes load the same model): each mechanism's kernel alone, whole prompts, prompts against
token-by-token decoding, portions down to two tokens, unequal batches, slots and pages that
are used again, keys just inside and just outside the window and the kept first keys, far keys and page borders that
one score makes stand out, the first tokens, long decoding through CUDA graphs, and greedy generation through
the scheduler.
"""
import copy

import numpy as np
import pytest

from helpers import write_model_dir
from plain import rupenex_plain as P
from test_gpu_sozarax import _ctx, _paged, _t, check_rows, engine_for, run_cut

pytestmark = pytest.mark.gpu


def _attn(heads, kv_heads, dim, vdim, scale, mask=None, rot=None):
    """mask: (size, keep_first) or (size,); rot: (dims, base) or (dims, base, factor)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if mask:
        m["mask"] = dict(zip(("size", "keep_first"), mask))
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = {"factor": rot[2]}
    return {"type": "attention", "mixer": m}


def _mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def _dense(layer, ff, limit):
    return dict(layer, mlp={"kind": "dense", "ff": ff, "limit": limit})


def _moe(layer, experts, top, ff, identity=0, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if identity:
        m["router"]["identity"] = identity
    if shared:
        m["shared"] = {"ff": shared}
    return dict(layer, mlp=m)


def _alone(layer):
    return dict(layer, mlp=None)


def _cfg(vocab, width, eps, logit_scale, layers):
    return {"architecture": "Rupenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": layers}


# A: sizes that suit vector widths; every kind of mask, rotation and feed-forward; parts of the norm that span heads, are a
# head, or lie inside one; windows shorter and longer than a page, kept keys below, at and above a page's border.
CFG_A = _cfg(96, 64, 1e-5, 1.7, [
    _moe(_attn(4, 2, 16, 24, 0.3, (24, 7), (16, 1000.0, 3.0)), 5, 2, 24, 3, 40),
    _dense(_mamba(4, 16, 24, 2, 4, 2), 72, 1.5),
    _alone(_attn(6, 1, 8, 8, 0.5, (5, 16), (4, 50.0))),
    _moe(_mamba(6, 8, 16, 3, 3, 3), 4, 1, 32),
    _dense(_attn(2, 2, 32, 16, 0.2, (70,)), 48, 7.0),
    _moe(_mamba(2, 24, 8, 1, 2, 4), 3, 3, 16, 1),
])
# B: sizes that fit no vector width or tile; plain causal attention; one tap, one head; more chosen than there are experts with matrices.
CFG_B = _cfg(61, 50, 1e-6, -0.6, [
    _dense(_mamba(3, 7, 5, 3, 1, 7), 22, 2.5),
    _moe(_attn(3, 3, 10, 6, 0.4), 2, 4, 14, 3, 9),
    _alone(_mamba(1, 30, 11, 1, 6, 1)),
    _dense(_attn(2, 1, 6, 9, 0.6, (33, 21), (6, 10.0, 0.5)), 13, 1.0),
])
# C: head sizes of the tensor-core attention with values narrower and wider than keys and of the same size, windows
# longer than the kernels' tiles, wide recurrent heads (several tiles of both sizes).
CFG_C = _cfg(80, 128, 1e-6, 3.0, [
    _moe(_attn(4, 2, 64, 128, 0.125, (90, 33), (64, 10000.0, 8.0)), 6, 3, 32, 2, 64),
    _dense(_mamba(2, 128, 160, 1, 4, 2), 96, 3.0),
    _dense(_attn(4, 4, 32, 64, 0.2, (17, 64), (16, 500.0)), 160, 0.7),
    _moe(_mamba(4, 80, 36, 2, 5, 1), 8, 2, 64, 4, 32),
    _moe(_attn(8, 2, 48, 48, 0.15, (64, 1), (48, 2000.0, 2.0)), 4, 2, 48, 1),
])
# D: sizes in steps of 16 as a small served model has them.
CFG_D = _cfg(160, 224, 1e-5, 0.5, [
    _moe(_mamba(8, 32, 64, 4, 4, 4), 6, 2, 48, 2, 112),
    _dense(_mamba(5, 48, 32, 5, 4, 5), 256, 2.0),
    _moe(_attn(7, 7, 64, 64, 0.17, (48, 32), (64, 20000.0, 4.0)), 4, 2, 64, 4, 48),
    _dense(_attn(8, 4, 80, 80, 0.11, (32, 16), (40, 20000.0, 16.0)), 128, 4.0),
])
CFGS = {"A": (CFG_A, 71), "B": (CFG_B, 72), "C": (CFG_C, 73), "D": (CFG_D, 74)}


def every_expert(cfg):
    """All experts chosen: in bfloat16 no close call of a router, which rounding may turn the other way and the states then
    carry on, stands between two runs."""
    cfg = copy.deepcopy(cfg)
    for L in cfg["layers"]:
        if L["mlp"] and L["mlp"]["kind"] == "moe":
            r = L["mlp"]["router"]
            r["top"] = r["experts"] + r.get("identity", 0)
    return cfg


def write(path, cfg, w):
    return write_model_dir(str(path), cfg, {k: np.asarray(v, dtype=np.float32) for k, v in w.items()})


def make_model(tmp_path, name, qk_gain=2.0, all_experts=False):
    cfg, seed = CFGS[name]
    cfg = every_expert(cfg) if all_experts else cfg
    w = P.random_weights(cfg, seed, qk_gain=qk_gain)
    return cfg, w, write(tmp_path / f"rupenex_{name}", cfg, w)


# ---- whole models --------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole_prompt_and_every_way_of_cutting(tmp_path, name, dtype):
    cfg, w, d = make_model(tmp_path, name, 2.0 if dtype == "float32" else 1.0, all_experts=dtype == "bfloat16")
    rng = np.random.default_rng(5)
    ids = rng.integers(0, cfg["vocab"], size=150).tolist()
    want, layers = P.forward(w, cfg, ids, return_layers=True)
    eng = engine_for(d, dtype)
    try:
        got_taps = []
        eng.model.tap = lambda i, x: got_taps.append(x.detach().float().cpu().numpy().copy())
        whole = run_cut(eng, ids, [len(ids)])
        eng.model.tap = None
        assert len(got_taps) == len(layers)
        for i, (g, t) in enumerate(zip(got_taps, layers)):      # the residual stream after every layer
            err = np.abs(g - t).max() / np.abs(t).max()
            assert err <= (1e-4 if dtype == "float32" else 1e-1), (name, i, err)
        check_rows(whole, want, dtype, f"{name} whole")
        check_rows(run_cut(eng, ids[:3], [3]), want[:3], dtype, f"{name} first tokens")
        check_rows(run_cut(eng, ids[:1], [1]), want[:1], dtype, f"{name} one token")
        check_rows(run_cut(eng, ids, [len(ids) - 70, 1]), want, dtype, f"{name} prompt then decode")
        check_rows(run_cut(eng, ids[:70], [1]), want[:70], dtype, f"{name} decode from the start")
        for cuts in ([2], [3, 2, 37, 16, 5, 2, 64, 1], [17], [16, 16, 1, 31, 2], [64, 64, 2], [65, 63]):
            got = run_cut(eng, ids, cuts)
            check_rows(got, want, dtype, f"{name} portions {cuts}")
            if dtype == "float32":
                # small steps take other product kernels than large ones, chunks other sums: another order
                assert np.abs(got - whole).max() <= 5e-5 * np.abs(want).max(), cuts
    finally:
        eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "D"])
def test_unequal_batches_and_reuse_of_slots_and_pages(tmp_path, name, dtype):
    """Four requests of unequal length in one batch, portions of some beside single tokens of
    others, then new requests in the slots and pages that the finished ones gave back; a pool
    that holds little more than what is live.  Every request also runs alone."""
    from kllm_b200.engine.step import StepEntry
    cfg, w, d = make_model(tmp_path, name, 2.0 if dtype == "float32" else 1.0, all_experts=dtype == "bfloat16")
    rng = np.random.default_rng(9)
    lens = [37, 130, 5, 64, 21, 50]
    seqs = [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lens]
    want = [P.forward(w, cfg, s) for s in seqs]
    eng = engine_for(d, dtype, num_blocks=20, max_batch=4)      # 320 tokens of pages, four slots
    try:
        got = [np.zeros_like(x) for x in want]
        fed = [0] * len(seqs)
        caches = {}
        queue = list(range(len(seqs)))
        sizes = [3, 1, 16, 2, 70, 1, 7]
        turn = 0
        slots_seen = []
        while queue or caches:
            while queue and len(caches) < 4:
                i = queue.pop(0)
                caches[i] = eng.cache.open()
                slots_seen.append(caches[i].state_slot)
            entries, order = [], []
            for i in list(caches):
                if len(caches) > 2 and (turn + i) % 5 == 0:
                    continue                                    # left out of this step, goes on later
                left = len(seqs[i]) - fed[i]
                n = 1 if left <= 8 else min(left, sizes[(turn + i) % len(sizes)])
                entries.append(StepEntry(caches[i], seqs[i][fed[i]:fed[i] + n], list(range(n))))
                order.append((i, n))
            lg = eng.runner.run(entries).float().cpu().numpy()
            r = 0
            for i, n in order:
                got[i][fed[i]:fed[i] + n] = lg[r:r + n]
                r += n
                fed[i] += n
                if fed[i] == len(seqs[i]):
                    eng.cache.close(caches.pop(i))
            turn += 1
            eng.cache.audit()
        assert len(slots_seen) > len(set(slots_seen)), "no state slot was used again"
        for i in range(len(seqs)):
            check_rows(got[i], want[i], dtype, f"request {i} in mixed batches")
            alone = run_cut(eng, seqs[i], [len(seqs[i])])
            if dtype == "float32":
                assert np.abs(alone - got[i]).max() <= 3e-5 * np.abs(want[i]).max(), f"request {i} alone against the batch"
            else:
                check_rows(alone, got[i], dtype, f"request {i} alone against the batch")
    finally:
        eng.close()


def test_long_decoding_gives_window_pages_back(tmp_path):
    """A short prompt and then hundreds of single tokens (graphs, pages added one by one, windows that pass over decoded
    tokens, states carried through hundreds of steps); the groups with a window hold their window's pages and those
    of the kept first keys, no more, and other requests use what came back."""
    cfg, w, d = make_model(tmp_path, "D")
    rng = np.random.default_rng(3)
    ids = rng.integers(0, cfg["vocab"], size=400).tolist()
    want = P.forward(w, cfg, ids)
    eng = engine_for(d, "float32", max_seq=448, num_blocks=26)
    try:
        check_rows(run_cut(eng, ids, [9, 1]), want, "float32", "long decoding")
        from kllm_b200.engine.step import StepEntry
        c = eng.cache.open()
        eng.runner.run([StepEntry(c, ids[:300], [])])
        eng.runner.run([StepEntry(c, ids[300:301], [0])])
        for g, table in zip(eng.cache.groups, c.tables):
            held = [j for j, p in enumerate(table) if p >= 0]
            first = (302 - g.need.window) // 16
            assert held == sorted(set(range(-(-g.need.keep_first // 16))) | set(range(first, 19))), (g.need, held)
        eng.cache.close(c)
        eng.cache.audit()
    finally:
        eng.close()


def test_greedy_generation_through_the_scheduler(tmp_path):
    """``Engine.generate`` (scheduler, sampler, pipelined steps whose token ids stay on the device) on several
    prompts at once against greedy decoding with the plain implementation."""
    cfg, w, d = make_model(tmp_path, "A")
    rng = np.random.default_rng(21)
    prompts = [rng.integers(0, cfg["vocab"], size=n).tolist() for n in (7, 30, 2, 19, 45)]
    steps = 12
    eng = engine_for(d, "float32", max_step_tokens=48, max_batch=3)
    try:
        outs = eng.generate(prompts, max_new_tokens=steps)
        alone = eng.generate(prompts[1], max_new_tokens=steps)
    finally:
        eng.close()
    assert alone == outs[1]
    for p, out in zip(prompts, outs):
        ids = list(p)
        for k in range(steps):
            z = P.forward(w, cfg, ids)[-1]
            best = int(z.argmax())
            assert out[k] == best or z[best] - z[out[k]] < 1e-4 * np.abs(z).max(), (len(p), k)
            ids.append(out[k])


@pytest.mark.parametrize("name", ["A", "D"])
def test_replay_program(tmp_path, name):
    """bin/trace_run on a model of this design: whole, decode, portions and mixed batches of up
    to four live requests in a pool as small as the trace allows."""
    from test_gpu_replay import build_trace
    from trace_tools import run_trace
    cfg, w, d = make_model(tmp_path, name, 1.0, all_experts=True)
    rng = np.random.default_rng(4)
    seqs = [rng.integers(0, cfg["vocab"], size=n).tolist() for n in (5, 33, 64, 100, 18)]
    want = [P.forward(w, cfg, s) for s in seqs]
    tb = build_trace(seqs, [7, 2, 13, 3, 1, 29], seed=8)
    for dtype in ("float32", "bfloat16"):
        rows = run_trace(d, dtype, tb, str(tmp_path / ("out_" + dtype)), cfg["vocab"])
        by_way = {}
        for (rid, pos), z in rows.items():
            by_way.setdefault((rid[0], int(rid[1:])), {})[pos] = z
        for (way, i), zs in by_way.items():
            pos = sorted(zs)
            check_rows(np.stack([zs[p] for p in pos]), want[i][pos], dtype, f"replay {way}{i}")


# ---- the recurrence's kernels alone ----------------------------------------------------------------

def _ssd_inputs(rng, n, H, dv, N, G, taps):
    inner, ch = H * dv, H * dv + 2 * G * N
    proj = rng.standard_normal((n, inner + ch + H))
    w = {"conv": rng.standard_normal((ch, taps)) * 0.6, "conv_b": rng.standard_normal(ch) * 0.3,
         "dt_bias": rng.uniform(-3, 1, H), "a_log": rng.uniform(-2, 1.5, H), "d": rng.standard_normal(H)}
    return proj, w


def _ssd_plain(proj, w, H, dv, N, G, rounded=None):
    """(gated rows, last state, inputs of the convolution) of one whole sequence; ``rounded`` [T]: rows whose x, B and C are
    rounded to bfloat16 behind silu."""
    T, inner, ch = proj.shape[0], H * dv, H * dv + 2 * G * N
    u = proj[:, inner:inner + ch]
    v = P.silu(P.short_conv(u, w["conv"], w["conv_b"]))
    if rounded is not None:
        v = np.where(np.asarray(rounded)[:, None], P.round_bf16(v).astype(np.float64), v)
    y, S = P.ssd_scan(v[:, :inner].reshape(T, H, dv), v[:, inner:inner + G * N].reshape(T, G, N), v[:, inner + G * N:].reshape(T, G, N),
                      P.softplus(proj[:, inner + ch:] + w["dt_bias"]), w["a_log"], w["d"])
    return y.reshape(T, inner) * P.silu(proj[:, :inner]), S, u


def _ssd_run(proj, ctx, w, state, ring, H, dv, N, G, dtype="float32"):
    import torch
    from kllm_b200 import kernels
    wide = np.concatenate([proj, np.zeros((proj.shape[0], -proj.shape[1] % 8))], axis=1)      # as a padded product leaves it
    return kernels.ssd(_t(wide), _t(w["conv"]), _t(w["conv_b"]), _t(w["dt_bias"]), _t(w["a_log"]), _t(w["d"]), state, ring, ctx, H, G,
                       N, dv, dtype=getattr(torch, dtype)).cpu().numpy()


# float32: float32 sums against float64 ones.  bfloat16: the plain scan rounds x, B and C where the kernels do, so what is
# left is the two bfloat16 terms of what is float32, and values of x, B and C that round the other way.
SSD_TOL = {"float32": 3e-5, "bfloat16": 1e-3}


def _tensor_cores(dtype, N, dv):
    return dtype == "bfloat16" and N % 16 == 0 and dv % 16 == 0 and N <= 256


SSD_SIZES = [(4, 16, 24, 2, 4), (3, 40, 8, 3, 3), (2, 64, 128, 1, 4), (1, 7, 5, 1, 1), (6, 10, 6, 2, 2), (2, 128, 160, 2, 4),
             (1, 300, 36, 1, 6), (8, 32, 64, 4, 4), (5, 3, 130, 5, 9), (2, 66, 32, 1, 5),
             (3, 16, 16, 1, 4), (4, 80, 48, 2, 4), (2, 192, 256, 1, 3), (6, 64, 144, 3, 2)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dv,N,G,taps", SSD_SIZES)
def test_state_space_scan_carries_its_states(H, dv, N, G, taps, dtype):
    """Three requests of unequal length in one launch (several chunks, one short chunk, one row), then portions that start
    from the slots at odd places (shorter than the convolution too), then steps of one row each, in slots 3, 0 and 2, against the
    plain token-by-token scan over each whole sequence; the states left in the slots too, and an untouched slot."""
    import torch
    rng = np.random.default_rng(H * dv + N)
    lens = [405, 32, 8]
    n, ch = sum(lens), H * dv + 2 * G * N
    row = -(-ch // 4) * 4
    proj, w = _ssd_inputs(rng, n, H, dv, N, G, taps)
    state, ring = torch.zeros((4, H * N * dv + 4), device="cuda"), torch.zeros((4, taps * row + 8), device="cuda")
    slots, offs = [3, 0, 2], np.concatenate([[0], np.cumsum(lens)])
    got = np.zeros((n, H * dv))
    # (first, last) rows of each request per launch
    plan = [[(0, 130), (0, 9), (0, 1)], [(130, 132), (9, 27), (1, 4)], [(132, 133), (27, 28), (4, 5)],
            [(133, 135), (28, 30), (5, 7)], [(135, 400), (30, 31), None], [(400, 401), (31, 32), (7, 8)],
            [(401, 402), None, None], [(402, 405), None, None]]
    rounded = np.zeros(n, dtype=bool)
    for part in plan:
        live = [(s, r) for s, r in enumerate(part) if r]
        pick = np.concatenate([np.arange(offs[s] + a, offs[s] + b) for s, (a, b) in live])
        ctx = _ctx([b - a for _, (a, b) in live], [a for _, (a, _) in live], [slots[s] for s, _ in live])
        got[pick] = _ssd_run(proj[pick], ctx, w, state, ring, H, dv, N, G, dtype)
        rounded[pick] = _tensor_cores(dtype, N, dv) and not ctx.all_single
    st, rg = state.cpu().numpy(), ring.cpu().numpy()
    for s in range(3):
        sl = slice(offs[s], offs[s + 1])
        want, S, u = _ssd_plain(proj[sl], w, H, dv, N, G, rounded[sl])
        assert np.abs(got[sl] - want).max() <= SSD_TOL[dtype] * np.abs(want).max(), s
        assert np.abs(st[slots[s], :H * N * dv].reshape(H, N, dv) - S).max() <= SSD_TOL[dtype] * np.abs(S).max()
        for p in range(max(0, lens[s] - taps), lens[s]):
            assert np.array_equal(rg[slots[s], (p % taps) * row:(p % taps) * row + ch], u[p].astype(np.float32)), (s, p)
    assert np.all(st[1] == 0) and np.all(rg[1] == 0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ["gone at once", "never", "steep and flat heads"])
def test_decays_at_their_ends(case, dtype):
    """Decays that leave nothing of the row before (logarithms of hundreds a row, sums of tens of thousands a chunk: a small
    difference of two such sums must not lose its digits), decays close to one (a row three hundred back still shows),
    and both in one launch; and steps that do not follow each other in size."""
    import torch
    rng = np.random.default_rng(1)
    H, dv, N, G, taps, T = 4, 16, 32 if dtype == "bfloat16" else 24, 2, 4, 330
    proj, w = _ssd_inputs(rng, T, H, dv, N, G, taps)
    w["a_log"] = {"gone at once": np.full(H, 4.6), "never": np.full(H, -12.0), "steep and flat heads": np.array([4.6, -12.0, 3.0, -3.0])}[case]
    w["dt_bias"] = np.full(H, 3.0 if case != "never" else -1.0)
    if case == "steep and flat heads":
        # long runs of tiny steps between large ones: within a run little decays, although the chunk's sum is large
        dt = proj[:, -H:]
        dt[:] = np.where((np.arange(T) % 40 < 6)[:, None], 4.0, -14.0) + 0.3 * dt
        w["dt_bias"][:] = 0.0
    want, _, _ = _ssd_plain(proj, w, H, dv, N, G, np.full(T, dtype == "bfloat16"))
    for cuts in ([(0, T)], [(0, 10), (10, 12), (12, 329), (329, T)]):
        state, ring = torch.zeros((1, H * N * dv), device="cuda"), torch.zeros((1, taps * (H * dv + 2 * G * N)), device="cuda")
        got = np.concatenate([_ssd_run(proj[a:b], _ctx([b - a], [a]), w, state, ring, H, dv, N, G, dtype) for a, b in cuts])
        assert np.isfinite(got).all()
        tol = SSD_TOL[dtype] if len(cuts) == 1 or dtype == "float32" else 1e-2        # a portion of one row rounds nothing
        assert np.abs(got - want).max() <= tol * np.abs(want).max(), cuts
    if case == "never":
        other = proj.copy()
        other[9, H * dv:2 * H * dv] += 40.0                     # the probe tells: a change of row 9 shows in the last rows
        assert np.abs(_ssd_plain(other, w, H, dv, N, G)[0][300:] - want[300:]).max() > 1e-2 * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("parts,width", [(1, 64), (4, 96), (6, 30), (2, 4096), (3, 3 * 700), (1, 9001), (16, 16)])
def test_norm_in_parts(parts, width, dtype):
    import torch
    from kllm_b200 import kernels
    rng = np.random.default_rng(width)
    y, gain = rng.standard_normal((5, width)) * np.exp(rng.uniform(-3, 3, (5, 1))), 1 + 0.2 * rng.standard_normal(width)
    y[1, :width // parts] = 0.0                                 # a part of zeros stays zero
    out = torch.empty((5, width + 8), dtype=getattr(torch, dtype), device="cuda")
    kernels.part_norm(out[:, :width], _t(y), _t(gain), parts, 1e-5)
    want = P.unit_rms(y.reshape(5, parts, -1), 1e-5).reshape(5, width) * gain
    assert np.abs(out[:, :width].float().cpu().numpy() - want).max() <= (1e-5 if dtype == "float32" else 6e-3) * np.abs(want).max()


# ---- norms ---------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d", [64, 50, 1, 2048, 5000, 8196])
def test_layer_norm_joins_the_stream_and_norms_the_embedding(d, dtype):
    """x += norm(y) * w * scale with the updated rows in the model dtype; the norm of an embedding's rows (ids, also one that is
    still on the device); rows whose mean is far from zero."""
    import torch
    from kllm_b200.parts.norm import LayerNorm
    from kllm_b200.parts.spec import BuildEnv, PartSpec
    rng = np.random.default_rng(d)
    td, eps, n, V = getattr(torch, dtype), 1e-5, 7, 11
    part = LayerNorm(PartSpec("layernorm", "", {"width": d, "eps": eps, "tensor": "w", "bias": False, "layer_scale": "s", "factor": 1.3}),
                     BuildEnv(dtype=td, device="cuda", hidden_size=d, max_position=16))
    assert sorted(t.name for t in part.tensor_specs()) == ["s", "w"]
    w, s = 1 + 0.2 * rng.standard_normal(d), 0.5 + 0.3 * rng.standard_normal(d)
    part.bind({"w": _t(w), "s": _t(s)})
    x, y = rng.standard_normal((n, d)) * 3, rng.standard_normal((n, d)) * 2 + 20.0 * np.arange(n)[:, None]
    xt = _t(x)
    rows = part.add_normed(xt, _t(y), then="rows")
    want = x + P.layer_norm(y, w * s * 1.3, eps)
    tol = 3e-5 if d > 1 else 1e-6
    assert np.abs(xt.cpu().numpy() - want).max() <= tol * np.abs(want).max()
    assert rows.dtype == td and torch.equal(rows, xt.to(td))
    xt = _t(x)
    assert part.add_normed(xt, _t(y)) is None
    assert np.abs(xt.cpu().numpy() - want).max() <= tol * np.abs(want).max()
    table = P.round_bf16(rng.standard_normal((V, d)) + 0.5)
    ids, last = np.array([3, 0, 10, -2, 3, -1, 5]), np.array([7, 9])
    ex, rows = part.embed(_t(table, dtype), _t(ids, "int32"), _t(last, "int32"), 2.0)
    real = np.where(ids < 0, last[np.clip(-ids - 1, 0, 1)], ids)
    want = P.layer_norm(table[real] * 2.0, w * s * 1.3, eps)
    assert np.abs(ex.cpu().numpy() - want).max() <= 1e-5 * max(1.0, np.abs(want).max())
    assert torch.equal(rows, ex.to(td))
    out = part.forward(_t(x), None, rows=_t([4, 1], "int32"))
    want = P.layer_norm(x[[4, 1]], w * s * 1.3, eps)
    assert np.abs(out.float().cpu().numpy() - want).max() <= (1e-5 if dtype == "float32" else 6e-3) * max(1.0, np.abs(want).max())


# ---- attention -----------------------------------------------------------------------------------

ATTN_SIZES = [(4, 2, 128, 128), (4, 2, 16, 24), (3, 1, 10, 6), (8, 2, 64, 64), (6, 3, 32, 48), (12, 12, 20, 20), (40, 2, 16, 16),
              (2, 1, 160, 160)]


# every pair of window and kept keys at four sizes, two of them at the others, the one beyond every tile's reach at two
ATTN_MASKS = [(40, 20), (130, 7), (1, 3), (64, 64), (100, 65), (299, 1), (17, 0), (40, 400)]
ATTN_CASES = [(m, z) for z in ATTN_SIZES[:4] for m in ATTN_MASKS] + [(m, z) for z in ATTN_SIZES[4:] for m in ATTN_MASKS[:2]] + \
    [((2100, 16), z) for z in (ATTN_SIZES[3], ATTN_SIZES[1])] + [((260, 100), ATTN_SIZES[3]), ((270, 10), ATTN_SIZES[0]), ((262, 30), ATTN_SIZES[1])]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mask,sizes", ATTN_CASES)
def test_window_edges_kept_keys_and_sinks(dtype, mask, sizes):
    """One key is made to stand out for every probed query: the first and the last kept key and the one behind it, the last key
    that the window still holds and the one before it, keys at page borders; in the rows of a prompt, in portions that start
    inside a page, in single tokens, in a mixed batch.  Pages that no query can see have no entry in the tables."""
    import torch
    from kllm_b200 import kernels
    (window, keep), (H, G, dk, dv) = mask, sizes
    long = window > 300
    rng = np.random.default_rng(H * 100 + dk + window)
    T, page, scale = (2400 if long else 380 if 256 < window < 290 else 300), 16, 0.5
    q, k = rng.standard_normal((T, H, dk)) * 0.2, rng.standard_normal((T, G, dk)) * 0.2
    v = rng.standard_normal((T, G, dv))
    probes = [T - 1, T - 2, T - 3, T - 4, T - 5, T - 6, T - 7, T - 60, T - 61, T - 62]
    for i, p in enumerate(probes):
        edge = p - window + 1                                  # the last key that the window holds
        kp = [0, keep - 1, keep, edge, edge - 1, 15, 16, edge, edge - 1, keep - 1][i]
        kp = min(max(kp, 0), p)
        u = rng.standard_normal(dk)
        u *= 5.0 / np.linalg.norm(u)
        hd = i % H
        q[p, hd] = u
        k[kp, hd // (H // G)] = u
        v[kp] += 4.0
    if dtype == "bfloat16":
        q, k, v = P.round_bf16(q), P.round_bf16(k), P.round_bf16(v)
    sinks = rng.standard_normal(H) * 2
    see = P.visible(np.arange(T), {"size": window, "keep_first": keep})
    rows_needed = np.arange(T) if not long else np.arange(T - 130, T)
    want = np.zeros((T, H * dv))
    want[rows_needed] = P.sink_attention(q[rows_needed], k, v, scale, see[rows_needed], sinks).reshape(-1, H * dv)
    n_pages = T // page + 6
    kc, vc, ids = _paged(k, v, page, n_pages, 3)
    kct, vct, qt = _t(np.nan_to_num(kc), dtype), _t(np.nan_to_num(vc), dtype), _t(q.reshape(T, H * dk), dtype)
    sk, tol = _t(sinks), 2e-5 if dtype == "float32" else 2e-2
    cases = [([107], [T - 107]), ([1, 1, 107], [T - 2, T - 61, T - 107]), ([1] * 10, probes)]
    if not long:
        cases = [([T], [0]), ([2, 60, 1], [T - 2, T - 62, T - 4])] + cases
    for n_new, start in cases:
        rows = np.concatenate([np.arange(s, s + c) for s, c in zip(start, n_new)])
        table = np.full((len(n_new), len(ids) + 2), -1, dtype=np.int32)
        for r, (s, c) in enumerate(zip(start, n_new)):
            seen = [j for j in range((s + c - 1) // page + 1) if see[s:s + c, j * page:(j + 1) * page].any()]
            table[r, seen] = ids[seen]
        out = torch.empty((len(rows), H * dv), dtype=qt.dtype, device="cuda")
        kernels.attention(out, qt[rows], kct, vct, _ctx(n_new, start), _t(table, "int32"), H, G, dk, window, scale, v_head_dim=dv,
                          exact_weights=True, sinks=sk, keep=keep)
        assert np.abs(out.float().cpu().numpy() - want[rows]).max() <= tol * np.abs(want).max(), n_new[:3]
    # the probe tells: one key more or less at either edge would show
    for other in ({"size": window + 1, "keep_first": keep}, {"size": window, "keep_first": keep + 1}):
        wrong = P.sink_attention(q[probes], k, v, scale, P.visible(np.arange(T), other)[probes], sinks).reshape(-1, H * dv)
        if not np.array_equal(P.visible(np.arange(T), other)[probes], see[probes]):
            assert np.abs(wrong - want[probes]).max() > 4 * tol * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,rot,factor", [(4, 2, 16, 24, 8, 3.0), (3, 3, 10, 6, 10, 0.5), (2, 1, 64, 32, 64, 8.0), (6, 2, 12, 12, 0, 1.0)])
def test_head_norms_stretched_rotation_and_cache_write(dtype, H, G, dk, dv, rot, factor):
    """Every head by its own root mean square, plain gains, then pairs (i, i + rot / 2) turned by frequencies that a factor
    divides, at positions far along; keys and values into shuffled pages."""
    import torch
    from kllm_b200 import kernels
    from kllm_b200.parts.rotary import rotary_frequencies
    rng = np.random.default_rng(H * dk)
    n_new, start = [5, 1, 9], [3, 100000, 0]
    ctx = _ctx(n_new, start)
    n, Q, K, V, page = sum(n_new), H * dk, G * dk, G * dv, 8
    qkv = rng.standard_normal((n, Q + K + V)) * 2
    table = np.full((3, 12501), -1, dtype=np.int32)
    table[0, 0], table[1, 12500], table[2, :2] = 3, 0, (2, 1)
    td = getattr(torch, dtype)
    kc, vc = torch.zeros((4, G, page, dk), dtype=td, device="cuda"), torch.zeros((4, G, page, dv), dtype=td, device="cuda")
    q_out = torch.empty((n, Q), dtype=td, device="cuda")
    r = {"dims": rot, "base": 300.0, "scaling": {"factor": factor}} if rot else None
    qg, kg, eps, freq = 1 + 0.3 * rng.standard_normal(dk), 1 + 0.3 * rng.standard_normal(dk), 1e-5, None
    if rot:
        freq, amp = rotary_frequencies(rot, 300.0, {"kind": "linear", "factor": factor})
        assert amp == 1.0 and np.allclose(freq.numpy(), P.frequencies(r), rtol=1e-13)
        freq = freq.cuda()
    kernels.headnorm_rope_append(q_out, _t(qkv), None, _t(qg), _t(kg), eps, freq, 1.0, rot, ctx.positions, ctx.token_req,
                                 _t(table, "int32"), kc, vc, H, G, G, dk, dv)
    pos, req = ctx.positions.cpu().numpy(), ctx.token_req.cpu().numpy()
    q = P.rotate(P.unit_rms(qkv[:, :Q].reshape(n, H, dk), eps) * qg, pos, r)
    k = P.rotate(P.unit_rms(qkv[:, Q:Q + K].reshape(n, G, dk), eps) * kg, pos, r)
    tol = 1e-5 if dtype == "float32" else 1e-2
    assert np.abs(q_out.float().cpu().numpy() - q.reshape(n, Q)).max() <= tol * np.abs(q).max()
    kcn, vcn = kc.float().cpu().numpy(), vc.float().cpu().numpy()
    for t in range(n):
        pg, sl = table[req[t], pos[t] // page], pos[t] % page
        assert np.abs(kcn[pg, :, sl] - k[t]).max() <= tol * np.abs(k).max()
        assert np.abs(vcn[pg, :, sl] - qkv[t, Q + K:].reshape(G, dv)).max() <= tol * np.abs(qkv).max()


# ---- feed-forwards --------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d,f,limit", [(1, 64, 96, 1.0), (3, 128, 160, 0.3), (8, 256, 128, 7.0), (13, 128, 64, 2.0), (40, 64, 72, 1.5),
                                         (5, 50, 22, 0.8), (1500, 128, 3072, 1.2)])
def test_clamped_gated_feed_forward(dtype, n, d, f, limit):
    """Values beyond the limit on every side, by the route that fits the rows (weights streamed, the tcgen05 product with the
    activation inside, or the library's products with a kernel behind them)."""
    import torch
    from kllm_b200 import kernels
    from kllm_b200.parts.mlp import GatedMLP
    from kllm_b200.parts.spec import BuildEnv, PartSpec
    if n > 1000:
        assert kernels.gemm_pays(n, f, "clamped")
    rng = np.random.default_rng(n)
    td = getattr(torch, dtype)
    part = GatedMLP(PartSpec("gated_mlp", "m", {"hidden": d, "intermediate": f, "activation": "clamped", "limit": limit, "alpha": 1.702,
                                                "tensors": {k: f"m.{k}" for k in ("gate", "up", "down")}}),
                    BuildEnv(dtype=td, device="cuda", hidden_size=d, max_position=16))
    w = {s.name: P.round_bf16(rng.standard_normal(s.shape) * 1.5 / np.sqrt(s.shape[1])) for s in part.tensor_specs()}
    part.bind({k: _t(v, dtype) for k, v in w.items()})
    h = P.round_bf16(rng.standard_normal((n, d)))
    want = P.dense_ff(h.astype(np.float64), w, "m", limit)
    assert (h @ w["m.gate"].T > limit).any() and (np.abs(h @ w["m.up"].T) > limit).any() or limit > 5
    tol = 1e-5 if dtype == "float32" else 1e-2
    y = part.forward(_t(h, dtype), None).float().cpu().numpy()
    assert np.abs(y - want).max() <= tol * np.abs(want).max()
    x = rng.standard_normal((n, d))
    xt = _t(x)
    part.forward_add(xt, _t(h, dtype), None)
    assert np.abs(xt.cpu().numpy() - x - want).max() <= tol * max(np.abs(want).max(), np.abs(x).max() * 0.1)


def _experts(dtype, d, E, I, top, f, shared, rng):
    import torch
    from kllm_b200.parts.moe import RoutedExperts
    from kllm_b200.parts.spec import BuildEnv, PartSpec
    part = RoutedExperts(PartSpec("routed_experts", "m", {
        "hidden": d, "experts": E, "identity": I, "top": top, "expert_ff": f, "activation": "relu2", "score": "softmax",
        "correction": "m.correction", "renormalize": True, "sum_eps": 1e-20, "weight_on": "output",
        "shared": {"ff": shared, "activation": "relu2", "tensors": {k: f"m.shared.{k}" for k in ("up", "down")}} if shared else None}),
        BuildEnv(dtype=getattr(torch, dtype), device="cuda", hidden_size=d, max_position=16))
    w = {}
    for s in part.tensor_specs():
        t = rng.standard_normal(s.shape)
        if s.name.endswith("correction"):
            t = rng.uniform(-0.5, 0.5, s.shape)
        elif s.name.endswith("router"):
            t = t * 2.0 / np.sqrt(d)
        else:
            t = t * 1.5 / np.sqrt(s.shape[1])
        w[s.name] = P.round_bf16(t)
    part.bind({k: _t(v, "float32" if k.endswith(("router", "correction")) else dtype) for k, v in w.items()})
    return part, w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d,E,I,top,f,shared", [(1, 64, 6, 3, 3, 40, 64), (5, 64, 4, 0, 1, 40, 0), (40, 64, 3, 2, 5, 24, 96), (20, 64, 8, 8, 2, 64, 32),
                                                  (7, 50, 2, 5, 4, 14, 9), (12, 128, 5, 1, 1, 128, 256), (700, 128, 4, 2, 3, 64, 128),
                                                  (300, 64, 1, 7, 2, 40, 0)])
def test_experts_without_gates_identity_experts_and_corrections(dtype, n, d, E, I, top, f, shared):
    """Choices by corrected scores, weights by the scores alone; identity experts between, beside and instead of the others;
    the expert that every token runs; steps that take the weight-streaming, the mma and the tcgen05 kernels."""
    from kllm_b200 import kernels
    rng = np.random.default_rng(n + E + I)
    part, w = _experts(dtype, d, E, I, top, f, shared, rng)
    h, x = P.round_bf16(rng.standard_normal((n, d))), rng.standard_normal((n, d))
    if n == 700:
        import torch
        assert kernels.moe_gemm_tcgen05_pays(_t(h, dtype), part.w_gate_up, n * top, True, False, "relu2") == (dtype == "bfloat16")
    m = {"router": {"experts": E, "identity": I, "top": top}, "shared": {"ff": shared} if shared else None}
    want = P.routed_ff(h.astype(np.float64), w, "m", m)
    idx, _ = P.route(h, w["m.router"], w["m.correction"], top)
    bare, _ = P.route(h, w["m.router"], np.zeros(E + I), top)
    if n > 5 and top < E + I:
        assert (np.sort(idx, axis=1) != np.sort(bare, axis=1)).any(), "the correction changed no choice"
    # a token whose choice is close falls where rounding puts it
    z = h.astype(np.float64) @ w["m.router"].T.astype(np.float64)
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s = np.sort(s / s.sum(axis=1, keepdims=True) + w["m.correction"], axis=1)[:, ::-1]
    clear = s[:, top - 1] - s[:, min(top, E + I - 1)] > 1e-6 if top < E + I else np.ones(n, bool)
    assert clear.mean() > 0.98
    tol = 1e-5 if dtype == "float32" else 1e-2
    y = part.forward(_t(h, dtype), None).cpu().numpy()
    assert np.abs(y - want)[clear].max() <= tol * np.abs(want).max()
    xt = _t(x)
    part.forward_add(xt, _t(h, dtype), None)
    assert np.abs(xt.cpu().numpy() - x - want)[clear].max() <= tol * np.abs(want).max()


def test_routing_weights_and_ties():
    """The weights are the chosen experts' scores over their sum, without the correction; among equal corrected scores the
    lower number goes first; a large correction forces a choice whose weight stays small."""
    from kllm_b200 import kernels
    rng = np.random.default_rng(3)
    n, d, E, top = 33, 40, 9, 4
    h, router, corr = rng.standard_normal((n, d)), rng.standard_normal((E, d)), np.zeros(E)
    corr[7] = 5.0
    idx, wt = kernels.moe_route(_t(h), _t(router), top, "softmax", True, correction=_t(corr), sum_eps=1e-20)
    pi, pw = P.route(h, router, corr, top)
    assert np.array_equal(idx.cpu().numpy(), pi) and np.all(pi[:, 0] == 7)
    assert np.abs(wt.cpu().numpy() - pw).max() <= 1e-5 and pw[:, 0].min() < 0.05
    zero = np.zeros((E, d))
    idx, wt = kernels.moe_route(_t(h), _t(zero), top, "softmax", True, correction=_t(np.zeros(E)))
    assert np.array_equal(idx.cpu().numpy(), np.tile(np.arange(top), (n, 1))) and np.allclose(wt.cpu().numpy(), 1 / top)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,k,N", [(1, 128, 50), (8, 256, 96), (16, 64, 40), (30, 50, 33), (1300, 256, 6656)])
def test_product_with_squared_relu(dtype, n, k, N):
    from kllm_b200 import kernels
    rng = np.random.default_rng(n)
    x, w = P.round_bf16(rng.standard_normal((n, k))), P.round_bf16(rng.standard_normal((N, k)) / np.sqrt(k))
    want = np.maximum(x.astype(np.float64) @ w.T, 0) ** 2
    assert n < 1000 or kernels.gemm_pays(n, N, "relu2")
    got = kernels.linear_relu2(_t(x, dtype), _t(w, dtype))
    assert got.dtype == _t(x, dtype).dtype
    assert np.abs(got.float().cpu().numpy() - want).max() <= (1e-5 if dtype == "float32" else 6e-3) * want.max()


# ---- configurations drawn at random ------------------------------------------------------------------

def _drawn(seed):
    """A configuration drawn at random: sizes in steps of 2 to 16, any order of layers, any mask."""
    rng = np.random.default_rng(2000 + seed)

    def pick(*xs):
        return xs[int(rng.integers(len(xs)))]
    step = pick(2, 4, 8, 16)

    def size(lo, hi):
        return max(step, int(rng.integers(lo, hi + 1)) // step * step)
    layers = []
    for _ in range(int(rng.integers(2, 6))):
        if rng.random() < 0.5:
            g = int(rng.integers(1, 4))
            heads, dv = g * int(rng.integers(1, 4)), size(4, 72)
            parts = pick(*[p for p in (1, 2, 3, 4, heads, g) if heads * dv % p == 0])
            layer = _mamba(heads, dv, size(4, 90), g, int(rng.integers(1, 7)), parts)
        else:
            g, dk = int(rng.integers(1, 4)), size(4, 100)
            rot = pick(None, (max(2, int(rng.integers(1, dk // 2 + 1)) * 2), float(rng.integers(10, 20000)), float(rng.uniform(0.5, 9))),
                       (dk // 2 * 2, 500.0))
            mask = pick(None, (int(rng.integers(1, 100)), int(rng.integers(0, 60))), (int(rng.integers(1, 30)), int(rng.integers(1, 20))))
            layer = _attn(g * int(rng.integers(1, 5)), g, dk, pick(dk, size(4, 100)), float(rng.uniform(0.1, 0.4)), mask, rot)
        kind = rng.random()
        if kind < 0.4:
            layer = _dense(layer, size(8, 120), float(rng.uniform(0.5, 6)))
        elif kind < 0.85:
            e, i = int(rng.integers(1, 9)), int(rng.integers(0, 5))
            layer = _moe(layer, e, int(rng.integers(1, e + i + 1)), size(4, 64), i, pick(None, size(4, 80)))
        else:
            layer = _alone(layer)
        layers.append(layer)
    return _cfg(int(rng.integers(30, 200)), size(16, 160), pick(1e-6, 1e-5), float(rng.uniform(0.2, 3)), layers), rng


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(14))
def test_configurations_drawn_at_random(tmp_path, seed, dtype):
    """Whole, cut, decoded and two in a batch."""
    from kllm_b200.engine.step import StepEntry
    cfg, rng = _drawn(seed)
    if dtype == "bfloat16":
        cfg = every_expert(cfg)
    w = P.random_weights(cfg, seed, qk_gain=1.5 if dtype == "float32" else 1.0)
    d = write(tmp_path / "drawn", cfg, w)
    a, b = (rng.integers(0, cfg["vocab"], size=n).tolist() for n in (140, 33))
    want_a, want_b = P.forward(w, cfg, a), P.forward(w, cfg, b)
    eng = engine_for(d, dtype, block_size=8, num_blocks=64)
    try:
        check_rows(run_cut(eng, a, [140]), want_a, dtype, "whole")
        check_rows(run_cut(eng, a, [70, 2, 1, 1, 40, 1]), want_a, dtype, "cut")
        ca, cb = eng.cache.open(), eng.cache.open()
        got_a, got_b = [], []
        for n, m in ((100, 1), (1, 20), (38, 11), (1, 1)):
            pa, pb = sum(len(x) for x in got_a), sum(len(x) for x in got_b)
            lg = eng.runner.run([StepEntry(cb, b[pb:pb + m], list(range(m))), StepEntry(ca, a[pa:pa + n], list(range(n)))])
            lg = lg.float().cpu().numpy().copy()
            got_b.append(lg[:m])
            got_a.append(lg[m:])
        check_rows(np.concatenate(got_a), want_a, dtype, "first of two")
        check_rows(np.concatenate(got_b), want_b, dtype, "second of two")
    finally:
        eng.close()
