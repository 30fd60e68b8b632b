"""The Dirarax design in the engine against its plain implementation (tests/plain/dirarax_plain.py).

Small configurations of their own, random weights whose values are bfloat16 numbers (so both
dtypes load the same model): each mechanism's kernel alone, whole prompts, prompts against
token-by-token decoding, portions down to two tokens, unequal batches, slots and pages that
are used again, keys far away, at page borders and at chunk edges that one score makes stand out,
the first tokens, long decoding through CUDA graphs, and greedy generation through the scheduler.
"""
import copy

import numpy as np
import pytest

from helpers import write_model_dir
from plain import dirarax_plain as P
from test_gpu_sozarax import _ctx, _paged, _t, check_rows, engine_for, run_cut

pytestmark = pytest.mark.gpu


def _gla(heads, dim, vdim, tau):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def _parallel(left, right, left_scale, right_scale):
    """left: heads, kv_heads, dim, vdim, scale, rot or None; right: dim, vdim, decay list, rot or None."""
    h, g, dk, dv, scale, rot = left
    a = {"heads": h, "kv_heads": g, "dim": dk, "vdim": dv, "scale": scale}
    if rot:
        a["rot"] = rot
    dim, vdim, decay, rrot = right
    r = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay}
    if rrot:
        r["rot"] = rrot
    return {"type": "parallel", "mixer": {"left": a, "right": r, "left_scale": left_scale, "right_scale": right_scale}}


def _rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def _dense(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def _moe(layer, experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return dict(layer, mlp=m)


def _alone(layer):
    return dict(layer, mlp=None)


# A: sizes that suit vector widths.  Layers before, inside and behind the loop, three passes; a parallel layer inside it (pages
# and states of its own in every pass); stretched and plain rotations, of part of a head and of all of it; all
# kinds of feed-forward, experts with and without the one that every token runs; a decay of exactly 1.
CFG_A = {
    "architecture": "Dirarax", "vocab": 96, "width": 64, "norm": {"eps": 1e-5},
    "layers": [
        _dense(_parallel((4, 2, 16, 24, 0.3, _rot(8, 1000.0, (4.0, 32, 8.0, 1.0))),
                         (16, 8, [0.5, 0.93, 1.0], _rot(16, 100.0)), 0.7, 1.3), 72),
        _moe(_gla(3, 16, 24, 4.0), 5, 2, 24, 40),
        _alone(_parallel((6, 1, 8, 8, 0.5, _rot(8, 50.0)), (24, 40, [0.8, 0.99], _rot(8, 5000.0)), 1.0, -0.5)),
        _moe(_gla(2, 40, 16, 16.0), 4, 1, 32),
        _dense(_gla(5, 8, 12, 1.0), 48),
    ],
    "loop": {"start": 1, "stop": 3, "times": 3},
}
# B: sizes that fit no vector width or tile; one head; no rotation; as many experts as are chosen; a loop that
# begins with the first layer and ends with the last, values wider and narrower than keys.
CFG_B = {
    "architecture": "Dirarax", "vocab": 61, "width": 50, "norm": {"eps": 1e-6},
    "layers": [
        _moe(_parallel((3, 3, 10, 6, 0.4, None), (7, 5, [0.9], None), 0.25, 2.0), 3, 3, 14, 9),
        _dense(_gla(1, 30, 7, 2.5), 22),
        _alone(_gla(3, 5, 21, 0.5)),
        _dense(_parallel((2, 1, 6, 9, 0.6, _rot(2, 10.0, (2.0, 16, 4.0, 0.5))), (6, 11, [0.7, 0.97], _rot(4, 30.0)), 1.5, 1.0), 13),
    ],
    "loop": {"start": 0, "stop": 4, "times": 2},
}
# C: head sizes of the tensor-core attention with values narrower and wider than keys and of the same size, wide recurrent heads
# (more than one slice of value channels), a rank of the decay that is no multiple of 8; no loop.
CFG_C = {
    "architecture": "Dirarax", "vocab": 80, "width": 128, "norm": {"eps": 1e-6},
    "layers": [
        _moe(_parallel((4, 2, 64, 128, 0.125, _rot(64, 10000.0, (8.0, 64, 32.0, 1.0))),
                       (64, 96, [0.9, 0.999], _rot(32, 10000.0)), 0.8, 0.9), 6, 3, 32, 64),
        _dense(_gla(2, 128, 192, 16.0), 96),
        _dense(_parallel((4, 4, 32, 64, 0.2, _rot(16, 500.0)), (130, 20, [0.95], _rot(130, 1000.0)), 1.2, 0.4), 160),
        _moe(_parallel((6, 2, 48, 48, 0.15, _rot(48, 2000.0)), (32, 16, [0.6, 0.7, 0.8], _rot(32, 100.0)), 0.5, 0.5), 8, 2, 64, 32),
    ],
}
# D: sizes in steps of 16 as a small served model has them; a loop of one pass over one layer.
CFG_D = {
    "architecture": "Dirarax", "vocab": 160, "width": 192, "norm": {"eps": 1e-6},
    "layers": [
        _moe(_gla(6, 16, 32, 8.0), 6, 2, 48, 96),
        _dense(_gla(3, 64, 48, 16.0), 256),
        _moe(_parallel((6, 3, 32, 48, 0.17, _rot(32, 20000.0, (4.0, 128, 16.0, 1.0))),
                       (48, 64, [0.97, 0.98, 0.99], _rot(32, 20000.0)), 0.9, 0.7), 4, 2, 64, 48),
        _moe(_gla(3, 48, 64, 16.0), 5, 3, 32, 64),
    ],
    "loop": {"start": 1, "stop": 2, "times": 1},
}
CFGS = {"A": (CFG_A, 61, 6), "B": (CFG_B, 62, 5), "C": (CFG_C, 63, 13), "D": (CFG_D, 64, 16)}       # configuration, seed, rank


def make_model(tmp_path, name, qk_boost=2.0, every_expert=False):
    """``every_expert``: all experts are chosen, so that in bfloat16 no close call of a router, which rounding may turn the
    other way and the states then carry on, stands between two runs."""
    cfg, seed, rank = CFGS[name]
    if every_expert:
        cfg = copy.deepcopy(cfg)
        for L in cfg["layers"]:
            if L["mlp"] and L["mlp"]["kind"] == "moe":
                L["mlp"]["router"]["top"] = L["mlp"]["router"]["experts"]
    w = P.random_weights(cfg, seed, qk_boost=qk_boost, rank=rank)
    d = write_model_dir(str(tmp_path / f"dirarax_{name}"), cfg, {k: np.asarray(v, dtype=np.float32) for k, v in w.items()})
    return cfg, w, d


# ---- whole models --------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole_prompt_and_every_way_of_cutting(tmp_path, name, dtype):
    cfg, w, d = make_model(tmp_path, name, 2.0 if dtype == "float32" else 1.0)
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
        for i, (g, t) in enumerate(zip(got_taps, layers)):      # the residual stream after every layer run
            err = np.abs(g - t).max(axis=-1) / np.abs(t).max()
            bound = 1e-4 if dtype == "float32" else 1e-1
            # in bfloat16 a row whose router meets a close call may choose another expert
            assert (err > bound).sum() <= (0 if dtype == "float32" else len(err) // 10), (name, i, err.max())
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
                assert np.abs(got - whole).max() <= 3e-5 * np.abs(want).max(), cuts
    finally:
        eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "D"])
def test_unequal_batches_and_reuse_of_slots_and_pages(tmp_path, name, dtype):
    """Four requests of unequal length in one batch, portions of some beside single tokens of
    others, then new requests in the slots and pages that the finished ones gave back; a pool
    that holds little more than what is live.  Every request also runs alone."""
    from kllm_b200.engine.step import StepEntry
    cfg, w, d = make_model(tmp_path, name, 2.0 if dtype == "float32" else 1.0, every_expert=dtype == "bfloat16")
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


def test_long_decoding(tmp_path):
    """A short prompt and then hundreds of single tokens: the decode route (graphs, pages added one by one, states
    carried through hundreds of steps)."""
    cfg, w, d = make_model(tmp_path, "A")
    rng = np.random.default_rng(3)
    ids = rng.integers(0, cfg["vocab"], size=420).tolist()
    want = P.forward(w, cfg, ids)
    eng = engine_for(d, "float32", max_seq=448, num_blocks=30)
    try:
        check_rows(run_cut(eng, ids, [9, 1]), want, "float32", "long decoding")
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
    cfg, w, d = make_model(tmp_path, name, 1.0, every_expert=name == "A")
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


# ---- each mechanism's kernel alone ----------------------------------------------------------------

def _run_gla(rows, ctx, state, heads, dk, dv, gain, eps, dtype, **kw):
    """The kernel on numpy rows q, k, v, g (, low), laid side by side as a product would leave them."""
    import torch
    from kllm_b200 import kernels
    parts = [rows[n] for n in ("q", "k", "v", "g", "low") if n in rows]
    proj = _t(np.concatenate(parts, axis=1))
    cols, off = [], 0
    for p in parts:
        cols.append(proj[:, off:off + p.shape[1]])
        off += p.shape[1]
    y = torch.empty((proj.shape[0], heads * dv + 8), dtype=getattr(torch, dtype), device="cuda")
    if "low" in rows:
        kw["low"] = cols[4]
    kernels.gla(y[:, :heads * dv], *cols[:4], state, ctx, heads, dk, dv, _t(gain), eps, **kw)
    return y[:, :heads * dv].float().cpu().numpy()


def _normed(o, g, gain, eps):
    n = o.shape[0]
    return (P.unit_rms(o, eps).reshape(n, -1) * gain) * P.silu(g)


GLA_SIZES = [(2, 16, 16), (3, 24, 40), (1, 64, 96), (2, 128, 128), (1, 7, 5), (2, 36, 66), (1, 256, 320), (4, 32, 64), (2, 130, 8)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dk,dv", GLA_SIZES)
def test_gated_decay_scan_carries_its_state(heads, dk, dv, dtype):
    """Three requests of unequal length in one launch (several chunks, one short chunk, one row), then portions that start
    from the slots at odd places, then a step of one row each, in slots 3, 0 and 2, against the plain
    token-by-token scan over each whole sequence; the states left in the slots too, and an untouched slot."""
    import torch
    rng = np.random.default_rng(dk + dv)
    R, tau, eps = 6, 3.0, 1e-5
    lens = [201, 30, 6]
    A, B, n = heads * dk, heads * dv, sum(lens)
    rows = {"q": rng.standard_normal((n, A)), "k": rng.standard_normal((n, A)), "v": rng.standard_normal((n, B)),
            "g": rng.standard_normal((n, B)) * 2, "low": rng.standard_normal((n, R))}
    w2, bias = P.round_bf16(rng.standard_normal((A, R))), rng.uniform(-3, 5, A)
    gain = 1 + 0.2 * rng.standard_normal(B)
    state = torch.zeros((4, heads * dk * dv + 4), device="cuda")
    slots, offs = [3, 0, 2], np.concatenate([[0], np.cumsum(lens)])
    got = np.zeros((n, B))
    # (first, last) rows of each request per launch
    plan = [[(0, 130), (0, 9), (0, 1)], [(130, 132), (9, 27), (1, 4)], [(132, 133), (27, 28), (4, 5)],
            [(133, 200), (28, 29), None], [(200, 201), (29, 30), (5, 6)]]
    kw = dict(w2=_t(w2, dtype), w2_bias=_t(bias), tau=tau, q_scale=dk ** -0.5)
    for part in plan:
        live = [(s, r) for s, r in enumerate(part) if r]
        pick = np.concatenate([np.arange(offs[s] + a, offs[s] + b) for s, (a, b) in live])
        ctx = _ctx([b - a for _, (a, b) in live], [a for _, (a, _) in live], [slots[s] for s, _ in live])
        got[pick] = _run_gla({k: v[pick] for k, v in rows.items()}, ctx, state, heads, dk, dv, gain, eps, dtype, **kw)
    st = state.cpu().numpy()
    alpha = P.sigmoid(rows["low"] @ w2.T.astype(np.float64) + bias).reshape(n, heads, dk) ** (1 / tau)
    tol = 3e-5 if dtype == "float32" else 1e-2
    for s in range(3):
        sl = slice(offs[s], offs[s + 1])
        o, S = P.decayed_scan(rows["q"][sl].reshape(-1, heads, dk) * dk ** -0.5, rows["k"][sl].reshape(-1, heads, dk),
                              rows["v"][sl].reshape(-1, heads, dv), alpha[sl])
        want = _normed(o, rows["g"][sl], gain, eps)
        assert np.abs(got[sl] - want).max() <= tol * np.abs(want).max(), s
        assert np.abs(st[slots[s], :heads * dk * dv].reshape(heads, dk, dv) - S).max() <= 3e-5 * np.abs(S).max()
    assert np.all(st[1] == 0)


@pytest.mark.parametrize("heads,dk,dv,rot", [(3, 16, 24, 16), (2, 64, 32, 64), (1, 30, 7, 12), (2, 128, 96, 64), (4, 8, 8, 0)])
def test_fixed_decay_scan_rotates_and_carries_its_state(heads, dk, dv, rot):
    """The fixed decay per head (one of them exactly 1) over rotated queries and keys at positions that do not start
    at 0, in chunks and single rows."""
    import torch
    rng = np.random.default_rng(heads * dk)
    T, eps, base = 170, 1e-6, 100.0
    decay = np.linspace(0.7, 1.0, heads) if heads > 1 else np.array([1.0])
    rows = {"q": rng.standard_normal((T, heads * dk)), "k": rng.standard_normal((T, heads * dk)),
            "v": rng.standard_normal((T, heads * dv)), "g": rng.standard_normal((T, heads * dv))}
    gain = np.full(heads * dv, 1.7)
    state = torch.zeros((2, heads * dk * dv), device="cuda")
    freq = _t(base ** (-2.0 * np.arange(rot // 2) / max(rot, 1)), "float64") if rot else None
    got = []
    for a, b in ((0, 67), (67, 68), (68, 69), (69, 71), (71, 170)):
        got.append(_run_gla({k: v[a:b] for k, v in rows.items()}, _ctx([b - a], [a], [1]), state, heads, dk, dv, gain, eps,
                            "float32", decay=_t(decay), freq=freq, k_scale=dk ** -0.5))
    r = {"dims": rot, "base": base} if rot else None
    q = P.rotate(rows["q"].reshape(T, heads, dk), np.arange(T), r, False)
    k = P.rotate(rows["k"].reshape(T, heads, dk), np.arange(T), r, False) * dk ** -0.5
    o, _ = P.decayed_scan(q, k, rows["v"].reshape(T, heads, dv), np.broadcast_to(decay[None, :, None], (T, heads, dk)))
    want = _normed(o, rows["g"], gain, eps)
    assert np.abs(np.concatenate(got) - want).max() <= 3e-5 * np.abs(want).max()


@pytest.mark.parametrize("case", ["gone at once", "never", "mixed"])
def test_decays_at_their_ends(case):
    """Decays that reach zero within a row (logits of -400 at tau 1: nothing of the past may be left, and nothing may
    turn into a NaN), decays of one (a key three hundred rows back shows undiminished), and both in one head."""
    import torch
    rng = np.random.default_rng(1)
    heads, dk, dv, T, eps = 2, 16, 24, 330, 1e-6
    z = {"gone at once": np.full(dk, -400.0), "never": np.full(dk, 60.0),
         "mixed": np.where(np.arange(dk) % 2 == 0, -400.0, 60.0)}[case]
    rows = {"q": rng.standard_normal((T, heads * dk)), "k": rng.standard_normal((T, heads * dk)) * 0.05,
            "v": rng.standard_normal((T, heads * dv)), "g": np.full((T, heads * dv), 3.0), "low": np.zeros((T, 4))}
    rows["k"][9] *= 400.0                        # one key that stands out, in the first chunk
    bias, gain = np.tile(z, heads), np.ones(heads * dv)
    alpha = np.broadcast_to(P.sigmoid(bias).reshape(1, heads, dk), (T, heads, dk))
    o, _ = P.decayed_scan(rows["q"].reshape(T, heads, dk), rows["k"].reshape(T, heads, dk), rows["v"].reshape(T, heads, dv), alpha)
    want = _normed(o, rows["g"], gain, eps)
    for cuts in ([(0, T)], [(0, 10), (10, 12), (12, 329), (329, T)]):
        state = torch.zeros((1, heads * dk * dv), device="cuda")
        got = np.concatenate([_run_gla({k: v[a:b] for k, v in rows.items()}, _ctx([b - a], [a]), state, heads, dk, dv, gain, eps,
                                       "float32", w2=_t(np.ones((heads * dk, 4))), w2_bias=_t(bias), tau=1.0) for a, b in cuts])
        assert np.isfinite(got).all()
        assert np.abs(got - want).max() <= 3e-5 * np.abs(want).max(), cuts
    if case == "never":
        # the probe tells: without that key the last rows would differ
        rows["k"][9] /= 400.0
        o2, _ = P.decayed_scan(rows["q"].reshape(T, heads, dk), rows["k"].reshape(T, heads, dk), rows["v"].reshape(T, heads, dv), alpha)
        assert np.abs(_normed(o2, rows["g"], gain, eps)[300:] - want[300:]).max() > 0.3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d", [64, 50, 2048, 5000, 4])
def test_norm_and_token_shift(d, dtype):
    """Norm with the shift towards the row before: requests of unequal length, one row and several, in slots 2, 0 and
    1 over three launches; the first row of a request sees zeros, the first row of a portion what the slot keeps."""
    import torch
    from kllm_b200 import kernels
    rng = np.random.default_rng(d)
    lens, slots, eps = [9, 4, 3], [2, 0, 1], 1e-5
    offs = np.concatenate([[0], np.cumsum(lens)])
    x, gain, mu = rng.standard_normal((sum(lens), d)) * 3, 1 + 0.2 * rng.standard_normal(d), rng.uniform(0, 1, d)
    state = torch.zeros((3, -(-d // 4) * 4), device="cuda")
    h, hs = np.zeros_like(x), np.zeros_like(x)
    for part in ([(0, 5), (0, 1), None], [(5, 6), (1, 2), (0, 1)], [(6, 9), (2, 4), (1, 3)]):
        live = [(s, r) for s, r in enumerate(part) if r]
        pick = np.concatenate([np.arange(offs[s] + a, offs[s] + b) for s, (a, b) in live])
        ctx = _ctx([b - a for _, (a, b) in live], [a for _, (a, _) in live], [slots[s] for s, _ in live])
        gh, ghs = kernels.norm_shift(_t(x[pick]), _t(gain), eps, _t(mu), state, ctx, getattr(torch, dtype))
        h[pick], hs[pick] = gh.float().cpu().numpy(), ghs.float().cpu().numpy()
    tol = 1e-5 if dtype == "float32" else 6e-3
    for s in range(3):
        sl = slice(offs[s], offs[s + 1])
        want = P.unit_rms(x[sl], eps) * gain
        assert np.abs(h[sl] - want).max() <= tol * np.abs(want).max()
        assert np.abs(hs[sl] - P.token_shift(want, mu)).max() <= tol * np.abs(want).max(), s
        assert np.abs(state[slots[s], :d].cpu().numpy() - want[-1]).max() <= 1e-5 * np.abs(want).max()


def test_norm_and_token_shift_over_many_rows():
    """A launch of more rows than one per CTA: rows whose neighbour another CTA has, beside request borders."""
    import torch
    from kllm_b200 import kernels
    rng = np.random.default_rng(0)
    lens, d, eps = [700, 1, 2, 600], 96, 1e-6
    x, gain, mu = rng.standard_normal((sum(lens), d)), 1 + 0.2 * rng.standard_normal(d), rng.uniform(0, 1, d)
    state = torch.zeros((4, d), device="cuda")
    _, hs = kernels.norm_shift(_t(x), _t(gain), eps, _t(mu), state, _ctx(lens, [0] * 4), torch.float32)
    offs = np.concatenate([[0], np.cumsum(lens)])
    for s in range(4):
        sl = slice(offs[s], offs[s + 1])
        want = P.token_shift(P.unit_rms(x[sl], eps) * gain, mu)
        assert np.abs(hs[sl].cpu().numpy() - want).max() <= 1e-5 * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_stream_entry(dtype):
    import torch
    from kllm_b200 import kernels
    rng = np.random.default_rng(6)
    n, d = 7, 42
    x, row, x0 = rng.standard_normal((n, d)), rng.standard_normal(d), rng.standard_normal((n, d))
    for first in (True, False):
        xt, cat = _t(x), _t(np.concatenate([np.zeros((n, d)), x0], axis=1), dtype)
        kernels.stream_entry(cat, xt, _t(row), first)
        assert torch.equal(cat[:, :d], _t(x).to(cat.dtype)) and torch.equal(cat[:, d:], _t(x if first else x0).to(cat.dtype))
        assert torch.equal(xt, _t(np.broadcast_to(row, (n, d))))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d,f", [(1, 64, 96), (3, 128, 160), (8, 256, 128), (13, 128, 64), (40, 64, 72), (5, 50, 22)])
def test_biased_gelu_gated_feed_forward(dtype, n, d, f):
    """down(gelu_tanh(gate h + b) * (up h + b)) + b added into the stream, by the route that fits the rows (weights
    streamed, or the library's products with kernels for activation and bias)."""
    import torch
    from kllm_b200.parts.mlp import GatedMLP
    from kllm_b200.parts.spec import BuildEnv, PartSpec
    rng = np.random.default_rng(n)
    td = getattr(torch, dtype)
    part = GatedMLP(PartSpec("gated_mlp", "m", {"hidden": d, "intermediate": f, "activation": "gelu_tanh", "bias": True,
                                                "tensors": {k: f"m.{k}" for k in ("gate", "up", "down")}}),
                    BuildEnv(dtype=td, device="cuda", hidden_size=d, max_position=16))
    w = {}
    for s in part.tensor_specs():
        w[s.name] = P.round_bf16(rng.standard_normal(s.shape) * (0.2 if len(s.shape) == 2 else 0.7))
    part.bind({k: _t(v, dtype if v.ndim == 2 else "float32") for k, v in w.items()})
    h, x = P.round_bf16(rng.standard_normal((n, d))), rng.standard_normal((n, d))
    xt = _t(x)
    part.forward_add(xt, _t(h, dtype), None)
    want = x + P.dense_ff(h.astype(np.float64), w, "m")
    tol = 1e-5 if dtype == "float32" else 1e-2
    assert np.abs(xt.cpu().numpy() - want).max() <= tol * np.abs(want).max()
    y = part.forward(_t(h, dtype), None).cpu().numpy()
    assert np.abs(y - (want - x)).max() <= tol * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,E,top,shared", [(1, 6, 3, 64), (5, 4, 1, 0), (40, 3, 3, 96), (20, 8, 2, 32)])
def test_experts_weighted_by_the_softmax_over_the_chosen(dtype, n, E, top, shared):
    """Logits far apart (the unchosen ones must not matter, the largest must not overflow), the expert that every
    token runs, the sum added into the stream."""
    import torch
    from kllm_b200.parts.moe import RoutedExperts
    from kllm_b200.parts.spec import BuildEnv, PartSpec
    rng = np.random.default_rng(n + E)
    d, f = 64, 40
    part = RoutedExperts(PartSpec("routed_experts", "m", {
        "hidden": d, "experts": E, "top": top, "expert_ff": f, "score": "softmax", "renormalize": True, "weight_on": "output",
        "shared": {"ff": shared, "tensors": {k: f"m.shared.{k}" for k in ("gate", "up", "down")}} if shared else None}),
        BuildEnv(dtype=getattr(torch, dtype), device="cuda", hidden_size=d, max_position=16))
    w = {s.name: P.round_bf16(rng.standard_normal(s.shape) * (2.0 if s.name.endswith("router") else 0.2)) for s in part.tensor_specs()}
    part.bind({k: _t(v, "float32" if k.endswith("router") else dtype) for k, v in w.items()})
    h, x = P.round_bf16(rng.standard_normal((n, d))), rng.standard_normal((n, d))
    xt = _t(x)
    part.forward_add(xt, _t(h, dtype), None)
    m = {"router": {"experts": E, "top": top}, "shared": {"ff": shared} if shared else None}
    want = x + P.routed_ff(h.astype(np.float64), w, "m", m)
    tol = 1e-5 if dtype == "float32" else 1e-2
    assert np.abs(xt.cpu().numpy() - want).max() <= tol * np.abs(want).max()
    y = part.forward(_t(h, dtype), None).cpu().numpy()
    assert np.abs(y - (want - x)).max() <= tol * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,rot", [(4, 2, 16, 24, 8), (3, 3, 10, 6, 10), (2, 1, 64, 32, 64), (6, 2, 12, 12, 4)])
def test_interleaved_rotation_with_an_amplitude_and_cache_write(dtype, H, G, dk, dv, rot):
    """Pairs (2i, 2i + 1) turned by stretched frequencies, cos and sin times the amplitude (on the rotated values
    alone), keys and values into shuffled pages."""
    import torch
    from kllm_b200 import kernels
    from kllm_b200.parts.rotary import rotary_frequencies
    rng = np.random.default_rng(H * dk)
    n_new, start = [5, 1, 9], [3, 40, 0]
    ctx = _ctx(n_new, start)
    n = sum(n_new)
    Q, K, V = H * dk, G * dk, G * dv
    qkv = rng.standard_normal((n, Q + K + V)) * 2
    page, pages = 8, 12
    table = np.full((3, 6), -1, dtype=np.int32)
    perm = rng.permutation(pages)
    used = 0
    for s in range(3):
        need = -(-(start[s] + n_new[s]) // page)
        table[s, :need] = perm[used:used + need]
        used += need
    td = getattr(torch, dtype)
    kc = torch.zeros((pages, G, page, dk), dtype=td, device="cuda")
    vc = torch.zeros((pages, G, page, dv), dtype=td, device="cuda")
    q_out = torch.empty((n, Q), dtype=td, device="cuda")
    r = {"dims": rot, "base": 300.0, "scaling": {"factor": 4.0, "original": 24, "fast": 6.0, "slow": 0.7}}
    freq, amp = rotary_frequencies(rot, 300.0, dict(r["scaling"], kind="ramp"))
    f_plain, amp_plain = P.frequencies(r)
    assert np.allclose(freq.numpy(), f_plain, rtol=1e-12) and abs(amp - amp_plain) < 1e-12 and amp > 1.1
    kernels.headnorm_rope_append(q_out, _t(qkv), None, None, None, 0.0, freq.cuda(), amp, rot, ctx.positions, ctx.token_req,
                                 _t(table, "int32"), kc, vc, H, G, G, dk, dv, interleaved=True)
    pos = ctx.positions.cpu().numpy()
    q = P.rotate(qkv[:, :Q].reshape(n, H, dk), pos, r, True)
    k = P.rotate(qkv[:, Q:Q + K].reshape(n, G, dk), pos, r, True)
    tol = 1e-5 if dtype == "float32" else 1e-2
    assert np.abs(q_out.float().cpu().numpy() - q.reshape(n, Q)).max() <= tol * np.abs(q).max()
    req = ctx.token_req.cpu().numpy()
    kcn, vcn = kc.float().cpu().numpy(), vc.float().cpu().numpy()
    for t in range(n):
        pg, sl = table[req[t], pos[t] // page], pos[t] % page
        assert np.abs(kcn[pg, :, sl] - k[t]).max() <= tol * np.abs(k).max()
        assert np.abs(vcn[pg, :, sl] - qkv[t, Q + K:].reshape(G, dv)).max() <= tol * np.abs(qkv).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 128, 64), (4, 2, 16, 24), (3, 1, 10, 6), (8, 2, 64, 64), (6, 3, 32, 48), (2, 2, 32, 64)])
def test_gated_attention_far_keys_and_page_borders(dtype, H, G, dk, dv):
    """One key is made to stand out for every probed query, far back (the first key of all, the last key of a
    page, the first of the next) or near; rows of a prompt, a portion that starts inside a page, single tokens; then the
    gate with its factor."""
    import torch
    from kllm_b200 import kernels
    rng = np.random.default_rng(H * 100 + dk)
    T, page, scale = 300, 16, 0.5
    q, k = rng.standard_normal((T, H, dk)) * 0.2, rng.standard_normal((T, G, dk)) * 0.2
    v = rng.standard_normal((T, G, dv))
    for qp, kp in ((299, 0), (298, 15), (297, 16), (200, 63), (150, 150), (131, 130)):
        u = rng.standard_normal(dk)
        u *= 6.0 / np.linalg.norm(u)
        hd = int(rng.integers(0, H))
        q[qp, hd] = k[kp, hd // (H // G)] = u
        v[kp] += 5.0
    if dtype == "bfloat16":
        q, k, v = P.round_bf16(q), P.round_bf16(k), P.round_bf16(v)
    want = P.causal_attention(q, k, v, scale).reshape(T, H * dv)
    kc, vc, ids = _paged(k, v, page, 24, 3)
    table = np.full((1, 20), -1, dtype=np.int32)
    table[0, :len(ids)] = ids
    kct, vct, qt = _t(np.nan_to_num(kc), dtype), _t(np.nan_to_num(vc), dtype), _t(q.reshape(T, H * dk), dtype)
    tol = 2e-5 if dtype == "float32" else 2e-2
    for n_new, start, rows in (([T], [0], np.arange(T)),
                               ([1, 1, 107], [298, 131, 193], np.concatenate([[298], [131], np.arange(193, 300)])),
                               ([1] * 6, [299, 298, 297, 200, 150, 131], np.array([299, 298, 297, 200, 150, 131]))):
        out = torch.empty((len(rows), H * dv), dtype=qt.dtype, device="cuda")
        kernels.attention(out, qt[rows], kct, vct, _ctx(n_new, start), _t(np.repeat(table, len(n_new), axis=0), "int32"), H, G, dk,
                          0, scale, v_head_dim=dv, exact_weights=True)
        assert np.abs(out.float().cpu().numpy() - want[rows]).max() <= tol * np.abs(want).max(), n_new[:3]
    gate = rng.standard_normal((6, H * dv + 3)) * 2
    y = torch.empty((6, H * dv + 8), dtype=qt.dtype, device="cuda")
    kernels.sigmoid_gate(y[:, :H * dv], out, _t(gate)[:, 3:], factor=-0.6)
    gated = out.float().cpu().numpy() * P.sigmoid(gate[:, 3:]) * -0.6
    assert np.abs(y[:, :H * dv].float().cpu().numpy() - gated).max() <= (1e-6 if dtype == "float32" else 1e-2) * np.abs(gated).max()


def test_side_by_side_members_and_their_weights(tmp_path):
    """Each of the two mixers of a parallel layer, and each of their factors, counts: with one of them changed the plain
    implementation and the engine change alike."""
    cfg, w, _ = make_model(tmp_path, "C")
    rng = np.random.default_rng(1)
    ids = rng.integers(0, cfg["vocab"], size=70).tolist()
    base = P.forward(w, cfg, ids)
    for key, value in (("left_scale", 0.0), ("right_scale", 0.0), ("left_scale", -1.0)):
        c2 = copy.deepcopy(cfg)
        c2["layers"][0]["mixer"][key] = value
        want = P.forward(w, c2, ids)
        assert np.abs(want - base).max() > 1e-2 * np.abs(base).max(), key
        d = write_model_dir(str(tmp_path / f"side_{key}_{value}"), c2, {k: np.asarray(v_, dtype=np.float32) for k, v_ in w.items()})
        eng = engine_for(d, "float32")
        try:
            check_rows(run_cut(eng, ids, [23, 1, 40, 1]), want, "float32", key)
        finally:
            eng.close()


def test_passes_keep_states_of_their_own(tmp_path):
    """Three passes over the same weights, each with its own step vector: with one pass's vector changed, or the loop run
    once less, plain implementation and engine change alike."""
    cfg, w, _ = make_model(tmp_path, "A")
    rng = np.random.default_rng(2)
    ids = rng.integers(0, cfg["vocab"], size=60).tolist()
    base = P.forward(w, cfg, ids)
    w2 = dict(w)
    w2["loop.step"] = P.round_bf16(np.asarray(w["loop.step"]) * np.array([[1.0], [1.0], [-2.0]]))
    c3, w3 = copy.deepcopy(cfg), dict(w)
    c3["loop"]["times"] = 2
    w3["loop.step"] = w["loop.step"][:2]
    for i, (c, ww) in enumerate(((cfg, w2), (c3, w3))):
        want = P.forward(ww, c, ids)
        assert np.abs(want - base).max() > 1e-2 * np.abs(base).max()
        d = write_model_dir(str(tmp_path / f"pass_{i}"), c, {k: np.asarray(v_, dtype=np.float32) for k, v_ in ww.items()})
        eng = engine_for(d, "float32")
        try:
            check_rows(run_cut(eng, ids, [20, 1, 2, 30, 1]), want, "float32", f"passes {i}")
        finally:
            eng.close()


def _drawn(seed):
    """A configuration drawn at random: sizes in steps of 2 to 16, any order of layers, any loop."""
    rng = np.random.default_rng(1000 + seed)

    def pick(*xs):
        return xs[int(rng.integers(len(xs)))]
    step = pick(2, 4, 8, 16)

    def size(lo, hi):
        return max(step, int(rng.integers(lo, hi + 1)) // step * step)

    def rot(dim, scaled):
        dims = max(2, int(rng.integers(1, dim // 2 + 1)) * 2)
        return pick(_rot(dims, float(rng.integers(10, 20000)), (pick(2.0, 8.0), int(rng.integers(16, 100)), pick(8.0, 32.0), 1.0)
                         if scaled and rng.random() < 0.7 else None), _rot(dim // 2 * 2, 500.0))
    layers = []
    for _ in range(int(rng.integers(2, 5))):
        if rng.random() < 0.5:
            layer = _gla(int(rng.integers(1, 6)), size(4, 72), size(4, 90), float(rng.uniform(1, 16)))
        else:
            g, dk, dim = int(rng.integers(1, 4)), size(4, 80), size(4, 72)
            layer = _parallel((g * int(rng.integers(1, 4)), g, dk, size(4, 72), float(rng.uniform(0.1, 0.4)), rot(dk, True)),
                              (dim, size(4, 72), rng.uniform(0.6, 1.0, int(rng.integers(1, 5))).tolist(), rot(dim, False)),
                              float(rng.uniform(-1.5, 1.5)), float(rng.uniform(-1.5, 1.5)))
        kind = rng.random()
        if kind < 0.4:
            layer = _dense(layer, size(8, 120))
        elif kind < 0.85:
            e = int(rng.integers(1, 9))
            layer = _moe(layer, e, int(rng.integers(1, e + 1)), size(4, 64), pick(None, size(4, 80)))
        else:
            layer = _alone(layer)
        layers.append(layer)
    cfg = {"architecture": "Dirarax", "vocab": int(rng.integers(30, 200)), "width": size(16, 160), "norm": {"eps": pick(1e-6, 1e-5)},
           "layers": layers}
    if rng.random() < 0.75:
        a = int(rng.integers(0, len(layers)))
        cfg["loop"] = {"start": a, "stop": int(rng.integers(a + 1, len(layers) + 1)), "times": int(rng.integers(1, 4))}
    return cfg, int(rng.integers(1, 20)), rng


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(tmp_path, seed, dtype):
    """Whole, cut, decoded and two in a batch."""
    from kllm_b200.engine.step import StepEntry
    cfg, rank, rng = _drawn(seed)
    if dtype == "bfloat16":
        for L in cfg["layers"]:                          # no close call of a router between two runs (see make_model)
            if L["mlp"] and L["mlp"]["kind"] == "moe":
                L["mlp"]["router"]["top"] = L["mlp"]["router"]["experts"]
    w = P.random_weights(cfg, seed, rank=rank)
    d = write_model_dir(str(tmp_path / "drawn"), cfg, {k: np.asarray(v, dtype=np.float32) for k, v in w.items()})
    a, b = (rng.integers(0, cfg["vocab"], size=n).tolist() for n in (140, 33))
    want_a, want_b = P.forward(w, cfg, a), P.forward(w, cfg, b)
    eng = engine_for(d, dtype, block_size=8, num_blocks=64)
    try:
        check_rows(run_cut(eng, a, [140]), want_a, dtype, "whole")
        check_rows(run_cut(eng, a, [70, 2, 1, 1, 40, 1]), want_a, dtype, "cut")
        ca, cb = eng.cache.open(), eng.cache.open()
        got_a, got_b = [], []
        for n, m in ((100, 1), (1, 20), (38, 11), (1, 1)):
            pa, pb = len(np.concatenate(got_a)) if got_a else 0, len(np.concatenate(got_b)) if got_b else 0
            lg = eng.runner.run([StepEntry(cb, b[pb:pb + m], list(range(m))), StepEntry(ca, a[pa:pa + n], list(range(n)))])
            lg = lg.float().cpu().numpy().copy()
            got_b.append(lg[:m])
            got_a.append(lg[m:])
        check_rows(np.concatenate(got_a), want_a, dtype, "first of two")
        check_rows(np.concatenate(got_b), want_b, dtype, "second of two")
    finally:
        eng.close()
