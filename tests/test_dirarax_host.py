"""Host-side tests of the Dirarax design: configuration, the model's description (tensors, schedule,
cache needs) against the plain implementation's own list, the cache manager with named states, random
weights, and the plain recurrence cut in pieces."""
import copy

import numpy as np
import pytest

from plain import dirarax_plain as P
from test_gpu_dirarax import CFG_A, CFG_B, CFG_C, CFGS


def test_config_round_trip_and_refusals():
    import kllm_b200.models  # noqa: F401  (registers the architectures)
    from kllm_b200.config import ConfigError, parse_config
    for cfg, _, _ in CFGS.values():
        c = parse_config(cfg)
        assert parse_config(c.to_dict()) == c
        assert c.to_dict() == cfg
        assert c.layer_order() == P.layer_runs(cfg)

    def broken(path, value):
        c = copy.deepcopy(CFG_A)
        at = c
        for k in path[:-1]:
            at = at[k]
        if value is KeyError:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        return c
    left, right = ("layers", 0, "mixer", "left"), ("layers", 0, "mixer", "right")
    for path, value in ((("vocab",), KeyError), (("norm", "eps"), 0.0), (("layers",), []), (left + ("heads",), 3),
                        (left + ("kv_heads",), 0), (left + ("rot", "dims"), 3), (left + ("rot", "dims"), 18),
                        (left + ("rot", "scaling", "factor"), 0), (left + ("rot", "scaling", "fast"), KeyError),
                        (left + ("scale",), KeyError), (right + ("decay",), [0.5]), (right + ("decay",), [0.5, 0.5, 1.5]),
                        (right + ("decay",), [0.0, 0.5, 0.5]), (right + ("vdim",), 0), (("layers", 0, "mixer", "left_scale"), KeyError),
                        (("layers", 0, "type"), "wkv"), (("layers", 0, "mlp", "ff"), 0), (("layers", 0, "mlp", "kind"), "plain"),
                        (("layers", 1, "mixer", "tau"), 0.0), (("layers", 1, "mlp", "router", "top"), 6),
                        (("layers", 1, "mlp", "shared"), {"ff": 0}), (("loop", "stop"), 1), (("loop", "stop"), 6),
                        (("loop", "times"), 0), (("loop",), 3)):
        with pytest.raises(ConfigError):
            parse_config(broken(path, value))


@pytest.mark.parametrize("name", sorted(CFGS))
def test_model_description(name):
    import torch
    import kllm_b200.models  # noqa: F401
    from kllm_b200.config import build_model_spec, parse_config
    from kllm_b200.parts.model import DecoderModel
    from kllm_b200.parts.spec import PagedKVNeed, StateNeed
    cfg, _, rank = CFGS[name]
    model = DecoderModel(build_model_spec(parse_config(cfg)), torch.float32, "cpu")
    shapes = P.tensor_shapes(cfg, rank)
    specs = {s.name: s for s in model.tensor_specs()}
    assert set(specs) == set(shapes)
    for n, shape in shapes.items():
        assert specs[n].fits(shape), (n, specs[n].shape, shape)
        assert specs[n].store == ("compute" if len(shape) == 2 and not n.endswith((".router", ".step")) else "float32"), n
        assert not specs[n].optional
    # every run of a layer has a cache slot of its own; a pass begins with the mix of the embedding's output
    runs = P.layer_runs(cfg)
    assert [(c.block, c.cache, c.writes_cache, c.entry) for c in model.schedule] == \
        [(i, k, True, None if t is None else (0, t)) for k, (i, t) in enumerate(runs)]
    for need, (i, _) in zip(model.cache_needs(), runs):
        m = cfg["layers"][i]["mixer"]
        shift = StateNeed((-(-cfg["width"] // 4) * 4,), "float32", "shift")
        if cfg["layers"][i]["type"] == "gla":
            assert need == [StateNeed((m["heads"] * m["dim"] * m["vdim"],), "float32"), shift]
        else:
            a, r = m["left"], m["right"]
            assert need == [PagedKVNeed(a["kv_heads"], a["dim"], None, None if a["vdim"] == a["dim"] else a["vdim"]),
                            StateNeed((r["heads"] * r["dim"] * r["vdim"],), "float32"), shift]


def test_side_by_side_joins_its_members_matrices():
    """The stacked projections and the joined output matrix hold every member's rows and columns where the member
    looks for them."""
    import torch
    import kllm_b200.models  # noqa: F401
    from kllm_b200.config import build_model_spec, parse_config
    from kllm_b200.parts.model import DecoderModel
    model = DecoderModel(build_model_spec(parse_config(CFG_B)), torch.float32, "cpu")
    w = P.random_weights(CFG_B, 1, rank=16)
    model.bind({k: torch.from_numpy(np.asarray(v)) for k, v in w.items()})
    mixer = model.blocks[3].mixer
    x = torch.randn(4, CFG_B["width"])
    proj, row = x @ mixer.w_in.t(), 0
    left, right = mixer.members
    assert mixer.w_in.shape[0] % 8 == 0 and left.w_in.shape[0] % 8 == 0
    for member, names in ((left, "gqkv"), (right, "qkvg")):
        off = row
        for n in names:
            t = torch.from_numpy(np.asarray(w[f"l3.mix.{'left' if member is left else 'right'}.{n}"]))
            assert torch.allclose(proj[:, off:off + t.shape[0]], x @ t.t(), atol=1e-5), n
            off += t.shape[0]
        row += member.w_in.shape[0]
    assert torch.equal(mixer.w_out, torch.cat([torch.from_numpy(np.asarray(w[f"l3.mix.{s}.o"])) for s in ("left", "right")], dim=1))
    assert left.w_in.data_ptr() == mixer.w_in.data_ptr()


def test_cache_manager_names_states_apart():
    """Unnamed and named states of a layer, zeroed when their slot is used again; two of one name are refused."""
    import torch
    import kllm_b200.models  # noqa: F401
    from kllm_b200.cache.manager import CacheManager
    from kllm_b200.config import build_model_spec, parse_config
    from kllm_b200.parts.model import DecoderModel
    from kllm_b200.parts.spec import StateNeed
    model = DecoderModel(build_model_spec(parse_config(CFG_A)), torch.float32, "cpu")
    cm = CacheManager(model.cache_needs(), 16, 12, max_requests=2, dtype=torch.float32, device="cpu")
    assert len(cm.groups) == 2                       # the two kinds of parallel layer; recurrent layers hold no pages
    a = cm.open()
    cm.reserve(a, 40)
    views = cm.layer_caches({g: torch.zeros((1, 4), dtype=torch.int32) for g in range(2)})
    assert len(views) == len(model.schedule)
    for v in views:
        v.state[a.state_slot] = 7.0
        v.states["shift"][a.state_slot] = 5.0
    ptrs = [v.state.data_ptr() for v in views] + [v.states["shift"].data_ptr() for v in views]
    assert len(set(ptrs)) == len(ptrs)               # the passes share weights, not states
    cm.commit(a, 40)
    slot = a.state_slot
    cm.close(a)
    b = cm.open()
    assert b.state_slot == slot
    for v in views:
        assert not v.state[slot].any() and not v.states["shift"][slot].any()
    cm.audit()
    with pytest.raises(ValueError):
        CacheManager([[StateNeed((4,)), StateNeed((8,))]], 16, 1, max_requests=1)
    with pytest.raises(ValueError):
        CacheManager([[StateNeed((4,), name="s"), StateNeed((8,), name="s")]], 16, 1, max_requests=1)


def test_random_weights_mode(tmp_path):
    import torch
    from kllm_b200.weights import write_random_model
    from kllm_b200.weights.safetensors_io import ModelFiles
    d = write_random_model(str(tmp_path / "m"), CFG_C, seed=3, dtype=torch.bfloat16)
    shapes = P.tensor_shapes(CFG_C, 16)
    with ModelFiles(d) as f:
        assert set(f.names()) == set(shapes)
        for n in f.names():
            assert tuple(f.entry(n).shape) == tuple(shapes[n])
        # weights stored around zero (one-plus norms) start at zero, plain gains at one, shifts between zero and one
        assert float(f.read("l0.norm1").abs().max()) == 0.0
        assert float((f.read("l1.mix.norm") - 1).abs().max()) == 0.0
        s = f.read("l2.shift").float()
        assert 0.0 <= float(s.min()) < float(s.max()) <= 1.0


def test_plain_recurrence_and_shift_in_pieces():
    """The plain scan and the plain shift carried over a cut equal those over the whole (their state arguments are what the
    tests of the kernels compare the slots with)."""
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((20, 2, 5)), rng.standard_normal((20, 2, 5)), rng.standard_normal((20, 2, 3))
    alpha = rng.uniform(0, 1, (20, 2, 5))
    whole, S = P.decayed_scan(q, k, v, alpha)
    a, Sa = P.decayed_scan(q[:7], k[:7], v[:7], alpha[:7])
    b, Sb = P.decayed_scan(q[7:], k[7:], v[7:], alpha[7:], Sa)
    assert np.allclose(np.concatenate([a, b]), whole) and np.allclose(Sb, S)
    h, mu = rng.standard_normal((20, 5)), rng.uniform(0, 1, 5)
    assert np.allclose(np.concatenate([P.token_shift(h[:7], mu), P.token_shift(h[7:], mu, h[6])]), P.token_shift(h, mu))


def test_plain_rotations_keep_lengths():
    """A plain rotation keeps every pair's length whatever the layout, a stretched one scales the rotated values by its
    amplitude and leaves the rest."""
    rng = np.random.default_rng(2)
    x = rng.standard_normal((6, 2, 12))
    rot = {"dims": 8, "base": 100.0}
    for inter in (True, False):
        y = P.rotate(x, np.arange(6) * 7, rot, inter)
        pair = (lambda t: t[..., 0:8:2] ** 2 + t[..., 1:8:2] ** 2) if inter else (lambda t: t[..., :4] ** 2 + t[..., 4:8] ** 2)
        assert np.allclose(pair(y), pair(x)) and np.array_equal(y[..., 8:], x[..., 8:]) and not np.allclose(y[1:, :, :8], x[1:, :, :8])
    sc = dict(rot, scaling={"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0})
    y = P.rotate(x, np.arange(6), sc, True)
    assert np.allclose((y[..., :8] ** 2).sum(-1), (1 + 0.1 * np.log(3.0)) ** 2 * (x[..., :8] ** 2).sum(-1))
    assert np.array_equal(y[..., 8:], x[..., 8:])
