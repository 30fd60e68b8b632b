"""Host-side tests of the Rupenex design: configuration, the model's description (tensors, schedule,
cache needs) against the plain implementation's own list, the cache manager with first keys that stay beside a window, random
weights, and the plain recurrence cut in pieces."""
import copy

import numpy as np
import pytest

from plain import rupenex_plain as P
from test_gpu_rupenex import CFG_A, CFG_C, CFG_D, CFGS


def test_config_round_trip_and_refusals():
    import kllm_b200.models  # noqa: F401  (registers the architectures)
    from kllm_b200.config import ConfigError, parse_config
    for cfg, _ in CFGS.values():
        c = parse_config(cfg)
        assert parse_config(c.to_dict()) == c
        assert c.to_dict() == cfg

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
    attn, mamba, moe = ("layers", 0, "mixer"), ("layers", 1, "mixer"), ("layers", 0, "mlp")
    for path, value in ((("vocab",), KeyError), (("norm", "eps"), 0.0), (("layers",), []), (("logit_scale",), "2"),
                        (attn + ("heads",), 3), (attn + ("kv_heads",), 0), (attn + ("rot", "dims"), 3), (attn + ("rot", "dims"), 18),
                        (attn + ("rot", "scaling", "factor"), 0), (attn + ("rot", "scaling"), {}), (attn + ("scale",), KeyError),
                        (attn + ("mask", "size"), 0), (attn + ("mask", "keep_first"), -1), (attn + ("mask",), 5),
                        (mamba + ("groups",), 3), (mamba + ("norm_groups",), 5), (mamba + ("conv",), 0), (mamba + ("state",), KeyError),
                        (("layers", 0, "type"), "gla"), (("layers", 1, "mlp", "ff"), 0), (("layers", 1, "mlp", "limit"), 0.0),
                        (("layers", 1, "mlp", "limit"), KeyError), (("layers", 1, "mlp", "kind"), "plain"), (moe + ("router", "top"), 9),
                        (moe + ("router", "identity"), -1), (moe + ("shared",), {"ff": 0}), (moe + ("expert",), KeyError)):
        with pytest.raises(ConfigError):
            parse_config(broken(path, value))
    assert parse_config(broken(("logit_scale",), KeyError)).logit_scale == 1.0
    # all of what a router chooses among may be chosen, identity experts included
    assert parse_config(broken(moe + ("router", "top"), 8)).layers[0].mlp.top == 8


@pytest.mark.parametrize("name", sorted(CFGS))
def test_model_description(name):
    import torch
    import kllm_b200.models  # noqa: F401
    from kllm_b200.config import build_model_spec, parse_config
    from kllm_b200.parts.model import DecoderModel
    from kllm_b200.parts.spec import PagedKVNeed, StateNeed
    cfg, _ = CFGS[name]
    model = DecoderModel(build_model_spec(parse_config(cfg)), torch.float32, "cpu")
    shapes = P.tensor_shapes(cfg)
    specs = {s.name: s for s in model.tensor_specs()}
    assert set(specs) == set(shapes)
    for n, shape in shapes.items():
        assert specs[n].fits(shape), (n, specs[n].shape, shape)
        assert specs[n].store == ("compute" if len(shape) == 2 and not n.endswith((".router", ".conv")) else "float32"), n
        assert not specs[n].optional
    assert [(c.block, c.cache, c.writes_cache) for c in model.schedule] == [(i, i, True) for i in range(len(cfg["layers"]))]
    for need, L in zip(model.cache_needs(), cfg["layers"]):
        m = L["mixer"]
        if L["type"] == "mamba2":
            row = -(-(m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]) // 4) * 4
            assert need == [StateNeed((m["heads"] * m["state"] * m["vdim"],), "float32"), StateNeed((m["conv"] * row,), "float32", "conv")]
        else:
            mask = m.get("mask") or {}
            assert need == PagedKVNeed(m["kv_heads"], m["dim"], mask.get("size"), None if m["vdim"] == m["dim"] else m["vdim"],
                                       keep_first=mask.get("keep_first", 0))


def test_weights_that_act_once():
    """The layer scale and the logits' factor act on the norms' weights when they are bound, in float32."""
    import torch
    import kllm_b200.models  # noqa: F401
    from kllm_b200.config import build_model_spec, parse_config
    from kllm_b200.parts.model import DecoderModel
    model = DecoderModel(build_model_spec(parse_config(CFG_A)), torch.bfloat16, "cpu")
    w = P.random_weights(CFG_A, 1)
    specs = {s.name: s for s in model.tensor_specs()}
    model.bind({k: torch.from_numpy(np.asarray(v)).to(torch.bfloat16 if specs[k].store == "compute" else torch.float32) for k, v in w.items()})
    b = model.blocks[0]
    assert torch.equal(b.mixer_norm.gain, torch.from_numpy(w["l0.norm1"] * w["l0.ls1"])) and b.mixer_norm.gain.dtype == torch.float32
    assert torch.equal(b.ff_norm.gain, torch.from_numpy(w["l0.norm2"] * w["l0.ls2"]))
    assert torch.allclose(model.final_norm.gain, torch.from_numpy(w["final.norm"]) * CFG_A["logit_scale"])
    assert torch.equal(model.embedding.norm.gain, torch.from_numpy(w["embed.norm"]))
    assert b.feed_forward.w_gate_up.shape == (5, 24, 64) and b.feed_forward.router.shape == (8, 64)
    assert model.blocks[2].feed_forward is None and model.blocks[2].ff_norm is None


def test_cache_keeps_the_first_keys_beside_a_window():
    """Pages wholly behind the window come back at commit except those of the kept first keys; groups of different windows or
    kept counts are apart; what a request can ever need counts both; nothing is lost."""
    from kllm_b200.cache.manager import CacheManager
    from kllm_b200.parts.spec import PagedKVNeed
    needs = [PagedKVNeed(2, 8, 40, keep_first=20), PagedKVNeed(2, 8, 40), PagedKVNeed(2, 8, 40, keep_first=20), PagedKVNeed(2, 8),
             PagedKVNeed(2, 8, 8, keep_first=16)]
    cm = CacheManager(needs, 16, 30, max_requests=2, allocate=False)
    assert [g.slots for g in cm.groups] == [[0, 2], [1], [3], [4]]
    assert cm.pages_ever_needed(1000) == [2 + 4, 4, 63, 1 + 2] and cm.pages_ever_needed(20) == [2, 2, 2, 2]
    r = cm.open()
    for _ in range(20):
        cm.reserve(r, 17)
        cm.commit(r, 17)
        cm.audit()
        n = r.length
        for g, table in zip(cm.groups, r.tables):
            W, K = g.need.window, g.need.keep_first
            alive = {j for j in range(-(-n // 16)) if W is None or j < -(-K // 16) or (j + 1) * 16 > n + 1 - W}
            assert {j for j, p in enumerate(table) if p >= 0} == alive, (n, W, K)
    cm.close(r)
    assert cm.free_pages() == [30] * 4
    for bad in (PagedKVNeed(2, 8, keep_first=3), PagedKVNeed(2, 8, 8, keep_first=-1)):
        with pytest.raises(ValueError):
            CacheManager([bad], 16, 4, max_requests=1, allocate=False)


def test_random_weights_mode(tmp_path):
    import torch
    from kllm_b200.weights import write_random_model
    from kllm_b200.weights.safetensors_io import ModelFiles
    d = write_random_model(str(tmp_path / "m"), CFG_C, seed=3, dtype=torch.bfloat16)
    shapes = P.tensor_shapes(CFG_C)
    with ModelFiles(d) as f:
        assert set(f.names()) == set(shapes)
        for n in f.names():
            assert tuple(f.entry(n).shape) == tuple(shapes[n])
        assert float((f.read("l0.ls1") - 1).abs().max()) == 0.0 and float(f.read("l0.mlp.correction").abs().max()) == 0.0
        a = f.read("l1.mix.A_log").float()
        assert 0.0 <= float(a.min()) < float(a.max()) <= 2.7


def test_parts_refuse_what_they_cannot_do():
    import torch
    from kllm_b200.parts.model import DecoderModel  # noqa: F401  (registers the parts)
    from kllm_b200.parts.spec import BuildEnv, PartSpec, part_factory
    env = BuildEnv(dtype=torch.float32, device="cpu", hidden_size=32, max_position=16)

    def make(family, kind, **p):
        return part_factory(family, kind)(PartSpec(kind, "p", dict(hidden=32, **p)), env)
    ssd = dict(heads=4, head_dim=8, state=6, groups=2, taps=4, norm_parts=4, eps=1e-5)
    make("mixer", "ssd", **ssd)
    moe = dict(experts=4, top=2, expert_ff=8, score="softmax", weight_on="output")
    make("feed_forward", "routed_experts", **moe, identity=2, correction="c")
    for family, kind, p in (("mixer", "ssd", dict(ssd, groups=3)), ("mixer", "ssd", dict(ssd, norm_parts=5)), ("mixer", "ssd", dict(ssd, taps=65)),
                            ("feed_forward", "routed_experts", dict(moe, top=7, identity=2)),
                            ("feed_forward", "routed_experts", dict(moe, weight_on="input", identity=2)),
                            ("feed_forward", "routed_experts", dict(moe, activation="gelu")),
                            ("feed_forward", "gated_mlp", dict(intermediate=8, activation="clamped")),
                            ("feed_forward", "gated_mlp", dict(intermediate=8, activation="clamped", limit=1.0, bias=True))):
        with pytest.raises(ValueError):
            make(family, kind, **p)


def test_plain_recurrence_and_convolution_in_pieces():
    """The plain scan and convolution carried over a cut equal those over the whole."""
    rng = np.random.default_rng(0)
    T, H, G, N, dv = 20, 4, 2, 5, 3
    x, B, C = rng.standard_normal((T, H, dv)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt, A, D = rng.uniform(0, 1, (T, H)), rng.standard_normal(H), rng.standard_normal(H)
    whole, S = P.ssd_scan(x, B, C, dt, A, D)
    a, Sa = P.ssd_scan(x[:7], B[:7], C[:7], dt[:7], A, D)
    b, Sb = P.ssd_scan(x[7:], B[7:], C[7:], dt[7:], A, D, Sa)
    assert np.allclose(np.concatenate([a, b]), whole) and np.allclose(Sb, S)
    u, k, bias = rng.standard_normal((T, 6)), rng.standard_normal((6, 4)), rng.standard_normal(6)
    c = P.short_conv(u, k, bias)
    assert np.allclose(np.concatenate([P.short_conv(u[:9], k, bias), P.short_conv(u[9:], k, bias, u[6:9])]), c)
    assert np.allclose(c[0], u[0] * k[:, 3] + bias)


def test_plain_mask_counts():
    see = P.visible(np.arange(50), {"size": 6, "keep_first": 4})
    assert see.sum(axis=1).tolist() == [min(i + 1, 6) + min(4, max(0, i + 1 - 6)) for i in range(50)]
    assert np.array_equal(P.visible(np.arange(9), None), np.tril(np.ones((9, 9), bool)))
    assert P.tensor_shapes(CFG_D)["l0.mlp.router"] == (8, 224)
