"""The Rupenex architecture as a ``ModelSpec``: a decoder whose sublayers read the residual stream itself and
are layer-normed (a weight, no bias) on their OUTPUT, each result scaled channel by channel before it joins the
stream; the embedding's rows are normed as well, and the logits multiplied by a constant.  Two kinds of mixer: grouped
attention in a sliding window that keeps the first keys of the sequence, with RMS norms per query and key head, a
rotation with evenly stretched frequencies, a learned sink per head and a sigmoid gate on the heads' outputs; and a
state-space recurrence with one decay per head and token behind a short convolution (Mamba-2).  The feed-forward is a
clamped gated one, or experts without a gate (the square of relu) chosen by corrected softmax scores, some of which
hand their input through, beside an expert that every token runs; or absent.

This file holds no sizes and no kernels: it translates ``RupenexConfig`` into part descriptions.  What the
design fixes is written here as parameters of general parts.  Tensor names: ``embed``, ``embed.norm``, ``head``,
``final.norm``, and ``l<i>.{norm1,ls1,norm2,ls2}``, ``l<i>.mix.*``, ``l<i>.mlp.*`` for layer i.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.rupenex import RupenexConfig
from ..parts.spec import BlockSpec, LayerCall, ModelSpec, PartSpec

MAX_POSITION = 1 << 24          # angles are formed on the device from the position: the cache's size is the only bound
SLOPE = 1.702                   # of the dense feed-forward's sigmoid
SUM_EPS = 1e-20                 # added to the sum of the chosen experts' scores


def _mixer(p, L, d, eps):
    m = L.mixer
    if L.type == "mamba2":
        return PartSpec("ssd", p, {"hidden": d, "heads": m.heads, "head_dim": m.vdim, "state": m.state, "groups": m.groups,
                                   "taps": m.conv, "norm_parts": m.norm_groups, "eps": eps})
    scaling = {"kind": "linear", "factor": m.rot.factor} if m.rot and m.rot.factor is not None else None
    return PartSpec("paged_attention", p, {
        "hidden": d, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
        "window": m.window, "keep_first": m.keep_first, "scale": m.scale, "position": None, "exact_weights": True,
        "tensors": {k: f"{p}.{k}" for k in "qkvo"}, "sink": p + ".sink", "out_gate": p + ".g",
        "qk_transform": PartSpec("head_rmsnorm_rotary", "", {
            "head_dim": m.dim, "eps": eps, "q_gain": p + ".q.norm", "k_gain": p + ".k.norm",
            "rotary_dim": m.rot.dims if m.rot else 0, "theta": m.rot.base if m.rot else 0.0, "scaling": scaling})})


def _feed_forward(p, mlp, d):
    if mlp is None:
        return None
    if mlp.kind == "dense":
        return PartSpec("gated_mlp", p, {"hidden": d, "intermediate": mlp.ff, "activation": "clamped", "limit": mlp.limit,
                                         "alpha": SLOPE, "tensors": {k: f"{p}.{k}" for k in ("gate", "up", "down")}})
    shared = None
    if mlp.shared_ff:
        shared = {"ff": mlp.shared_ff, "activation": "relu2", "tensors": {k: f"{p}.shared.{k}" for k in ("up", "down")}}
    return PartSpec("routed_experts", p, {
        "hidden": d, "experts": mlp.experts, "top": mlp.top, "identity": mlp.identity, "expert_ff": mlp.ff,
        "activation": "relu2", "score": "softmax", "correction": p + ".correction", "renormalize": True,
        "sum_eps": SUM_EPS, "weight_on": "output", "shared": shared})


def build_rupenex_spec(cfg: RupenexConfig) -> ModelSpec:
    d = cfg.width

    def norm(name, scale=None, factor=1.0):
        return PartSpec("layernorm", "", {"width": d, "eps": cfg.norm_eps, "tensor": name, "bias": False, "layer_scale": scale,
                                          "factor": factor})

    blocks = [BlockSpec(kind="output_norm", prefix=f"l{i}", mixer=_mixer(f"l{i}.mix", L, d, cfg.norm_eps),
                        feed_forward=_feed_forward(f"l{i}.mlp", L.mlp, d), mixer_norm=norm(f"l{i}.norm1", f"l{i}.ls1"),
                        ff_norm=norm(f"l{i}.norm2", f"l{i}.ls2") if L.mlp else None)
              for i, L in enumerate(cfg.layers)]
    return ModelSpec(
        hidden_size=d, vocab_size=cfg.vocab, max_position=MAX_POSITION,
        embedding=PartSpec("token_embedding", "", {"vocab": cfg.vocab, "width": d, "tensor": "embed", "norm": norm("embed.norm")}),
        blocks=blocks, schedule=[LayerCall(block=i, cache=i) for i in range(len(blocks))],
        # the logits' factor acts on the head's input: the head is linear
        final_norm=norm("final.norm", factor=cfg.logit_scale),
        head=PartSpec("linear_head", "", {"vocab": cfg.vocab, "width": d, "tied_to": None, "tensor": "head"}),
        eos_token_ids=())


register_architecture("Rupenex", RupenexConfig, build_rupenex_spec)
