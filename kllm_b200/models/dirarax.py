"""The Dirarax architecture as a ``ModelSpec``: a decoder whose layers have one norm (an RMS norm whose weight is
stored around zero and acts as 1 + w) that the mixer and the feed-forward both read, the mixer through a token shift, and whose
two results join the stream together.  A mixer is linear attention with a gated decay per key channel, or two
mixers side by side: gated softmax attention with an interleaved, stretched rotation, and linear attention with a fixed
decay per head over rotated queries and keys.  The feed-forward is a biased gelu-gated one, or experts with a softmax over the
chosen logits and an expert that every token runs.  A run of layers may repeat with the same weights; before each of
its passes the stream is mixed with the embedding's output and a vector of the pass is added.  The head is the embedding table.

This file holds no sizes and no kernels: it translates ``DiraraxConfig`` into part descriptions.  What the
design fixes is written here as parameters of general parts.  Tensor names: ``embed``, ``loop.in``, ``loop.step``,
``final.norm``, and ``l<i>.{norm1,shift}``, ``l<i>.mix.*`` (``.mix.left.*``, ``.mix.right.*``), ``l<i>.mlp.*`` for layer i.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.dirarax import DiraraxConfig
from ..parts.spec import BlockSpec, LayerCall, ModelSpec, PartSpec

MAX_POSITION = 1 << 24          # angles are formed on the device from the position: the cache's size is the only bound


def _ramp(rot):
    sc = rot.scaling_dict() if rot else None
    return None if sc is None else dict(sc, kind="ramp")


def _mixer(p, L, d, eps):
    m = L.mixer
    if L.type == "gla":
        return PartSpec("gated_linear_attention", p, {
            "hidden": d, "heads": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim, "tau": m.tau, "eps": eps})
    a, r = m.left, m.right
    left = PartSpec("paged_attention", p + ".left", {
        "hidden": d, "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "v_head_dim": a.vdim, "window": None,
        "scale": a.scale, "position": None, "exact_weights": True, "tensors": {k: f"{p}.left.{k}" for k in "qkvo"},
        "out_gate": p + ".left.g", "out_factor": m.left_scale,
        "qk_transform": PartSpec("head_rmsnorm_rotary", "", {
            "head_dim": a.dim, "rotary_dim": a.rot.dims if a.rot else 0, "theta": a.rot.base if a.rot else 0.0,
            "scaling": _ramp(a.rot), "interleaved": True})})
    right = PartSpec("retention", p + ".right", {
        "hidden": d, "heads": r.heads, "head_dim": r.dim, "v_head_dim": r.vdim, "decay": list(r.decay), "eps": eps,
        "rotary_dim": r.rot.dims if r.rot else 0, "theta": r.rot.base if r.rot else 0.0, "out_factor": m.right_scale})
    return PartSpec("side_by_side", p, {"members": [left, right]})


def _feed_forward(p, mlp, d):
    if mlp is None:
        return None
    if mlp.kind == "dense":
        return PartSpec("gated_mlp", p, {"hidden": d, "intermediate": mlp.ff, "activation": "gelu_tanh", "bias": True,
                                         "tensors": {k: f"{p}.{k}" for k in ("gate", "up", "down")}})
    shared = None
    if mlp.shared_ff:
        shared = {"ff": mlp.shared_ff, "tensors": {k: f"{p}.shared.{k}" for k in ("gate", "up", "down")}}
    return PartSpec("routed_experts", p, {
        "hidden": d, "experts": mlp.experts, "top": mlp.top, "expert_ff": mlp.ff, "score": "softmax", "renormalize": True,
        "weight_on": "output", "shared": shared})


def build_dirarax_spec(cfg: DiraraxConfig) -> ModelSpec:
    d = cfg.width

    def norm(name):
        return PartSpec("rmsnorm", "", {"width": d, "eps": cfg.norm_eps, "tensor": name, "offset": 1.0})

    blocks = [BlockSpec(kind="parallel", prefix=f"l{i}", mixer=_mixer(f"l{i}.mix", L, d, cfg.norm_eps),
                        feed_forward=_feed_forward(f"l{i}.mlp", L.mlp, d), mixer_norm=norm(f"l{i}.norm1"), ff_norm=None,
                        params={"shift": f"l{i}.shift"})
              for i, L in enumerate(cfg.layers)]
    entries = []
    if cfg.loop_times:
        entries = [PartSpec("embedding_mix", "loop", {"hidden": d, "passes": cfg.loop_times, "in": "loop.in",
                                                      "step": "loop.step"})]
    return ModelSpec(
        hidden_size=d, vocab_size=cfg.vocab, max_position=MAX_POSITION,
        embedding=PartSpec("token_embedding", "", {"vocab": cfg.vocab, "width": d, "tensor": "embed"}),
        blocks=blocks,
        schedule=[LayerCall(block=b, cache=run, entry=None if t is None else (0, t))
                  for run, (b, t) in enumerate(cfg.layer_order())],
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", "", {"vocab": cfg.vocab, "width": d, "tied_to": "embed", "tensor": "embed"}),
        eos_token_ids=(), entries=entries)


register_architecture("Dirarax", DiraraxConfig, build_dirarax_spec)
