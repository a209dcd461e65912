"""Gesuvik decoder: configuration -> model description.

x = embed[id].  Layers are pre-norm with RMS norms, x += mixer(norm1 x) and, with a feed-forward, x += ff(norm2 x).
Mixers: grouped-query attention whose queries and keys are normed over the whole projection, with YaRN rotation of
halves, a sliding window and a learned sink score per head (``parts/attention.py``); attention through a low-rank latent
with plain queries, a rotation of neighbours, a window, sinks and a gate per head (``parts/latent_attention.py``); or
retention, linear attention with fixed decays and rotated keys (``parts/recurrent.py``).  Feed-forward: routed experts of
the clamped gated form, chosen by corrected softmax scores, some of them the identity, beside a shared expert
(``parts/moe.py``).  A layer may use another layer's weights with a cache or state of its own: its schedule entry
names that layer again.  Output: RMS norm, then cap * tanh(scale * head x / cap).

Tensor names: ``embed``, ``final.norm``, ``head``, per layer i with tensors ``l<i>.norm1``, ``l<i>.norm2``,
``l<i>.mix.*`` and ``l<i>.mlp.*``.  This module only names parts and sizes; the parts know nothing of Gesuvik.
"""

from __future__ import annotations

from ..config.gesuvik import (ClampedExpert, GesuvikAttention, GesuvikConfig, GesuvikExperts, GesuvikLatentAttention,
                              GesuvikRetention, Rotation)
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunSpec, TensorSpec
from ..registry import register_architecture

MAX_POSITIONS = 1 << 30      # the design sets no limit; positions are 32-bit on the device


def _position(rot: Rotation):
    if rot is None or rot.dims == 0:
        return None
    params = {"rotary_dim": rot.dims, "theta": rot.base}
    if rot.scaling is not None:
        params.update(rot.scaling.to_dict())
    return PartSpec("rope_stretched", params)


def _mixer(cfg: GesuvikConfig, m, p: str) -> PartSpec:
    if isinstance(m, GesuvikAttention):
        return PartSpec(
            "attention",
            {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
             "value_dim": m.vdim, "scale": m.scale, "qk_norm_eps": cfg.norm_eps, "qk_norm_over": "projection",
             "window": m.window, "sinks": True, "position": _position(m.rot)},
            {"q": p + "q", "k": p + "k", "v": p + "v", "q_norm": p + "q.norm", "k_norm": p + "k.norm",
             "sink": p + "sink", "o": p + "o"})
    if isinstance(m, GesuvikLatentAttention):
        return PartSpec(
            "latent_attention",
            {"hidden_size": cfg.width, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_dim": m.vdim,
             "q_rank": None, "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps, "window": m.window,
             "pairing": "neighbours", "position": _position(m.rot), "sink": True, "head_gate": True},
            {"q": p + "q", "dkv": p + "dkv", "dkv_norm": p + "dkv.norm", "uk": p + "uk", "uv": p + "uv",
             "sink": p + "sink", "gate": p + "g", "o": p + "o"})
    assert isinstance(m, GesuvikRetention)
    return PartSpec(
        "retention",
        {"hidden_size": cfg.width, "num_heads": m.heads, "head_dim": m.dim, "v_dim": m.vdim, "decay": m.decay,
         "eps": cfg.norm_eps, "position": _position(m.rot)},
        {n: p + n for n in ("q", "k", "v", "g", "o")})


def _shared(cfg: GesuvikConfig, e: ClampedExpert, p: str) -> PartSpec:
    return PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": e.ff, "activation": "clamped",
                                  "limit": e.limit, "name": "shared_expert"},
                    {"gate": p + "gate", "up": p + "up", "down": p + "down"})


def _experts(cfg: GesuvikConfig, mlp: GesuvikExperts, p: str) -> PartSpec:
    weights = {"router": p + "router", "correction": p + "correction"}
    for e in range(mlp.experts):
        weights[f"gate_{e}"] = f"{p}e{e}.gate"
        weights[f"up_{e}"] = f"{p}e{e}.up"
        weights[f"down_{e}"] = f"{p}e{e}.down"
    return PartSpec(
        "routed_experts",
        {"hidden_size": cfg.width, "intermediate_size": mlp.expert.ff, "experts": mlp.experts, "identity": mlp.identity,
         "top": mlp.top, "activation": "clamped", "limit": mlp.expert.limit, "gated": True, "weights": "softmax",
         "corrected": True, "shared": None if mlp.shared is None else _shared(cfg, mlp.shared, p + "shared.")},
        weights)


def build_gesuvik(cfg: GesuvikConfig) -> ModelSpec:
    def norm(name):
        return PartSpec("rms_norm", {"size": cfg.width, "eps": cfg.norm_eps}, {"gain": name})

    layers, ignorable, place_of = [], [], {}
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is not None:
            continue
        p = f"l{i}."
        norms, ffn = {"pre_mixer": norm(p + "norm1")}, None
        if layer.mlp is not None:
            norms["pre_feed_forward"] = norm(p + "norm2")
            ffn = _experts(cfg, layer.mlp, p + "mlp.")
        else:                                   # a file may keep the unused sublayer's norm
            ignorable.append(p + "norm2")
        place_of[i] = len(layers)
        layers.append(LayerSpec(PartSpec("pre_norm"), _mixer(cfg, layer.mixer, p + "mix."), ffn, norms))
    # every run keeps a cache entry of its own, also where layers share their weights
    schedule = [RunSpec(place_of[cfg.owner(i)], i) for i in range(len(cfg.layers))]

    spec = ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embedding=TensorSpec("embed", (cfg.vocab, cfg.width), "embedding"), layers=layers, schedule=schedule,
        final_norm=norm("final.norm"), lm_head=TensorSpec("head", (cfg.vocab, cfg.width), "linear"),
        logit_multiplier=cfg.logit_scale, logit_softcap=cfg.logit_softcap, ignorable=tuple(ignorable))
    spec.check()
    return spec


register_architecture(GesuvikConfig.architecture, GesuvikConfig, build_gesuvik)
