"""Kamosun decoder: configuration -> model description.

x = embed[id].  A layer's two sublayers run side by side on two norms of the same x, each result gated by the sigmoid
of a projection of what the sublayer read, and the layer's result X_n = x + m (g1 mixer(n1 x) + g2 ff(n2 x)) is not what
goes on: the next layer (after the last one, the output) reads a learned average over the embedding output and all
results so far (``parts/block.py``, ``gated_parallel``).  All norms of the stream are dynamic tanh
(``parts/norm.py``).  Mixers: grouped-query attention within chunks of positions, with biases, a gained norm of
queries and keys and a rotation of halves, optionally with the keys and values of an earlier layer
(``parts/attention.py``); or two mixers side by side (``parts/pair.py``): full attention with a soft cap on its
scores and a rotation of neighbours whose long wavelengths are slowed down, and linear attention with a fixed decay
per head (``fixed_decay_memory`` in ``parts/recurrent.py``), both results normed over the width and averaged.
Feed-forward: a gated one with clamped halves (``gated_mlp``), or routed experts of that form chosen by sigmoid
scores, the score multiplying the expert's input, beside a shared expert (``parts/moe.py``).  Output: a dynamic tanh,
then logits against ``head``.

Tensor names: ``embed``, ``final.norm`` (``.alpha``, ``.b``), ``head``, per layer i ``l<i>.norm1``, ``norm2`` (``.alpha``,
``.b``), ``l<i>.rg1``, ``rg2`` (``.b``), ``l<i>.dwa``, ``l<i>.mix.*`` and ``l<i>.mlp.*``.  This module only names parts and
sizes; the parts know nothing of Kamosun.
"""

from __future__ import annotations

from ..config.kamosun import ClampedGlu, Experts, KamosunAttention, KamosunConfig, SideBySide
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunSpec, TensorSpec
from ..registry import register_architecture

MAX_POSITIONS = 1 << 30      # the design sets no limit; positions are 32-bit on the device


def _attention(cfg: KamosunConfig, m: KamosunAttention, p: str, pairing: str, bias, cache_window=None) -> PartSpec:
    position = None
    if m.rot is not None and m.rot.dims > 0:
        rot = {"rotary_dim": m.rot.dims, "theta": m.rot.base}
        if m.rot.scaling is not None:
            rot.update(m.rot.scaling.to_dict())
        position = PartSpec("rope_by_wavelength", rot)
    weights = {"q": p + "q", "o": p + "o", "q_norm": p + "q.norm"}
    if m.kv_from is None:
        weights.update(k=p + "k", v=p + "v", k_norm=p + "k.norm")
    weights.update({which + "_bias": f"{p}{which}.b" for which in bias})
    return PartSpec(
        "attention",
        {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
         "value_dim": m.vdim, "scale": m.scale, "qk_norm_eps": cfg.norm_eps, "bias": bias, "chunk": m.chunk,
         "cache_window": cache_window, "softcap": m.softcap, "pairing": pairing, "kv_projection": m.kv_from is None,
         "keep_all_keys": cache_window is None, "position": position},
        weights)


def _mixer(cfg: KamosunConfig, m, p: str, cache_window) -> PartSpec:
    if isinstance(m, KamosunAttention):
        return _attention(cfg, m, p, "halves", ("q", "k", "v", "o"), cache_window)
    assert isinstance(m, SideBySide)
    r, rp = m.right, p + "right."
    right = PartSpec(
        "fixed_decay_memory",
        {"hidden_size": cfg.width, "num_heads": r.heads, "head_dim": r.dim, "v_dim": r.vdim, "decay": r.decay,
         "eps": cfg.norm_eps},
        {n: rp + n for n in ("q", "k", "v", "g", "norm", "o")})
    return PartSpec(
        "mixer_pair",
        {"hidden_size": cfg.width, "first": _attention(cfg, m.left, p + "left.", "neighbours", ()), "second": right,
         "weight_first": 0.5, "weight_second": 0.5, "result_eps": cfg.norm_eps},
        {"first_gain": p + "left.out", "second_gain": p + "right.out"})


def _clamped(cfg: KamosunConfig, g: ClampedGlu, p: str, name: str) -> PartSpec:
    return PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": g.ff, "activation": "clamped",
                                  "limit": g.limit, "name": name},
                    {"gate": p + "gate", "up": p + "up", "down": p + "down"})


def _feed_forward(cfg: KamosunConfig, mlp, p: str) -> PartSpec:
    if isinstance(mlp, ClampedGlu):
        return _clamped(cfg, mlp, p, "mlp")
    assert isinstance(mlp, Experts)
    weights = {"router": p + "router"}
    for e in range(mlp.experts):
        weights[f"gate_{e}"] = f"{p}e{e}.gate"
        weights[f"up_{e}"] = f"{p}e{e}.up"
        weights[f"down_{e}"] = f"{p}e{e}.down"
    return PartSpec(
        "routed_experts",
        {"hidden_size": cfg.width, "intermediate_size": mlp.expert.ff, "experts": mlp.experts, "top": mlp.top,
         "activation": "clamped", "limit": mlp.expert.limit, "gated": True, "weights": "sigmoid", "weigh": "input",
         "shared": None if mlp.shared is None else _clamped(cfg, mlp.shared, p + "shared.", "shared_expert")},
        weights)


def build_kamosun(cfg: KamosunConfig) -> ModelSpec:
    def norm(name):
        return PartSpec("dynamic_tanh", {"size": cfg.width}, {"alpha": name + ".alpha", "gain": name, "shift": name + ".b"})

    # how many of its last keys each attention layer's cache entry keeps: the largest chunk among the layers that
    # read it (None: all of them)
    keeps = {}
    for i, layer in enumerate(cfg.layers):
        if layer.type == "attention":
            src = i if layer.mixer.kv_from is None else layer.mixer.kv_from
            keeps.setdefault(src, []).append(layer.mixer.chunk)

    layers, schedule, ignorable, entry_of, entries = [], [], [], {}, 0
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        norms = {"pre_mixer": norm(p + "norm1")}
        weights = {"mixer_gate": p + "rg1", "mixer_gate_bias": p + "rg1.b", "depth": p + "dwa"}
        ffn = None
        if layer.mlp is not None:
            norms["pre_feed_forward"] = norm(p + "norm2")
            weights.update(feed_forward_gate=p + "rg2", feed_forward_gate_bias=p + "rg2.b")
            ffn = _feed_forward(cfg, layer.mlp, p + "mlp.")
        else:                                   # a file may keep the unused sublayer's norm and gate
            ignorable += [p + "norm2", p + "norm2.alpha", p + "norm2.b", p + "rg2", p + "rg2.b"]
        src = getattr(m, "kv_from", None)
        window = None
        if layer.type == "attention":
            sizes = keeps[i if src is None else src]
            window = None if None in sizes else max(sizes)
        block = PartSpec("gated_parallel", {"hidden_size": cfg.width, "multiplier": cfg.residual_mult, "depth": i + 1,
                                            "layers": len(cfg.layers)}, weights)
        layers.append(LayerSpec(block, _mixer(cfg, m, p + "mix.", window), ffn, norms))
        if src is not None:                     # reads what layer `src` stored in this step and before
            schedule.append(RunSpec(i, entry_of[src], writes_cache=False))
            continue
        pair = isinstance(m, SideBySide)
        entry_of[i] = entries
        schedule.append(RunSpec(i, entries, more_caches=(entries + 1,) if pair else ()))
        entries += 2 if pair else 1

    spec = ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embedding=TensorSpec("embed", (cfg.vocab, cfg.width), "embedding"), layers=layers, schedule=schedule,
        final_norm=norm("final.norm"), lm_head=TensorSpec("head", (cfg.vocab, cfg.width), "linear"),
        ignorable=tuple(ignorable))
    spec.check()
    return spec


register_architecture(KamosunConfig.architecture, KamosunConfig, build_kamosun)
