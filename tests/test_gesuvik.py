"""Gesuvik without a GPU: reading the configuration, the schedule with layers that run on another's weights, the tensors
the model asks for, what the parts refuse, seeded random weights, and the plain implementation against closed forms."""

import copy
import json
import math

import pytest
import torch

from enginekernel_b200 import registry
from enginekernel_b200.config.base import ConfigError
from enginekernel_b200.config.gesuvik import GesuvikConfig
from enginekernel_b200.engine.model import DecoderModel, expected_tensors, ignorable_tensors
from enginekernel_b200.parts.spec import PartSpec
from tests.plain import gesuvik_models as models
from tests.plain import gesuvik_plain as plain

F64 = torch.float64


def test_registered_and_chosen_by_the_architecture_key(tmp_path):
    assert "Gesuvik" in registry.architectures()
    for tag, raw in models.SHAPES.items():
        folder = models.write_folder(str(tmp_path / tag), raw, {})
        cfg = registry.config_from_folder(folder)
        assert isinstance(cfg, GesuvikConfig)
        assert cfg.to_dict() == raw
        assert GesuvikConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg


@pytest.mark.parametrize("tag", list(models.SHAPES))
def test_schedule_parts_and_tensors_follow_the_configuration(tag):
    raw = models.SHAPES[tag]
    spec = registry.model_spec_for(GesuvikConfig.from_dict(raw))
    want = models.tensor_shapes(raw)
    got = expected_tensors(spec)
    assert set(got) == set(want)
    for name, shape in want.items():
        assert got[name].fits(shape), (name, got[name].shape, shape)
    own = [i for i in range(len(raw["layers"])) if raw["layers"][i].get("weights_of") is None]
    assert len(spec.layers) == len(own)
    assert [r.cache for r in spec.schedule] == list(range(len(raw["layers"])))     # an entry of its own for every run
    for i, run in enumerate(spec.schedule):
        assert run.writes_cache and run.layer == own.index(plain.owner(raw, i))
        ls = spec.layers[run.layer]
        assert ls.block.kind == "pre_norm" and ls.mixer.kind == raw["layers"][i]["type"]
        assert (ls.feed_forward is None) == (raw["layers"][i]["mlp"] is None)
    for i in own:
        assert (f"l{i}.norm2" in ignorable_tensors(spec)) == (raw["layers"][i]["mlp"] is None)
    assert spec.logit_multiplier == raw["logit_scale"] and spec.logit_softcap == raw["logit_softcap"]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tag", list(models.SHAPES))
def test_cache_entries_keep_a_window_or_a_state(tag, dtype):
    raw = models.SHAPES[tag]
    model = DecoderModel(registry.model_spec_for(GesuvikConfig.from_dict(raw)), dtype, "cpu")
    for spec, layer in zip(model.cache_entry_specs(), raw["layers"]):
        m = layer["mixer"]
        if layer["type"] == "retention":
            assert spec.kind == "state" and spec.shape[0] >= m["heads"] * m["dim"] * m["vdim"]
            continue
        assert spec.kind == "kv" and spec.window == (m.get("mask") or {}).get("size")
        if layer["type"] == "latent_attention":
            assert spec.planes == 1 and spec.heads == 1 and spec.head_dim >= m["kv_rank"] + m["rot_dim"]
        else:
            assert spec.planes == 2 and spec.heads == m["kv_heads"] and spec.head_dim >= max(m["dim"], m["vdim"])


def test_borrowed_weights_are_held_once():
    raw = models.SHAPES["flat"]
    model = DecoderModel(registry.model_spec_for(GesuvikConfig.from_dict(raw)), torch.float32, "cpu")
    model.load(models.make_tensors(raw, 1, torch.float32))
    assert len(model.blocks) == 3 and [r.layer for r in model.spec.schedule] == [0, 1, 2, 2, 2]


def test_what_the_configuration_refuses():
    base = models.SHAPES["early"]

    def broken(change):
        raw = copy.deepcopy(base)
        change(raw)
        return raw

    def cycle(r):
        r["layers"][0]["weights_of"] = 3

    cases = {
        "vocab": lambda r: r.pop("vocab"),
        "norm": lambda r: r.pop("norm"),
        "logit_scale": lambda r: r.pop("logit_scale"),
        "logit_softcap": lambda r: r.update(logit_softcap=0.0),
        "layers": lambda r: r.update(layers=[]),
        "type": lambda r: r["layers"][1].update(type="mamba2"),
        "mixer": lambda r: r["layers"][1].pop("mixer"),
        "decay": lambda r: r["layers"][1]["mixer"].update(decay=[0.5]),
        "heads": lambda r: r["layers"][2]["mixer"].update(kv_heads=3),
        "kv_rank": lambda r: r["layers"][0]["mixer"].pop("kv_rank"),
        "rot.dims": lambda r: r["layers"][0]["mixer"]["rot"].update(dims=18),
        "scaling": lambda r: r["layers"][2]["mixer"]["rot"]["scaling"].pop("fast"),
        "rot.scaling.factor": lambda r: r["layers"][2]["mixer"]["rot"]["scaling"].update(factor=0.0),
        "mask.size": lambda r: r["layers"][2]["mixer"]["mask"].update(size=0),
        "another layer": cycle,
        "must equal": lambda r: r["layers"][3]["mixer"].update(vdim=24),
        "weights_of": lambda r: r["layers"][3].update(weights_of=9),
        "kind": lambda r: r["layers"][0]["mlp"].update(kind="dense"),
        "top": lambda r: r["layers"][2]["mlp"]["router"].update(top=9),
        "identity": lambda r: r["layers"][2]["mlp"]["router"].update(identity=-1),
        "expert.limit": lambda r: r["layers"][2]["mlp"]["expert"].update(limit=0.0),
        "shared.limit": lambda r: r["layers"][0]["mlp"]["shared"].pop("limit"),
        "width": lambda r: r.update(width=96.5),
    }
    for word, change in cases.items():
        with pytest.raises(ConfigError, match=word.replace(".", r"\.")):
            GesuvikConfig.from_dict(broken(change))


def test_parts_refuse_what_they_cannot_do():
    from enginekernel_b200.parts.attention import Attention
    from enginekernel_b200.parts.latent_attention import LatentAttention
    from enginekernel_b200.parts.moe import RoutedExperts
    from enginekernel_b200.parts.recurrent import Retention
    base = {"hidden_size": 64, "num_heads": 2, "num_kv_heads": 1, "head_dim": 32, "scale": 1.0}
    for more, word in (({"sinks": True, "sink": 0.0}, "sink"), ({"qk_norm_over": "row", "qk_norm_eps": 1e-6}, "projection"),
                       ({"qk_norm_over": "projection"}, "qk_norm_eps"),
                       ({"qk_norm_over": "projection", "qk_norm_eps": 1e-6, "bias": ("q",)}, "biases")):
        with pytest.raises(ValueError, match=word):
            Attention(PartSpec("attention", {**base, **more}), torch.float32, "cpu")
    lat = {"hidden_size": 64, "num_heads": 2, "head_dim": 16, "rot_dim": 8, "v_dim": 16, "q_rank": None, "kv_rank": 24,
           "scale": 1.0, "eps": 1e-6}
    for more, word in (({"pairing": "thirds"}, "pairing"), ({"window": 0}, "window"), ({"head_gate": True, "q_rank": 8}, "gate"),
                       ({"kv_rank": 1100}, "limit")):
        with pytest.raises(Exception, match=word):
            LatentAttention(PartSpec("latent_attention", {**lat, **more}), torch.float32, "cpu")
    moe = {"hidden_size": 8, "intermediate_size": 8, "experts": 4, "top": 2, "weights": "softmax", "activation": "silu", "gated": True}
    for more, word in (({"top": 7, "identity": 2}, "top"), ({"corrected": True, "weights": "sigmoid"}, "correction"),
                       ({"identity": 1, "weigh": "input"}, "identity"), ({"identity": -1}, "identity")):
        with pytest.raises(ValueError, match=word):
            RoutedExperts(PartSpec("routed_experts", {**moe, **more}), torch.float32, "cpu")
    with pytest.raises(ValueError, match="decay"):
        Retention(PartSpec("retention", {"hidden_size": 8, "num_heads": 2, "head_dim": 4, "v_dim": 4, "eps": 1e-6,
                                         "decay": [0.5]}), torch.float32, "cpu")


def test_random_weights_cover_corrections_and_sinks():
    from enginekernel_b200.weights.random_init import random_tensors
    raw = models.SHAPES["early"]
    t = random_tensors(expected_tensors(registry.model_spec_for(GesuvikConfig.from_dict(raw))), 3, dtype=torch.float32)
    assert {n: tuple(x.shape) for n, x in t.items()} == models.tensor_shapes(raw)
    c = t["l2.mlp.correction"]
    assert c.abs().max() > 0 and (c < 0).any() and (c > 0).any()


@pytest.mark.parametrize("rot", [models.rotation(64, 5e5, (8.0, 8192, 32.0, 1.0)), models.rotation(8, 500.0, (4.0, 40, 8.0, 1.0)),
                                 models.rotation(10, 1e6, (2.0, 100, 4.0, 1.0)), models.rotation(12, 1e4)])
def test_tables_of_the_slowed_rotation(rot):
    from enginekernel_b200.parts.rope import RopeStretched
    part = RopeStretched(PartSpec("rope_stretched", {"rotary_dim": rot["dims"], "theta": rot["base"], **rot.get("scaling", {})}),
                         torch.float32, "cpu")
    speeds, factor = plain.rotation_speeds(rot)
    part.prepare(700)
    ang = torch.arange(700, dtype=F64)[:, None] * speeds[None]
    assert (part.cos.double() - factor * ang.cos()).abs().max() < 1e-6
    assert (part.sin.double() - factor * ang.sin()).abs().max() < 1e-6


# ------------------------------------------------------------------ the plain implementation against closed forms
def test_retention_is_a_decayed_sum_of_past_values():
    t, nh, d, e = 7, 2, 3, 4
    g = torch.Generator().manual_seed(0)
    q, k = torch.randn(t, nh, d, generator=g, dtype=F64), torch.randn(t, nh, d, generator=g, dtype=F64)
    v = torch.randn(t, nh, e, generator=g, dtype=F64)
    decay = [0.7, 1.0]
    out, _ = plain.retention_scan(q, k, v, decay)
    for n in range(t):
        for h in range(nh):
            want = sum(decay[h] ** (n - j) * (q[n, h] @ k[j, h]) * v[j, h] for j in range(n + 1))
            assert torch.allclose(out[n, h], want)
    again, _ = plain.retention_scan(q[4:], k[4:], v[4:], decay, state=plain.retention_scan(q[:4], k[:4], v[:4], decay)[1])
    assert torch.allclose(again, out[4:])


def test_windows_and_sinks():
    assert [[plain.sees(i, j, 3) for j in range(6)] for i in (0, 2, 3, 5)] == [
        [True] + [False] * 5, [True] * 3 + [False] * 3, [False] + [True] * 3 + [False] * 2, [False] * 3 + [True] * 3]
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(9, 2, 6, generator=g, dtype=F64) for _ in range(3))
    none = torch.full((2,), -1e9, dtype=F64)
    alone = plain.attend(q, k, v, 1.0, 1, none)                         # a window of one token: the token's own value
    assert torch.allclose(alone, v)
    half = plain.attend(q, k, v, 0.0, None, torch.tensor([math.log(9.0), -1e9], dtype=F64))
    assert torch.allclose(half[8, 0], v[:, 0].mean(0) / 2) and torch.allclose(half[8, 1], v[:, 1].mean(0))


def test_latent_keys_share_one_rotated_part_and_neighbours_turn():
    raw = models.SHAPES["early"]
    w, m = models.make_tensors(raw, 3), raw["layers"][0]["mixer"]
    h = torch.randn(5, raw["width"], generator=torch.Generator().manual_seed(2), dtype=F64)
    pos = torch.tensor([0, 1, 2, 50, 51])
    _, k, _ = plain.latent_queries_keys_values(h, w, "l0.mix.", m, 1e-5, pos)
    d = m["dim"]
    for head in range(1, m["heads"]):
        assert torch.equal(k[:, 0, d:], k[:, head, d:])
    raw_part = plain.project(h, w, "l0.mix.dkv")[:, m["kv_rank"]:]
    norm = lambda x: x[:, 0::2] ** 2 + x[:, 1::2] ** 2                  # a pair's length does not change
    assert torch.allclose(norm(k[:, 0, d:]), norm(raw_part)) and not torch.allclose(k[1:, 0, d:], raw_part[1:])
    rot, x = models.rotation(8, 100.0), torch.randn(5, 1, 10, dtype=F64)
    order = [0, 2, 4, 6, 1, 3, 5, 7, 8, 9]
    assert torch.allclose(plain.rotate(x, pos, rot, True)[..., order], plain.rotate(x[..., order], pos, rot, False))


def test_the_norm_of_queries_runs_over_all_heads():
    raw = models.SHAPES["early"]
    w, m = models.make_tensors(raw, 3, F64), dict(raw["layers"][2]["mixer"], rot=None)
    w["l2.mix.q.norm"] = torch.ones_like(w["l2.mix.q.norm"])
    h = torch.randn(4, raw["width"], dtype=F64, generator=torch.Generator().manual_seed(7))
    q, _, _ = plain.make_queries_keys_values(h, w, "l2.mix.", m, 0.0, torch.arange(4))
    assert torch.allclose((q ** 2).mean((1, 2)), torch.ones(4, dtype=F64))
    assert ((q ** 2).mean(2) - 1).abs().max() > 0.05


def test_corrections_choose_and_identity_experts_return_the_input():
    g = torch.Generator().manual_seed(5)
    n, ident, width = 3, 2, 4
    w = {f"e{e}.{name}": torch.randn(4, 4, generator=g, dtype=F64) for e in range(n) for name in ("gate", "up", "down")}
    w["router"], w["correction"] = torch.randn(n + ident, width, generator=g, dtype=F64), torch.tensor([-9.0, 0.0, 0.0, 9.0, 0.0])
    m = models.moe(n, ident, 2, 4, limit=0.7)
    x = torch.randn(6, width, generator=g, dtype=F64)
    s = torch.softmax(x @ w["router"].T, -1)
    got = plain.experts_ff(x, w, "", m)
    for t in range(6):
        second = max((1, 2, 4), key=lambda e: float(s[t, e]))            # 3 is always in, 0 never
        other = x[t] if second == 4 else plain.clamped_glu(x[t][None], w, f"e{second}.", 0.7)[0]
        assert torch.allclose(got[t], s[t, 3] * x[t] + s[t, second] * other)


@pytest.mark.parametrize("tag", ["early", "odd"])
def test_the_plain_model_is_causal_and_capped(tag):
    cfg = models.SHAPES[tag]
    w = models.make_tensors(cfg, 4)
    a = models.random_prompts(cfg, [30], seed=1)[0]
    b = list(a)
    b[20] = (a[20] + 1) % cfg["vocab"]
    la, lb = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    assert torch.equal(la[:20], lb[:20]) and (la[20:] - lb[20:]).abs().max() > 1e-6
    assert la.abs().max() < cfg["logit_softcap"]
    wide = plain.forward(dict(cfg, logit_softcap=1e7), w, a)
    assert torch.allclose(plain.cap(wide, cfg["logit_softcap"]), la, atol=1e-6) and (wide - la).abs().max() > 1e-3
