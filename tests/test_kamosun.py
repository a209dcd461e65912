"""Kamosun without a GPU: reading the configuration, the schedule with its cache entries and borrowed keys, the
tensors the model asks for, the tables of a rotation slowed by wavelength, seeded random weights, and the plain
implementation against closed forms."""

import copy
import json
import math

import pytest
import torch

from enginekernel_b200 import registry
from enginekernel_b200.config.base import ConfigError
from enginekernel_b200.config.kamosun import KamosunConfig
from enginekernel_b200.engine.model import DecoderModel, expected_tensors, ignorable_tensors
from enginekernel_b200.parts.rope import RopeByWavelength
from enginekernel_b200.parts.spec import PartSpec
from tests.plain import kamosun_models as models
from tests.plain import kamosun_plain as plain

F64 = torch.float64


def test_registered_and_chosen_by_the_architecture_key(tmp_path):
    assert "Kamosun" in registry.architectures()
    for tag, raw in models.SHAPES.items():
        folder = models.write_folder(str(tmp_path / tag), raw, {})
        cfg = registry.config_from_folder(folder)
        assert isinstance(cfg, KamosunConfig)
        assert cfg.to_dict() == raw
        assert KamosunConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg


@pytest.mark.parametrize("tag", list(models.SHAPES))
def test_schedule_parts_and_tensors_follow_the_configuration(tag):
    raw = models.SHAPES[tag]
    spec = registry.model_spec_for(KamosunConfig.from_dict(raw))
    want = models.tensor_shapes(raw)
    got = expected_tensors(spec)
    assert set(got) == set(want)
    for name, shape in want.items():
        assert got[name].fits(shape), (name, got[name].shape, shape)
    assert [r.layer for r in spec.schedule] == list(range(len(raw["layers"])))
    own = []
    for i, (run, layer, ls) in enumerate(zip(spec.schedule, raw["layers"], spec.layers)):
        assert ls.block.kind == "gated_parallel" and ls.block.params["depth"] == i + 1
        assert ls.block.params["layers"] == len(raw["layers"]) and ls.block.params["multiplier"] == raw["residual_mult"]
        assert ls.mixer.kind == {"attention": "attention", "parallel": "mixer_pair"}[layer["type"]]
        src = layer["mixer"].get("kv_from")
        if src is not None:
            assert run.cache == spec.schedule[src].cache and not run.writes_cache
        else:
            assert run.writes_cache
            own += [run.cache, *run.more_caches]
        assert len(run.more_caches) == (1 if layer["type"] == "parallel" else 0)
        assert (ls.feed_forward is None) == (layer["mlp"] is None)
        assert (f"l{i}.rg2" in ignorable_tensors(spec)) == (layer["mlp"] is None)
    assert sorted(own) == list(range(spec.num_cache_entries()))


def test_a_shared_entry_keeps_what_its_widest_reader_sees():
    """Layers that share keys may cut different chunks: the entry keeps the largest, or everything."""
    def windows(raw):
        model = DecoderModel(registry.model_spec_for(KamosunConfig.from_dict(raw)), torch.float32, "cpu")
        return [s.window for s in model.cache_entry_specs() if s.kind == "kv"]

    assert windows(models.EARLY) == [None, 17, None]
    assert windows(models.FLAT) == [70, None]
    assert windows(models.ODD) == [None, None, 5]
    assert windows(models.WIDE) == [None, 130, 96, None]


def test_what_the_configuration_refuses():
    base = models.SHAPES["early"]

    def broken(change):
        raw = copy.deepcopy(base)
        change(raw)
        return raw

    cases = {
        "vocab": lambda r: r.pop("vocab"),
        "norm": lambda r: r.pop("norm"),
        "residual_mult": lambda r: r.pop("residual_mult"),
        "layers": lambda r: r.update(layers=[]),
        "type": lambda r: r["layers"][1].update(type="mamba2"),
        "left": lambda r: r["layers"][0]["mixer"].pop("left"),
        "decay": lambda r: r["layers"][0]["mixer"]["right"].update(decay=[0.5]),
        "heads": lambda r: r["layers"][1]["mixer"].update(kv_heads=4),
        "rot.dims": lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=26),
        "high": lambda r: r["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(high=0.5),
        "mask.size": lambda r: r["layers"][1]["mixer"]["mask"].update(size=0),
        "kv_from": lambda r: r["layers"][2]["mixer"].update(kv_from=0),
        "whose keys": lambda r: r["layers"][2]["mixer"].update(dim=24),
        "softcap": lambda r: r["layers"][0]["mixer"]["left"].update(softcap=-1.0),
        "kind": lambda r: r["layers"][0]["mlp"].update(kind="gelu"),
        "top": lambda r: r["layers"][0]["mlp"]["router"].update(top=7),
        "limit": lambda r: r["layers"][2]["mlp"].update(limit=0.0),
        "shared.limit": lambda r: r["layers"][0]["mlp"]["shared"].pop("limit"),
        "width": lambda r: r.update(width=96.5),
    }
    for word, change in cases.items():
        with pytest.raises(ConfigError, match=word.replace(".", r"\.")):
            KamosunConfig.from_dict(broken(change))


@pytest.mark.parametrize("rot", [models.rotation(64, 5e5, (8.0, 1.0, 4.0, 8192)), models.rotation(16, 500.0, (4.0, 1.0, 3.0, 40)),
                                 models.rotation(8, 100.0, (2.0, 2.0, 2.5, 30)), models.rotation(12, 1e4)])
def test_tables_of_the_rotation_slowed_by_wavelength(rot):
    params = {"rotary_dim": rot["dims"], "theta": rot["base"], **rot.get("scaling", {})}
    part = RopeByWavelength(PartSpec("rope_by_wavelength", params), torch.float32, "cpu")
    want = plain.frequencies(rot)
    assert torch.allclose(part.frequencies(), want, rtol=1e-12, atol=0)
    part.prepare(3000)
    ang = torch.arange(3000, dtype=F64)[:, None] * want[None]
    assert (part.cos.double() - ang.cos()).abs().max() < 1e-6 and (part.sin.double() - ang.sin()).abs().max() < 1e-6
    plain_f = plain.frequencies({"base": rot["base"], "dims": rot["dims"]})
    if "scaling" in rot:                       # the fastest stay, the slowest turn `factor` times slower
        assert part.frequencies()[0] == plain_f[0]
        assert torch.isclose(part.frequencies()[-1], plain_f[-1] / rot["scaling"]["factor"])


def test_random_weights_of_an_average_lean_on_the_last_result():
    from enginekernel_b200.weights.random_init import random_tensors
    t = random_tensors(expected_tensors(registry.model_spec_for(KamosunConfig.from_dict(models.FLAT))), 3, dtype=torch.float32)
    for i in range(3):
        w = t[f"l{i}.dwa"]
        assert w.shape == (i + 2,) and abs(float(w[-1]) - 1) < 0.2 and w[:-1].abs().max() < 0.2
    assert t["l0.norm1.alpha"].shape == () and 0.5 < float(t["l0.norm1.alpha"]) < 1.5


def test_parts_refuse_what_they_cannot_do():
    from enginekernel_b200.parts.attention import Attention
    from enginekernel_b200.parts.mlp import GatedMLP
    from enginekernel_b200.parts.moe import RoutedExperts
    base = {"hidden_size": 64, "num_heads": 2, "num_kv_heads": 1, "head_dim": 32, "scale": 1.0}
    for more, word in (({"chunk": 0}, "chunk"), ({"chunk": 4, "window": 4}, "chunk"), ({"softcap": 0.0}, "cap"),
                       ({"pairing": "thirds"}, "pairing"), ({"bias": ("x",)}, "bias"),
                       ({"unit_norm_after_rotation": 1e-6, "bias": ("q",)}, "biases"),
                       ({"kv_projection": False, "values": "keys"}, "key projection")):
        with pytest.raises(ValueError, match=word):
            Attention(PartSpec("attention", {**base, **more}), torch.float32, "cpu")
    with pytest.raises(ValueError, match="limit"):
        GatedMLP(PartSpec("gated_mlp", {"hidden_size": 8, "intermediate_size": 8, "activation": "clamped"}), torch.float32, "cpu")
    moe = {"hidden_size": 8, "intermediate_size": 8, "experts": 4, "top": 2, "weights": "sigmoid"}
    for more, word in (({"activation": "clamped", "gated": True}, "limit"), ({"activation": "clamped", "limit": 1.0}, "gated"),
                       ({"weigh": "router"}, "weight"), ({"weights": "tanh"}, "weights")):
        with pytest.raises(ValueError, match=word):
            RoutedExperts(PartSpec("routed_experts", {**moe, **more}), torch.float32, "cpu")


# ------------------------------------------------------------------ the plain implementation against closed forms
def test_memory_with_fixed_decays_is_a_weighted_sum_of_past_values():
    t, nh, d, e = 7, 2, 3, 4
    g = torch.Generator().manual_seed(0)
    q, k = torch.randn(t, nh, d, generator=g, dtype=F64), torch.randn(t, nh, d, generator=g, dtype=F64)
    v = torch.randn(t, nh, e, generator=g, dtype=F64)
    decay = [0.7, 1.0]
    out, s = plain.fixed_decay_scan(q, k, v, decay)
    for n in range(t):
        for h in range(nh):
            want = sum(decay[h] ** (n - j) * (q[n, h] @ k[j, h]) * v[j, h] for j in range(n + 1))
            assert torch.allclose(out[n, h], want)
    again, _ = plain.fixed_decay_scan(q[4:], k[4:], v[4:], decay, state=plain.fixed_decay_scan(q[:4], k[:4], v[:4], decay)[1])
    assert torch.allclose(again, out[4:])


def test_chunks_hide_other_chunks_and_a_cap_bounds_the_scores():
    assert [[plain.sees(i, j, 4) for j in range(8)] for i in (3, 4, 7)] == [
        [True] * 4 + [False] * 4, [False] * 4 + [True] + [False] * 3, [False] * 4 + [True] * 4]
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(9, 2, 6, generator=g, dtype=F64) for _ in range(3))
    whole = plain.attend(q, k, v, 1.0, chunk=4)
    for lo in (0, 4, 8):                       # every chunk alone gives the same
        part = plain.attend(q[lo:lo + 4], k[lo:lo + 4], v[lo:lo + 4], 1.0)
        assert torch.allclose(whole[lo:lo + 4], part)
    assert torch.allclose(plain.attend(q, k, v, 0.3, softcap=1e7), plain.attend(q, k, v, 0.3), atol=1e-6)
    tight = plain.attend(q, k, v, 50.0, softcap=1e-6)                          # a tiny cap: all visible keys alike
    assert torch.allclose(tight.view(9, 2, 6)[8], v.mean(0), atol=1e-5)


def test_pairs_of_halves_and_of_neighbours_differ_by_an_order_only():
    rot = models.rotation(8, 100.0)
    x = torch.randn(5, 1, 10, generator=torch.Generator().manual_seed(2), dtype=F64)
    pos = torch.tensor([0, 1, 2, 50, 51])
    order = [0, 2, 4, 6, 1, 3, 5, 7, 8, 9]
    assert torch.allclose(plain.rotate(x, pos, rot, True)[..., order], plain.rotate(x[..., order], pos, rot, False))
    assert torch.equal(plain.rotate(x, pos, rot, True)[..., 8:], x[..., 8:])


def test_clamps_of_the_gated_feed_forward_and_weights_on_the_input():
    w = {"gate": torch.eye(3), "up": torch.eye(3), "down": torch.eye(3)}
    h = torch.tensor([[-9.0, 0.5, 9.0]])
    y = plain.clamped_glu(h.double(), w, "", 2.0)[0]
    want = [(-9 / (1 + math.exp(1.702 * 9))) * (-2 + 1), (0.5 / (1 + math.exp(-1.702 * 0.5))) * 1.5,
            (2 / (1 + math.exp(-1.702 * 2))) * 3]
    assert torch.allclose(y, torch.tensor(want, dtype=F64))
    full = {f"e{e}.{n}": torch.randn(4, 4, generator=torch.Generator().manual_seed(e * 3 + i), dtype=F64)
            for e in range(3) for i, n in enumerate(("gate", "up", "down"))}
    full["router"] = torch.randn(3, 4, generator=torch.Generator().manual_seed(99), dtype=F64)
    m = models.moe(3, 2, 4, limit=0.7)
    x = torch.randn(6, 4, generator=torch.Generator().manual_seed(5), dtype=F64)
    got = plain.experts_ff(x, full, "", m)
    s = torch.sigmoid(x @ full["router"].T)
    for n in range(6):
        best = sorted(range(3), key=lambda e: -float(s[n, e]))[:2]
        want = sum(plain.clamped_glu((s[n, e] * x[n])[None], full, f"e{e}.", 0.7)[0] for e in best)
        assert torch.allclose(got[n], want)


@pytest.mark.parametrize("tag", ["early", "odd"])
def test_the_plain_model_is_causal_and_every_result_reaches_the_average(tag):
    cfg = models.SHAPES[tag]
    w = models.make_tensors(cfg, 4)
    a = models.random_prompts(cfg, [30], seed=1)[0]
    b = list(a)
    b[20] = (a[20] + 1) % cfg["vocab"]
    la, lb = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    assert torch.equal(la[:20], lb[:20]) and (la[20:] - lb[20:]).abs().max() > 1e-6
    n = len(cfg["layers"])
    for j in range(n + 1):                     # only X_j goes into the last average: the output is its norm alone
        w2 = dict(w)
        w2[f"l{n - 1}.dwa"] = torch.eye(n + 1)[j]
        logits, after = plain.model_forward(cfg, w2, a, return_layers=True)
        x0 = w["embed"].double()[a]
        if j == 0:
            assert torch.equal(after[-1], x0)
        assert torch.allclose(logits, plain.dynamic_tanh(after[-1], w, "final.norm") @ w["head"].double().T)
