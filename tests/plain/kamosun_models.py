"""Small Kamosun configurations for tests and a writer of model folders of the tests' own.

The shapes differ from one another in everything the configuration can say: the order of the two kinds of mixer;
attention with value heads larger, smaller or equal to the key size, one to all key heads per query head, rotations
over a part, all or none of the head, with and without slowed wavelengths, chunks from a few tokens to more than a
page or no mask, keys of an earlier layer read under a smaller or larger chunk; soft caps; fixed decays from strong to
none, unlike key and value sizes; dense feed-forwards, experts with 1 to 3 chosen, with and without a shared one,
and none at all; widths that are no multiple of 8; multipliers of 1 and others.  Weights are drawn wide enough for
attention, gates and clamps to be far from trivial.
"""

from __future__ import annotations

import json
import math
import os

import torch


def rotation(dims, base=10000.0, scaling=None):
    """``scaling``: (factor, low, high, original) or None."""
    out = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return out


def _heads(heads, kv_heads, dim, vdim, rot, scale):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim,
         "scale": scale if scale is not None else 3.0 / math.sqrt(dim)}
    if rot is not None:
        m["rot"] = rot
    return m


def attention(heads, kv_heads, dim, vdim, rot, chunk, kv_from=None, scale=None):
    m = _heads(heads, kv_heads, dim, vdim, rot, scale)
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def left(heads, kv_heads, dim, vdim, rot, softcap, scale=None):
    return dict(_heads(heads, kv_heads, dim, vdim, rot, scale), softcap=softcap)


def right(heads, dim, vdim, decay=None):
    return {"decay": decay if decay is not None else [1.0 - 0.5 ** (h + 1) for h in range(heads)], "dim": dim,
            "heads": heads, "vdim": vdim}


def parallel(left_record, right_record):
    return {"type": "parallel", "mixer": {"left": left_record, "right": right_record}}


def dense(ff, limit=1.1):
    return {"ff": ff, "kind": "dense", "limit": limit}


def moe(experts, top, ff, shared=None, limit=0.8, shared_limit=1.3):
    out = {"expert": {"ff": ff, "limit": limit}, "kind": "moe", "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared, "limit": shared_limit}
    return out


def config(width, vocab, layers, eps=1e-5, residual_mult=0.6):
    """``layers``: (mixer entry, mlp entry or None) pairs."""
    return {"architecture": "Kamosun", "layers": [dict(m, mlp=f) for m, f in layers], "norm": {"eps": eps},
            "residual_mult": residual_mult, "vocab": vocab, "width": width}


# value heads larger and smaller than keys; a layer without feed-forward; keys read under a larger chunk than
# the layer that stores them has
EARLY = config(96, 211, [
    (parallel(left(4, 2, 24, 40, rotation(16, 500.0, (4.0, 1.0, 3.0, 40)), 8.0), right(3, 16, 24)), moe(6, 2, 40, 56)),
    (attention(6, 2, 20, 28, rotation(8), 9), None),
    (attention(4, 2, 20, 28, rotation(8), 17, kv_from=1), dense(72)),
    (parallel(left(3, 3, 16, 12, rotation(16), 30.0), right(2, 24, 8, [1.0, 0.3])), dense(40, 0.5))])
# equal key and value sizes, everything rotated, chunks around a page; dense only; a multiplier of 1
FLAT = config(128, 157, [
    (attention(3, 3, 32, 32, rotation(32, 2000.0), 70), dense(64)),
    (parallel(left(4, 4, 32, 32, rotation(32), 15.0), right(4, 32, 32)), dense(48)),
    (attention(6, 3, 32, 32, rotation(32, 2000.0), 64, kv_from=0), dense(88))], eps=1e-6, residual_mult=1.0)
# a width no product kernel takes; all query heads on one key head; no rotation, no mask; experts without a shared one
ODD = config(100, 89, [
    (attention(6, 1, 20, 20, None, None), moe(5, 1, 36)),
    (parallel(left(5, 1, 12, 20, None, 3.0), right(3, 12, 20, [0.9, 0.99, 0.0])), moe(3, 3, 20, 28)),
    (attention(2, 1, 20, 20, None, 33, kv_from=0), dense(44)),
    (attention(4, 4, 12, 8, rotation(6, 1e6), 5), None)], eps=1e-4, residual_mult=1.7)
# heads of 128 and 64, fully rotated: the products with fused epilogues and the kernels fed by TMA
WIDE = config(256, 301, [
    (parallel(left(8, 4, 128, 128, rotation(128, 2e5, (8.0, 1.0, 4.0, 64)), 25.0), right(4, 64, 32)), moe(7, 3, 64, 96)),
    (attention(4, 2, 128, 128, rotation(128, 1e5), 130), moe(9, 2, 48, 64)),
    (attention(8, 2, 128, 128, rotation(128, 1e5), 50, kv_from=1), dense(192)),
    (attention(4, 4, 64, 64, rotation(64), 96), moe(4, 1, 32)),
    (parallel(left(4, 4, 64, 64, rotation(32), 60.0), right(2, 128, 64)), dense(64))], residual_mult=0.8)

SHAPES = {"early": EARLY, "flat": FLAT, "odd": ODD, "wide": WIDE}


def tensor_shapes(cfg):
    w, v = cfg["width"], cfg["vocab"]
    shapes = {"embed": (v, w), "head": (v, w)}

    def norm(name):
        shapes.update({name: (w,), name + ".alpha": (), name + ".b": (w,)})

    def glu(p, ff):
        shapes.update({p + "gate": (ff, w), p + "up": (ff, w), p + "down": (w, ff)})

    def heads(p, m, biased):
        h, g, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        own = m.get("kv_from") is None
        shapes.update({p + "q": (h * d, w), p + "q.norm": (d,), p + "o": (w, h * e)})
        if own:
            shapes.update({p + "k": (g * d, w), p + "k.norm": (d,), p + "v": (g * e, w)})
        if biased:
            shapes.update({p + "q.b": (h * d,), p + "o.b": (w,)})
            if own:
                shapes.update({p + "k.b": (g * d,), p + "v.b": (g * e,)})

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        m, mlp, p = layer["mixer"], layer["mlp"], f"l{i}."
        norm(p + "norm1")
        shapes.update({p + "rg1": (w, w), p + "rg1.b": (w,), p + "dwa": (i + 2,)})
        if layer["type"] == "attention":
            heads(p + "mix.", m, True)
        else:
            heads(p + "mix.left.", m["left"], False)
            r, q = m["right"], p + "mix.right."
            h, d, e = r["heads"], r["dim"], r["vdim"]
            shapes.update({q + "q": (h * d, w), q + "k": (h * d, w), q + "v": (h * e, w), q + "g": (h * e, w),
                           q + "norm": (h * e,), q + "o": (w, h * e), p + "mix.left.out": (w,), p + "mix.right.out": (w,)})
        if mlp is None:
            continue
        norm(p + "norm2")
        shapes.update({p + "rg2": (w, w), p + "rg2.b": (w,)})
        if mlp["kind"] == "dense":
            glu(p + "mlp.", mlp["ff"])
            continue
        shapes[p + "mlp.router"] = (mlp["router"]["experts"], w)
        for e in range(mlp["router"]["experts"]):
            glu(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            glu(p + "mlp.shared.", mlp["shared"]["ff"])
    return shapes


def make_tensors(cfg, seed, dtype=torch.bfloat16):
    """Matrices N(0, 1/in), routers three times as wide; norm weights around 1, shifts and biases a few tenths, the
    norms' alpha between a half and one and a half; averages over the depth of both signs."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in sorted(tensor_shapes(cfg).items()):
        t = torch.randn(shape, generator=g, dtype=torch.float32)
        last = name.rsplit(".", 1)[-1]
        if last == "alpha":
            t = 0.5 + torch.sigmoid(t)
        elif last == "b":
            t = 0.3 * t
        elif last in ("norm", "norm1", "norm2") or name.endswith(("left.out", "right.out")):
            t = 1.0 + 0.2 * t
        elif last == "dwa":
            t = 0.3 * t
            t[-1] += 0.8
        elif last == "router":
            t = t * (3.0 / math.sqrt(shape[-1]))
        elif name != "embed":
            t = t / math.sqrt(shape[-1])
        out[name] = t.to(dtype)
    return out


def write_folder(folder, cfg, tensors):
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(folder, "model.safetensors"))
    return folder


def random_prompts(cfg, lengths, seed):
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in lengths]
