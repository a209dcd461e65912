"""Small Gesuvik configurations for tests and a writer of model folders of the tests' own.

The shapes differ from one another in everything the configuration can say: the order of the three mixers and which
layers borrow another's weights (also from one that borrows itself); query heads per key head from one to all; value
heads larger, smaller or equal to the key size; rotations over a part, all or none of the head, with and without slowed
pairs; windows from one token to more than a page, in the latent attention unlike the others'; latents wider and
narrower than the values; decays from none to total; 1 to 3 of the experts chosen, with none to more identity experts
than real ones, limits that differ between experts and the shared one; layers without experts; widths that are no
multiple of 8; caps that bite and caps that do not.  Weights are drawn wide enough for attention, gates, clamps and the
router's choice to be far from trivial.
"""

from __future__ import annotations

import copy
import json
import math
import os

import torch


def rotation(dims, base=10000.0, scaling=None):
    """``scaling``: (factor, original, fast, slow) or None."""
    out = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def _finish(m, window, rot):
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = rot
    return m


def attention(heads, kv_heads, dim, vdim, rot, window, scale=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim,
         "scale": scale if scale is not None else 3.0 / math.sqrt(dim)}
    return {"type": "attention", "mixer": _finish(m, window, rot)}


def latent(heads, dim, rot_dim, vdim, kv_rank, window, base=10000.0, scale=None):
    m = {"dim": dim, "heads": heads, "kv_rank": kv_rank, "rot_dim": rot_dim, "vdim": vdim,
         "scale": scale if scale is not None else 3.0 / math.sqrt(dim + rot_dim)}
    return {"type": "latent_attention", "mixer": _finish(m, window, rotation(rot_dim, base))}


def retention(heads, dim, vdim, rot, decay=None):
    m = {"decay": decay if decay is not None else [1.0 - 0.5 ** (h + 2) for h in range(heads)], "dim": dim,
         "heads": heads, "vdim": vdim}
    return {"type": "retention", "mixer": _finish(m, None, rot)}


def moe(experts, identity, top, ff, shared=None, limit=0.8, shared_limit=1.3):
    out = {"expert": {"ff": ff, "limit": limit}, "kind": "moe",
           "router": {"experts": experts, "identity": identity, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared, "limit": shared_limit}
    return out


def config(width, vocab, layers, eps=1e-5, logit_scale=0.7, logit_softcap=4.0):
    """``layers``: (mixer entry, mlp entry or None), or the number of the layer whose weights are used again."""
    made = []
    for entry in layers:
        if isinstance(entry, int):
            src = {k: v for k, v in copy.deepcopy(made[entry]).items() if k != "weights_of"}
            made.append(dict(src, weights_of=entry))
        else:
            made.append(dict(entry[0], mlp=entry[1]))
    return {"architecture": "Gesuvik", "layers": made, "logit_scale": logit_scale, "logit_softcap": logit_softcap,
            "norm": {"eps": eps}, "vocab": vocab, "width": width}


# value heads larger than keys; the latent attention comes back with the same weights, and so does retention
EARLY = config(96, 211, [
    (latent(3, 24, 16, 20, 40, 11), moe(6, 3, 2, 40, 56)),
    (retention(3, 16, 24, rotation(8)), None),
    (attention(4, 2, 20, 28, rotation(8, 500.0, (4.0, 40, 8.0, 1.0)), 9), moe(3, 5, 3, 24, 32, 0.5, 0.9)),
    0,
    1])
# equal sizes, everything rotated, windows around a page; one borrowed from a borrower; no identity experts
FLAT = config(128, 157, [
    (attention(6, 3, 32, 32, rotation(32, 2000.0, (8.0, 256, 16.0, 2.0)), 70), moe(4, 0, 1, 64, 48)),
    (retention(4, 32, 32, rotation(32)), moe(5, 2, 2, 32, 40)),
    (latent(4, 32, 32, 32, 32, 64), moe(4, 1, 2, 48, 32)),
    2,
    3], eps=1e-6, logit_scale=1.0, logit_softcap=30.0)
# a width no product kernel takes; all query heads on one key head; no rotation; windows of one token and none at all
ODD = config(100, 89, [
    (retention(5, 12, 20, None, [0.9, 1.0, 0.0, 0.99, 0.5]), moe(5, 1, 2, 36, 28)),
    (attention(6, 1, 10, 6, None, 5), moe(2, 6, 2, 20, 12)),
    (latent(2, 12, 6, 28, 10, 1), moe(3, 1, 3, 12, 20)),
    (attention(3, 3, 20, 20, rotation(10, 1e6, (2.0, 100, 4.0, 1.0)), None), None),
    (latent(5, 20, 10, 12, 70, 33), None),
    1], eps=1e-4, logit_scale=1.3, logit_softcap=3.0)
# heads of 64 and 128: the kernels on tcgen05 and those fed by TMA; more shared and identity experts
WIDE = config(256, 301, [
    (attention(8, 2, 128, 128, rotation(64, 1e5, (4.0, 512, 32.0, 1.0)), 130), moe(7, 9, 3, 64, 96)),
    (retention(4, 64, 128, rotation(64, 1e6)), moe(9, 2, 2, 48, 64)),
    (attention(4, 4, 64, 64, rotation(64), 96), None),
    (latent(8, 64, 64, 96, 160, 100, 1e5), moe(4, 4, 1, 32, 64)),
    (retention(2, 128, 40, rotation(128)), moe(4, 1, 4, 32, 128)),
    0], logit_softcap=9.0)

SHAPES = {"early": EARLY, "flat": FLAT, "odd": ODD, "wide": WIDE}


def tensor_shapes(cfg):
    w, v = cfg["width"], cfg["vocab"]
    shapes = {"embed": (v, w), "head": (v, w), "final.norm": (w,)}

    def glu(p, ff):
        shapes.update({p + "gate": (ff, w), p + "up": (ff, w), p + "down": (w, ff)})

    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, mlp, p = layer["mixer"], layer["mlp"], f"l{i}."
        q = p + "mix."
        h, d, e = m["heads"], m["dim"], m["vdim"]
        shapes.update({p + "norm1": (w,), q + "o": (w, h * e)})
        if layer["type"] == "attention":
            g = m["kv_heads"]
            shapes.update({q + "q": (h * d, w), q + "k": (g * d, w), q + "v": (g * e, w), q + "q.norm": (h * d,),
                           q + "k.norm": (g * d,), q + "sink": (h,)})
        elif layer["type"] == "latent_attention":
            r, c = m["rot_dim"], m["kv_rank"]
            shapes.update({q + "q": (h * (d + r), w), q + "dkv": (c + r, w), q + "dkv.norm": (c,), q + "uk": (h * d, c),
                           q + "uv": (h * e, c), q + "sink": (h,), q + "g": (h, w)})
        else:
            shapes.update({q + "q": (h * d, w), q + "k": (h * d, w), q + "v": (h * e, w), q + "g": (h * e, w)})
        if mlp is None:
            continue
        n = mlp["router"]["experts"]
        routed = n + mlp["router"]["identity"]
        shapes.update({p + "norm2": (w,), p + "mlp.router": (routed, w), p + "mlp.correction": (routed,)})
        for x in range(n):
            glu(f"{p}mlp.e{x}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            glu(p + "mlp.shared.", mlp["shared"]["ff"])
    return shapes


def make_tensors(cfg, seed, dtype=torch.bfloat16):
    """Matrices N(0, 1/in), routers three times as wide; norm weights around 1; sinks of both signs; corrections as large
    as the scores they join."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in sorted(tensor_shapes(cfg).items()):
        t = torch.randn(shape, generator=g, dtype=torch.float32)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.2 * t
        elif last == "correction":
            t = 0.3 * t
        elif last == "sink":
            t = 1.5 * t
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
