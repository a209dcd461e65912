"""A plain, slow implementation of the Gesuvik decoder in 64-bit, one function per mechanism.

Written from the design's equations, token by token where the design is a recurrence; it shares
no code with ``enginekernel_b200``.  ``weights`` is a dict name -> tensor (any float dtype),
``config`` the parsed ``config.json``.  Everything is computed in float64 on the CPU, for ONE
sequence whose positions count from 0.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


# ----------------------------------------------------------------------------- small pieces
def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, name, eps):
    return rms_unit(x, eps) * w[name].to(F64)


def silu(z):
    return z * torch.sigmoid(z)


def project(h, w, name):
    return h @ w[name].to(F64).T


# ----------------------------------------------------------------------------- rotations
def rotation_speeds(rot):
    """(angle per position of every rotated pair, factor on cosines and sines); ``scaling`` makes slow pairs slower."""
    dims, base = int(rot["dims"]), float(rot["base"])
    speeds = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(speeds, dtype=F64), 1.0
    factor, original = float(s["factor"]), float(s["original"])

    def place(turns):                       # the pair (as a real number) that turns `turns` times over `original`
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(float(s["fast"]))), 0)
    hi = min(math.ceil(place(float(s["slow"]))), dims - 1)
    for i, f in enumerate(speeds):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        speeds[i] = f / factor * ramp + f * (1.0 - ramp)
    return torch.tensor(speeds, dtype=F64), 0.1 * math.log(factor) + 1.0


def rotate(x, positions, rot, neighbours):
    """x [T, heads, d]; pairs (2i, 2i+1) if ``neighbours`` else (i, i + dims/2) of the first dims values."""
    if not rot or not int(rot["dims"]):
        return x
    dims = int(rot["dims"])
    speeds, factor = rotation_speeds(rot)
    ang = positions.to(F64)[:, None] * speeds[None, :]
    c, s = factor * ang.cos()[:, None, :], factor * ang.sin()[:, None, :]
    out = x.clone()
    if neighbours:
        first, second = slice(0, dims, 2), slice(1, dims, 2)
    else:
        first, second = slice(0, dims // 2), slice(dims // 2, dims)
    u, v = x[..., first], x[..., second]
    out[..., first] = u * c - v * s
    out[..., second] = v * c + u * s
    return out


# ----------------------------------------------------------------------------- attention
def sees(i, j, window):
    """Position i sees itself and the window - 1 positions before it."""
    return 0 <= i - j and (window is None or i - j < window)


def attend(q, k, v, scale, window, sinks):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; exp(sink_h) joins every denominator of head h."""
    t, nh, _ = q.shape
    per = nh // k.shape[1]
    mask = torch.tensor([[sees(i, j, window) for j in range(t)] for i in range(t)])
    heads = []
    for h in range(nh):
        s = ((q[:, h] @ k[:, h // per].T) * scale).masked_fill(~mask, float("-inf"))
        with_sink = torch.cat([s, torch.full((t, 1), float(sinks[h]), dtype=F64)], 1)
        heads.append(torch.softmax(with_sink, -1)[:, :t] @ v[:, h // per])
    return torch.stack(heads, 1)


def make_queries_keys_values(h, w, p, m, eps, positions):
    """Queries and keys normed over the whole projection, then cut into heads and rotated."""
    t, nh, g, d, e = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_norm(project(h, w, p + "q"), w, p + "q.norm", eps).view(t, nh, d)
    k = rms_norm(project(h, w, p + "k"), w, p + "k.norm", eps).view(t, g, d)
    v = project(h, w, p + "v").view(t, g, e)
    return rotate(q, positions, m.get("rot"), False), rotate(k, positions, m.get("rot"), False), v


def window_of(m):
    return (m.get("mask") or {}).get("size")


def attention_mixer(h, w, p, m, eps, positions):
    q, k, v = make_queries_keys_values(h, w, p, m, eps, positions)
    o = attend(q, k, v, float(m["scale"]), window_of(m), w[p + "sink"].to(F64))
    return project(o.reshape(h.shape[0], -1), w, p + "o")


def latent_queries_keys_values(h, w, p, m, eps, positions):
    """(q, k [T, H, dim + rot_dim], v [T, H, vdim]): keys and values spelled out per head from the latent."""
    t, nh, d, r, e, c = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    rot = m.get("rot")
    q = project(h, w, p + "q").view(t, nh, d + r)
    q = torch.cat([q[..., :d], rotate(q[..., d:], positions, rot, True)], -1)
    down = project(h, w, p + "dkv")
    latent = rms_norm(down[:, :c], w, p + "dkv.norm", eps)
    turned = rotate(down[:, c:].view(t, 1, r), positions, rot, True)
    k = torch.cat([project(latent, w, p + "uk").view(t, nh, d), turned.expand(t, nh, r)], -1)
    return q, k, project(latent, w, p + "uv").view(t, nh, e)


def latent_mixer(h, w, p, m, eps, positions):
    q, k, v = latent_queries_keys_values(h, w, p, m, eps, positions)
    o = attend(q, k, v, float(m["scale"]), window_of(m), w[p + "sink"].to(F64))
    o = o * torch.sigmoid(project(h, w, p + "g"))[:, :, None]
    return project(o.reshape(h.shape[0], -1), w, p + "o")


# ----------------------------------------------------------------------------- retention
def retention_scan(q, k, v, decay, state=None):
    """Per head S <- decay_h S + k v^T, o = S^T q.  q, k [T, H, d]; v [T, H, e]; S [H, d, e] from zero."""
    t, nh, d = q.shape
    s = torch.zeros(nh, d, v.shape[-1], dtype=F64) if state is None else state.clone()
    out = torch.zeros(t, nh, v.shape[-1], dtype=F64)
    keep = torch.as_tensor(decay, dtype=F64)[:, None, None]
    for n in range(t):
        s = keep * s + k[n][:, :, None] * v[n][:, None, :]
        out[n] = (s * q[n][:, :, None]).sum(1)
    return out, s


def retention_mixer(h, w, p, m, eps, positions):
    t, nh, d, e = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate(project(h, w, p + "q").view(t, nh, d), positions, m.get("rot"), False)
    k = rotate(project(h, w, p + "k").view(t, nh, d), positions, m.get("rot"), False) / math.sqrt(d)
    o, _ = retention_scan(q, k, project(h, w, p + "v").view(t, nh, e), m["decay"])
    return project(rms_unit(o, eps).reshape(t, nh * e) * silu(project(h, w, p + "g")), w, p + "o")


# ----------------------------------------------------------------------------- feed-forward
def clamped_glu(h, w, p, limit):
    g = torch.clamp(project(h, w, p + "gate"), max=limit)
    u = torch.clamp(project(h, w, p + "up"), min=-limit, max=limit)
    return project(g * torch.sigmoid(1.702 * g) * (u + 1.0), w, p + "down")


def choose(h, w, p, m):
    """(experts, weights) of every token: the largest corrected scores choose, the bare scores weigh."""
    s = torch.softmax(project(h, w, p + "router"), -1)
    expert = (s + w[p + "correction"].to(F64)).topk(int(m["router"]["top"]), dim=-1).indices
    return expert, s.gather(1, expert)


def experts_ff(h, w, p, m):
    """Chosen experts' outputs times their weights; numbers past the experts' count name the input itself."""
    n_experts = int(m["router"]["experts"])
    out = torch.zeros_like(h)
    expert, weight = choose(h, w, p, m)
    for n in range(h.shape[0]):
        for e, s in zip(expert[n].tolist(), weight[n]):
            y = h[n] if e >= n_experts else clamped_glu(h[n][None], w, f"{p}e{e}.", float(m["expert"]["limit"]))[0]
            out[n] += s * y
    if m.get("shared"):
        out = out + clamped_glu(h, w, p + "shared.", float(m["shared"]["limit"]))
    return out


# ----------------------------------------------------------------------------- layer, model
MIXERS = {"attention": attention_mixer, "latent_attention": latent_mixer, "retention": retention_mixer}


def owner(config, i):
    """The layer whose tensors layer ``i`` uses."""
    while config["layers"][i].get("weights_of") is not None:
        i = int(config["layers"][i]["weights_of"])
    return i


def layer(x, config, w, i, positions):
    spec, eps, p = config["layers"][i], float(config["norm"]["eps"]), f"l{owner(config, i)}."
    x = x + MIXERS[spec["type"]](rms_norm(x, w, p + "norm1", eps), w, p + "mix.", spec["mixer"], eps, positions)
    if spec.get("mlp") is not None:
        x = x + experts_ff(rms_norm(x, w, p + "norm2", eps), w, p + "mlp.", spec["mlp"])
    return x


def cap(z, limit):
    return limit * torch.tanh(z / limit)


def model_forward(config, w, tokens, return_layers=False):
    tokens = list(tokens)
    positions = torch.arange(len(tokens))
    x = w["embed"].to(F64)[tokens]
    after = []
    for i in range(len(config["layers"])):
        x = layer(x, config, w, i, positions)
        after.append(x.clone())
    z = rms_norm(x, w, "final.norm", float(config["norm"]["eps"])) @ w["head"].to(F64).T
    logits = cap(z * float(config["logit_scale"]), float(config["logit_softcap"]))
    return (logits, after) if return_layers else logits


def forward(config, w, tokens):
    """Logits [T, vocab] of one sequence."""
    return model_forward(config, w, tokens)


def greedy(config, w, tokens, n_new):
    """``n_new`` tokens by arg-max, the whole sequence run again for each (slow and plain)."""
    seq, out = list(tokens), []
    for _ in range(n_new):
        nxt = int(model_forward(config, w, seq)[-1].argmax())
        out.append(nxt)
        seq.append(nxt)
    return out
