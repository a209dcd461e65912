"""A plain, slow implementation of the Kamosun decoder in 64-bit, one function per mechanism.

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


def dynamic_tanh(x, w, name):
    """tanh(alpha x) w + b, alpha one number, w and b vectors."""
    alpha, gain, shift = w[name + ".alpha"].to(F64), w[name].to(F64), w[name + ".b"].to(F64)
    return torch.tanh(alpha * x) * gain + shift


def silu(z):
    return z * torch.sigmoid(z)


def project(h, w, name):
    """W h, plus the bias if the file has one."""
    y = h @ w[name].to(F64).T
    return y + w[name + ".b"].to(F64) if name + ".b" in w else y


# ----------------------------------------------------------------------------- rotations
def frequencies(rot):
    """Angle per position of every rotated pair; with ``scaling`` long wavelengths turn slower."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        s = rot.get("scaling")
        if s:
            factor, low, high, original = (float(s[k]) for k in ("factor", "low", "high", "original"))
            wavelength = 2.0 * math.pi / f
            if wavelength > original / low:
                f = f / factor
            elif wavelength >= original / high:
                blend = (original / wavelength - low) / (high - low)
                f = (1.0 - blend) * f / factor + blend * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate(x, positions, rot, neighbours):
    """x [T, heads, d]; pairs (2i, 2i+1) if ``neighbours`` else (i, i + dims/2) of the first dims values."""
    if not rot or not int(rot["dims"]):
        return x
    dims = int(rot["dims"])
    ang = positions.to(F64)[:, None] * frequencies(rot)[None, :]
    c, s = ang.cos()[:, None, :], ang.sin()[:, None, :]
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
def sees(i, j, chunk):
    """Position i sees j: earlier or equal, and in the same chunk when there are chunks."""
    return j <= i and (chunk is None or i // chunk == j // chunk)


def attend(q, k, v, scale, chunk=None, softcap=None):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H * e]."""
    t, nh, _ = q.shape
    per = nh // k.shape[1]
    mask = torch.tensor([[sees(i, j, chunk) for j in range(t)] for i in range(t)])
    heads = []
    for h in range(nh):
        s = (q[:, h] @ k[:, h // per].T) * scale
        if softcap is not None:
            s = softcap * torch.tanh(s / softcap)
        heads.append(torch.softmax(s.masked_fill(~mask, float("-inf")), -1) @ v[:, h // per])
    return torch.stack(heads, 1).reshape(t, -1)


def make_queries(h, w, p, m, eps, positions, neighbours):
    q = project(h, w, p + "q").view(h.shape[0], int(m["heads"]), int(m["dim"]))
    return rotate(rms_unit(q, eps) * w[p + "q.norm"].to(F64), positions, m.get("rot"), neighbours)


def make_keys_values(h, w, p, m, eps, positions, neighbours):
    t, g = h.shape[0], int(m["kv_heads"])
    k = rms_unit(project(h, w, p + "k").view(t, g, int(m["dim"])), eps) * w[p + "k.norm"].to(F64)
    return rotate(k, positions, m.get("rot"), neighbours), project(h, w, p + "v").view(t, g, int(m["vdim"]))


def attention_mixer(h, w, p, m, eps, positions, kept, layer):
    """Chunked attention with biases; ``kept`` holds every layer's keys and values for those that borrow."""
    if m.get("kv_from") is None:
        kept[layer] = make_keys_values(h, w, p, m, eps, positions, neighbours=False)
        k, v = kept[layer]
    else:
        k, v = kept[int(m["kv_from"])]
    q = make_queries(h, w, p, m, eps, positions, neighbours=False)
    mask = m.get("mask") or {}
    o = attend(q, k, v, float(m["scale"]), chunk=mask.get("size"))
    return project(o, w, p + "o")


def capped_attention(h, w, p, m, eps, positions):
    """The left mixer of a pair: neighbouring pairs turn, scores pass a soft cap, every earlier key is seen."""
    k, v = make_keys_values(h, w, p, m, eps, positions, neighbours=True)
    q = make_queries(h, w, p, m, eps, positions, neighbours=True)
    return project(attend(q, k, v, float(m["scale"]), softcap=float(m["softcap"])), w, p + "o")


# ----------------------------------------------------------------------------- lightning attention
def fixed_decay_scan(q, k, v, decay, state=None):
    """Per head S <- decay_h S + k v^T, o = S^T q.  q, k [T, H, d]; v [T, H, e]; S [H, d, e] from zero."""
    t, nh, d = q.shape
    e = v.shape[-1]
    s = torch.zeros(nh, d, e, dtype=F64) if state is None else state.clone()
    out = torch.zeros(t, nh, e, dtype=F64)
    lam = torch.as_tensor(decay, dtype=F64)[:, None, None]
    for n in range(t):
        s = lam * s + k[n][:, :, None] * v[n][:, None, :]
        out[n] = (s * q[n][:, :, None]).sum(1)
    return out, s


def lightning_mixer(h, w, p, m, eps):
    t, nh, d, e = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(project(h, w, p + "q")).view(t, nh, d)
    k = silu(project(h, w, p + "k")).view(t, nh, d)
    v = silu(project(h, w, p + "v")).view(t, nh, e)
    o, _ = fixed_decay_scan(q, k, v, m["decay"])
    o = rms_unit(o.reshape(t, nh * e), eps) * w[p + "norm"].to(F64)
    return project(o * torch.sigmoid(project(h, w, p + "g")), w, p + "o")


def side_by_side(h, w, p, m, eps, positions):
    """Half the sum of both results, each normed over the width with a gain of its own."""
    left = capped_attention(h, w, p + "left.", m["left"], eps, positions)
    right = lightning_mixer(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms_unit(left, eps) * w[p + "left.out"].to(F64) + rms_unit(right, eps) * w[p + "right.out"].to(F64))


# ----------------------------------------------------------------------------- feed-forward
def clamped_glu(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].to(F64).T, max=limit)
    u = torch.clamp(h @ w[p + "up"].to(F64).T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].to(F64).T


def choose(h, w, p, m):
    """Experts of every token and their weights: the largest sigmoid scores, as they are."""
    s = torch.sigmoid(h @ w[p + "router"].to(F64).T)
    weight, expert = s.topk(int(m["router"]["top"]), dim=-1)
    return expert, weight


def experts_ff(h, w, p, m):
    """Each chosen expert runs on its weight times the input; the shared one on the input itself."""
    out = torch.zeros_like(h)
    expert, weight = choose(h, w, p, m)
    for n in range(h.shape[0]):
        for e, s in zip(expert[n].tolist(), weight[n]):
            out[n] += clamped_glu((s * h[n])[None], w, f"{p}e{e}.", float(m["expert"]["limit"]))[0]
    if m.get("shared"):
        out = out + clamped_glu(h, w, p + "shared.", float(m["shared"]["limit"]))
    return out


def feed_forward(h, w, p, m):
    return clamped_glu(h, w, p, float(m["limit"])) if m["kind"] == "dense" else experts_ff(h, w, p, m)


# ----------------------------------------------------------------------------- layer, model
def residual_gate(h, w, name):
    return torch.sigmoid(h @ w[name].to(F64).T + w[name + ".b"].to(F64))


def layer_result(x, config, w, i, positions, kept):
    """x + m (gate1 * mixer(norm1 x) + gate2 * ff(norm2 x)), before the average over the depth."""
    spec = config["layers"][i]
    eps, mult = float(config["norm"]["eps"]), float(config["residual_mult"])
    p = f"l{i}."
    h = dynamic_tanh(x, w, p + "norm1")
    if spec["type"] == "attention":
        y = attention_mixer(h, w, p + "mix.", spec["mixer"], eps, positions, kept, i)
    elif spec["type"] == "parallel":
        y = side_by_side(h, w, p + "mix.", spec["mixer"], eps, positions)
    else:
        raise ValueError(spec["type"])
    total = residual_gate(h, w, p + "rg1") * y
    if spec.get("mlp") is not None:
        h = dynamic_tanh(x, w, p + "norm2")
        total = total + residual_gate(h, w, p + "rg2") * feed_forward(h, w, p + "mlp.", spec["mlp"])
    return x + mult * total


def depth_average(history, weights):
    """sum_j weights[j] * history[j] over the embedding output and every layer's result so far."""
    out = torch.zeros_like(history[0])
    for j, x in enumerate(history):
        out = out + float(weights[j]) * x
    return out


def model_forward(config, w, tokens, return_layers=False):
    tokens = list(tokens)
    positions = torch.arange(len(tokens))
    x = w["embed"].to(F64)[tokens]
    history, after, kept = [x], [], {}
    for i in range(len(config["layers"])):
        history.append(layer_result(x, config, w, i, positions, kept))
        x = depth_average(history, w[f"l{i}.dwa"].to(F64).reshape(-1))
        after.append(x.clone())
    logits = dynamic_tanh(x, w, "final.norm") @ w["head"].to(F64).T
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
