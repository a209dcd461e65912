"""The Kamosun decoder in the engine against the plain implementation, mechanism by mechanism and then whole models
under every way of cutting the work.

Part one drives the new kernels and options alone: the dynamic tanh for one and two readers, the join of two gated
results with the average over the depth, attention within chunks and under a soft cap in all five attention
kernels (one key made to stand out at every edge), biases before the head norm in the wide prepare kernel, the
memory with fixed decays from a carried state with its gated output norm, clamped gates in every product that has
them, the sigmoid router and experts that weigh their input.  Part two runs one-mixer models, and part three four
small models of unlike shapes (tests/plain/kamosun_models.py) through ``Engine``: whole prompts, prompts in portions
down to two tokens, token-by-token decoding, unequal batches, slots, pages and states used again, long decoding, and
greedy generation through the scheduler.
"""

import json

import pytest
import torch

from tests import helpers
from tests.plain import kamosun_models as models
from tests.plain import kamosun_plain as plain
from tests.test_kernels_gpu import DEV, DTYPES, TOL, K, Pages, rel, rnd

pytestmark = pytest.mark.gpu
F32, F64, BF16 = torch.float32, torch.float64, torch.bfloat16


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ===================================================================== mechanisms alone
def _tanh_norm(width, seed):
    return (torch.tensor([0.4 + 0.3 * seed], device=DEV), 1 + 0.2 * rnd(width, seed=10 + seed), 0.3 * rnd(width, seed=20 + seed))


def _apply(norm, x):
    alpha, w, b = (t.double().cpu() for t in norm)
    return torch.tanh(alpha * x) * w + b


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width", [(1, 40), (17, 90), (5, 96), (33, 2560), (3, 1001)])
def test_dynamic_tanh_for_one_and_two_readers(dtype, rows, width):
    k = K()
    stream, add = rnd(rows, width, seed=1, scale=3.0), rnd(rows, width, dtype=dtype, seed=2)
    n1, n2 = _tanh_norm(width, 1), _tanh_norm(width, 2)
    x = stream.double().cpu()
    y, z = (torch.full((rows, width), 7.0, dtype=dtype, device=DEV) for _ in range(2))
    k.dynamic_tanh(y, stream, n1)
    assert rel(y, _apply(n1, x)) <= TOL[dtype]
    k.dynamic_tanh(y, stream, n1, z, n2)
    assert rel(y, _apply(n1, x)) <= TOL[dtype] and rel(z, _apply(n2, x)) <= TOL[dtype]
    s = stream.clone()
    k.dynamic_tanh(y, s, n2, add=add, write_back=False)
    assert torch.equal(s, stream) and rel(y, _apply(n2, x + add.double().cpu())) <= TOL[dtype]
    k.dynamic_tanh(y, s, n2, add=add)
    assert rel(s, x + add.double().cpu()) <= 1e-6
    pick = i32([rows - 1, 0, rows // 2])
    got = torch.empty(3, width, dtype=dtype, device=DEV)
    k.dynamic_tanh(got, stream, n1, add=add, rows=pick, write_back=False)
    assert rel(got, _apply(n1, x + add.double().cpu())[pick.long().cpu()]) <= TOL[dtype]
    if dtype == BF16:                          # the 16-bit form's tanh keeps small and large arguments
        tiny = torch.linspace(-30, 30, width, device=DEV)[None] * torch.tensor([[1e-3], [1.0]], device=DEV)
        one = (torch.ones(1, device=DEV), torch.ones(width, device=DEV), torch.zeros(width, device=DEV))
        out = torch.empty(2, width, dtype=dtype, device=DEV)
        k.dynamic_tanh(out, tiny.contiguous(), one)
        assert ((out.double() - torch.tanh(tiny.double())).abs() <= 2 ** -8 * torch.tanh(tiny.double()).abs() + 1e-6).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width", [(1, 40), (9, 90), (400, 96), (3, 2560), (2, 4100)])
def test_join_of_gated_results_and_average_over_the_depth(dtype, rows, width):
    """Layers in a row from the same history: one with a bias on its result, one with a pair of normed results,
    one without a second sublayer, with readers and without; the history holds every result, the stream the
    average, and the embedding output stays untouched."""
    k = K()
    mult, layers = 0.7, 5
    first = rnd(rows, width, seed=1, scale=2.0)
    keep_first = first.clone()
    kept = torch.full((layers - 1, rows + 2, width), 9.0, device=DEV)
    buffer = torch.empty(rows, width, device=DEV)
    x = first
    history, xr = [first.double().cpu()], first.double().cpu()
    unit = lambda t, eps: t / torch.sqrt((t * t).mean(-1, keepdim=True) + eps)
    d = lambda t: t.double().cpu()
    for n in range(1, layers + 1):
        a, f, za, zf, b = (rnd(rows, width, dtype=dtype, seed=100 * n + i, scale=1.5) for i in range(5))
        ba, bf, bias, ga, gb = (rnd(width, seed=100 * n + 10 + i) for i in range(5))
        depth = rnd(n + 1, seed=100 * n + 50)
        depth[-1] += 1
        use_pair, use_bias, use_f, readers = n in (2, 5), n in (1, 3), n != 3, n % 3
        m = d(a)
        if use_bias:
            m = m + d(bias)
        if use_pair:
            m = 0.5 * (unit(d(a), 1e-5) * d(ga) + unit(d(b), 1e-5) * d(gb))
        r = torch.sigmoid(d(za) + d(ba)) * m
        if use_f:
            r = r + torch.sigmoid(d(zf) + d(bf)) * d(f)
        history.append(xr + mult * r)
        xr = sum(float(depth[j]) * h for j, h in enumerate(history))
        n1, n2 = _tanh_norm(width, 1), _tanh_norm(width, 2)
        y1 = torch.empty(rows, width, dtype=dtype, device=DEV) if readers >= 1 else None
        y2 = torch.empty(rows, width, dtype=dtype, device=DEV) if readers >= 2 else None
        k.depth_join(buffer, x, first, kept, n, depth, mult, a, (za, ba), f=f if use_f else None,
                     gate_f=(zf, bf) if use_f else None, bias_a=bias if use_bias else None,
                     pair=(b, ga, gb, 1e-5, 0.5) if use_pair else None, keep=n < layers, y1=y1,
                     norm1=n1 if y1 is not None else None, y2=y2, norm2=n2 if y2 is not None else None, n_rows=rows)
        x = buffer
        assert rel(x, xr) <= 2e-6 * n, n
        if n < layers:
            assert rel(kept[n - 1, :rows], history[n]) <= 2e-6 * n and (kept[n - 1, rows:] == 9.0).all()
        for y, norm in ((y1, n1), (y2, n2)):
            assert y is None or rel(y, _apply(norm, xr)) <= TOL[dtype]
    assert torch.equal(first, keep_first)


def _plain_row(q, keys, values, pos, scale, chunk, cap):
    """One token's heads against the keys it sees, in 64-bit: q [H, d], keys and values [n, G, d]."""
    nh, g = q.shape[0], keys.shape[1]
    idx = [j for j in range(pos + 1) if plain.sees(pos, j, chunk)]
    kk = keys[idx].double().cpu().repeat_interleave(nh // g, 1)
    vv = values[idx].double().cpu().repeat_interleave(nh // g, 1)
    s = torch.einsum("hd,khd->hk", q.double().cpu(), kk) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    return torch.einsum("hk,khd->hd", torch.softmax(s, -1), vv).reshape(-1)


def _kernels_for(dtype, d, nq, nkv):
    k = K()
    out = ["generic", "generic_split"]
    if k.attention_prefill_supported(dtype, d, nq, nkv):
        out.append("prefill")
    if dtype == BF16 and k.attention_prefill_tc_supported(dtype, d, nq, nkv):
        out.append("prefill_tc")
    if k.attention_decode_supported(dtype, d):
        out += ["decode", "decode_split"]
    if dtype == BF16 and k.attention_decode_tma_supported(dtype, d, nq, nkv):
        out += ["decode_tma", "decode_tma_split"]
    return out


def _attend(which, q, pos, pages, nq, nkv, d, scale, chunk, cap):
    """Rows of ``q`` at positions ``pos`` of slot 1 through one of the kernels (prompt kernels: consecutive positions)."""
    k = K()
    n = len(pos)
    out = torch.full((n, nq * d), 7.0, dtype=q.dtype, device=DEV)
    args = (out, q, n, i32(pos), i32([1] * n))
    tail = (pages.k, pages.v, pages.table, nq, nkv, d, scale)
    kw = {"chunk": chunk, "softcap": cap}
    splits = 3 if which.endswith("split") else 1
    acc = torch.empty(n, nq, splits, d, device=DEV) if splits > 1 else None
    ml = torch.empty(n, nq, splits, 2, device=DEV) if splits > 1 else None
    if which.startswith("generic"):
        per = -(-(max(pos) + 1) // splits) if splits > 1 else 0
        k.attention_generic(*args, *tail, n_splits=splits, keys_per_split=per, part_acc=acc, part_ml=ml, **kw)
    elif which.startswith("decode_tma"):
        k.attention_decode_tma(*args, *tail, n_splits=2 if splits > 1 else 1, **kw)
        k.check_tc_status(DEV)
    elif which.startswith("decode"):
        k.attention_decode_bf16(*args, *tail, n_splits=splits, part_acc=acc, part_ml=ml, **kw)
    else:
        fn = k.attention_prefill_tc if which == "prefill_tc" else k.attention_prefill_bf16
        fn(*args, i32([0, n]), 1, *tail, **kw)
        if which == "prefill_tc":
            k.check_tc_status(DEV)
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,nq,nkv", [(20, 3, 1), (64, 4, 2), (96, 6, 1), (128, 8, 4), (256, 2, 2)])
@pytest.mark.parametrize("chunk,cap", [(9, None), (64, None), (70, 5.0), (130, 60.0), (None, 5.0), (None, 60.0), (1, None)])
def test_attention_within_chunks_and_under_a_soft_cap(dtype, d, nq, nkv, chunk, cap):
    """Every attention kernel against the plain rule: rows at the chunks' and pages' edges, a prompt whole and
    behind a cached prefix; scores far beyond the cap (and a cap beyond what needs no running maximum)."""
    length, scale = 300, 0.4
    pages = Pages(2, length, nkv, d, dtype, seed=d)
    keys, values = rnd(length, nkv, d, dtype=dtype, seed=1), rnd(length, nkv, d, dtype=dtype, seed=2)
    pages.fill(1, keys, values)
    width = -(-(nq * d + 8) // 8) * 8
    q = rnd(length, width, dtype=dtype, seed=3)
    edge = chunk or 128
    picks = sorted({0, 1, edge - 1, edge, edge + 1, 2 * edge - 1, 2 * edge, 63, 64, 65, 127, 128, 255, 256, length - 1} & set(range(length)))
    want = torch.stack([_plain_row(q[p, :nq * d].view(nq, d), keys, values, p, scale, chunk, cap) for p in picks])
    cut = 101
    for which in _kernels_for(dtype, d, nq, nkv):
        if which.startswith("decode"):
            got = _attend(which, q[picks].contiguous(), picks, pages, nq, nkv, d, scale, chunk, cap)
            assert rel(got, want) <= TOL[dtype], which
            dead = _attend(which, q[:2].contiguous(), [-1, -1], pages, nq, nkv, d, scale, chunk, cap)
            assert dead.abs().sum() == 0, which
            continue
        got = _attend(which, q, list(range(length)), pages, nq, nkv, d, scale, chunk, cap)
        assert rel(got[picks], want) <= TOL[dtype], which
        late = [i for i, p in enumerate(picks) if p >= cut]
        got = _attend(which, q[cut:], list(range(cut, length)), pages, nq, nkv, d, scale, chunk, cap)
        assert rel(got[[picks[i] - cut for i in late]], want[late]) <= TOL[dtype], (which, "behind a prefix")


@pytest.mark.parametrize("d,nq,nkv", [(96, 4, 2), (128, 4, 2)])
@pytest.mark.parametrize("chunk", [50, 64, 100])
def test_one_key_that_stands_out_at_every_edge_of_a_chunk(d, nq, nkv, chunk):
    """A key that takes nearly all the weight, put just inside and just outside the last row's chunk, in every
    16-bit kernel: the row gives that key's value where it is seen and nothing of it where it is not."""
    length = 2 * chunk + chunk // 2
    pos, lo = length - 1, (length - 1) // chunk * chunk
    keys, values = 0.1 * rnd(length, nkv, d, seed=1), rnd(length, nkv, d, seed=2)
    q = 0.1 * rnd(length, nq * d, seed=3)
    direction = torch.ones(d, device=DEV)
    q[pos] = direction.repeat(nq)
    for key_pos in sorted({0, lo - 1, lo, lo + 1, pos - 1, pos}):
        kk, vv = keys.clone(), values.clone()
        kk[key_pos] = direction
        vv[key_pos] = 50.0
        pages = Pages(2, length, nkv, d, BF16, seed=key_pos)
        pages.fill(1, kk.to(BF16), vv.to(BF16))
        for which in _kernels_for(BF16, d, nq, nkv):
            if which.startswith("decode"):
                row = _attend(which, q[pos:].to(BF16), [pos], pages, nq, nkv, d, 0.3, chunk, None)[0]
            else:
                row = _attend(which, q.to(BF16), list(range(length)), pages, nq, nkv, d, 0.3, chunk, None)[pos]
            if key_pos >= lo:
                assert (row.float() - 50.0).abs().max() <= 0.5, (which, key_pos)
            else:
                assert row.float().abs().max() < 10.0, (which, key_pos)


@pytest.mark.parametrize("d,nq,nkv,rot", [(128, 4, 2, 128), (64, 6, 3, 64), (128, 4, 2, 64), (256, 2, 1, 256)])
def test_biases_before_the_head_norm_and_rotation_of_many_tokens(d, nq, nkv, rot):
    """Enough 16-bit tokens for the wide prepare kernel (fully rotated heads) and its fallback, against 64-bit."""
    k = K()
    t = 150
    rows = rnd(t, (nq + 2 * nkv) * d, dtype=BF16, seed=1)
    bias = {n: rnd(c * d, seed=i + 2, scale=0.5) for i, (n, c) in enumerate((("q", nq), ("k", nkv), ("v", nkv)))}
    gq, gk = 1 + 0.2 * rnd(d, seed=6), 1 + 0.2 * rnd(d, seed=7)
    ang = torch.arange(t, dtype=F64)[:, None] * plain.frequencies(models.rotation(rot, 1e4))[None]
    cos, sin = ang.cos().float().to(DEV), ang.sin().float().to(DEV)
    cpu = rows.double().cpu().view(t, nq + 2 * nkv, d) + torch.cat([bias[n].double().cpu().view(-1, d) for n in "qkv"])[None]
    pos = torch.arange(t)
    turn = lambda x, g: plain.rotate(plain.rms_unit(x, 1e-5) * g.double().cpu(), pos, models.rotation(rot, 1e4), False)
    want_q, want_k, want_v = turn(cpu[:, :nq], gq), turn(cpu[:, nq:nq + nkv], gk), cpu[:, nq + nkv:]
    pages = Pages(2, t, nkv, d, BF16, seed=3)
    got = rows.clone()
    k.qk_prepare_kv(got, t, gq, gk, cos, sin, rot, i32(list(range(t))), i32([1] * t), pages.k, pages.v, pages.table, nq, nkv, d,
                    1e-5, q_bias=bias["q"], k_bias=bias["k"], v_bias=bias["v"])
    assert rel(got[:, :nq * d].view(t, nq, d), want_q) <= TOL[BF16]
    kk, vv = pages.dense(1, t)
    assert rel(kk, want_k) <= TOL[BF16] and rel(vv, want_v) <= TOL[BF16]
    # a layer that borrows its keys brings queries alone and stores nothing
    alone = rows[:, :nq * d].contiguous()
    before = pages.k.clone()
    k.qk_prepare_kv(alone, t, gq, None, cos, sin, rot, i32(list(range(t))), i32([1] * t), pages.k, pages.v, pages.table, nq, nkv,
                    d, 1e-5, write_kv=False, q_bias=bias["q"])
    assert torch.equal(alone, got[:, :nq * d]) and torch.equal(pages.k, before)


@pytest.mark.parametrize("heads,dim,vdim", [(3, 16, 24), (2, 64, 33), (5, 20, 12), (2, 200, 40), (4, 128, 128)])
def test_memory_with_fixed_decays_from_a_carried_state(heads, dim, vdim):
    """Three unequal sequences at once, then each continued from its state in slots that others used before."""
    k = K()
    lens, slots = [9, 1, 150], [2, 0, 3]
    n = sum(lens)
    decay = [1.0 - 0.6 ** (h + 1) for h in range(heads)]
    q, kk = rnd(2 * n, heads * dim + 4, seed=1), rnd(2 * n, heads * dim, seed=2, scale=0.5)
    v = rnd(2 * n, heads * vdim, seed=3)
    state = torch.zeros(4, -(-heads * vdim * k.decay_scan_rows(dim) // 4) * 4, device=DEV)
    a, b = torch.tensor(decay, device=DEV), torch.ones(heads, device=DEV)
    cu = [0]
    for ln in lens:
        cu.append(cu[-1] + ln)
    tok_slots = [s for s, ln in zip(slots, lens) for _ in range(ln)]
    for half in (0, 1):
        sl = slice(half * n, (half + 1) * n)
        pos = [half * ln + j for ln in lens for j in range(ln)]
        out = torch.empty(n, heads * vdim, device=DEV)
        k.decay_scan(out, q[sl], kk[sl], v[sl], a, b, state, i32(cu), i32(pos), i32(tok_slots), 3, heads, heads, dim, vdim,
                     n_tokens=n)
        for j, ln in enumerate(lens):
            rows = list(range(cu[j], cu[j] + ln)) + list(range(n + cu[j], n + cu[j] + ln))
            want, _ = plain.fixed_decay_scan(q[rows, :heads * dim].double().cpu().view(-1, heads, dim),
                                             kk[rows].double().cpu().view(-1, heads, dim),
                                             v[rows].double().cpu().view(-1, heads, vdim), decay)
            assert rel(out[cu[j]:cu[j + 1]].view(ln, heads, vdim), want[half * ln:(half + 1) * ln]) <= 1e-5, (half, j)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("inner,col", [(72, 8), (90, 3), (2048, 4), (5000, 1), (20000, 16)])
def test_output_norm_over_all_heads_with_its_gate(dtype, inner, col):
    k = K()
    o, proj, w = rnd(6, inner, seed=1, scale=3.0), rnd(6, inner + col + 4, seed=2), 1 + 0.2 * rnd(inner, seed=3)
    y = torch.full((6, inner), 7.0, dtype=dtype, device=DEV)
    k.norm_gate_out(y, o, proj, col, w, 1e-5, i32([0, 5, -1, 3, 2, 9]), 6)
    want = plain.rms_unit(o.double().cpu(), 1e-5) * w.double().cpu() * torch.sigmoid(proj[:, col:col + inner].double().cpu())
    live = [0, 1, 3, 4, 5]
    assert rel(y[live], want[live]) <= TOL[dtype] and (y[2] == 7.0).all()


def _glu_ref(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


@pytest.mark.parametrize("limit", [0.7, 7.0])
def test_clamped_gate_on_rows_and_in_the_products_epilogues(limit):
    k = K()
    for dtype in DTYPES:
        for rows, inter in ((1, 176), (19, 1000), (4, 1001), (3, 1004)):
            gu = rnd(rows, 2 * inter, dtype=dtype, seed=5, scale=3.0)
            out = torch.empty(rows, inter, dtype=dtype, device=DEV)
            k.act_mul(out, gu, "clamped", limit=limit)
            assert rel(out, _glu_ref(gu.double()[:, :inter], gu.double()[:, inter:], limit)) <= TOL[dtype]
    for m, inter, width in ((1, 96, 256), (8, 640, 2048), (40, 200, 512), (64, 64, 64), (300, 256, 512), (700, 1024, 256)):
        x, w = rnd(m, width, dtype=BF16, seed=m), rnd(2 * inter, width, dtype=BF16, seed=7, scale=2 * width ** -0.5)
        prod = x.double() @ w.double().T
        want = _glu_ref(prod[:, :inter], prod[:, inter:], limit)
        out = torch.empty(m, inter, dtype=BF16, device=DEV)
        if m <= 64:
            for split, cluster in ((1, True), (None, True), (2, True), (4, False)):
                out.fill_(7.0)
                k.gemm_tc_bf16(out, x, w, k.GATED_EPILOGUES["clamped"], swap=True, k_split=split, cluster=cluster,
                               gate_limit=limit)
                assert rel(out, want) <= TOL[BF16], (m, split, cluster)
        else:
            k.gemm_pair_bf16(out, x, w, k.PAIR_GATED_EPILOGUES["clamped"], gate_limit=limit)
            assert rel(out, want) <= TOL[BF16]
            out.fill_(7.0)
            k.gemm_tc_bf16(out, x, w, k.GATED_EPILOGUES["clamped"], swap=False, gate_limit=limit)
            assert rel(out, want) <= TOL[BF16]
    k.check_tc_status(DEV)


@pytest.mark.parametrize("experts,top", [(8, 2), (5, 3), (16, 6), (12, 1), (40, 33)])
def test_sigmoid_router(experts, top):
    """The largest scores in order and the scores themselves as weights, also where a score rounds to 1 or to 0."""
    k = K()
    for scale in (1.0, 40.0):
        logits = rnd(70, experts, seed=experts + top, scale=scale)
        chosen = torch.empty(70, top, dtype=torch.int32, device=DEV)
        weight = torch.empty(70, top, device=DEV)
        k.moe_route(chosen, weight, logits, 70, 1, 1, top, 1.5, weights="sigmoid")
        vals, idx = torch.topk(logits.double().cpu(), top, dim=-1)
        assert torch.equal(chosen.cpu().long(), idx)
        assert rel(weight, 1.5 * torch.sigmoid(vals)) <= 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff,experts,top,shared,tokens", [(96, 48, 8, 2, 56, 50), (100, 36, 2, 2, None, 7),
                                                                (256, 32, 16, 6, 128, 300), (128, 40, 6, 3, 20, 1),
                                                                (96, 20, 3, 1, 96, 130), (128, 64, 1, 1, 64, 9)])
def test_experts_that_weigh_their_input_beside_a_shared_one(dtype, width, ff, experts, top, shared, tokens):
    from enginekernel_b200.parts.moe import RoutedExperts
    from enginekernel_b200.parts.spec import PartSpec
    mlp = models.moe(experts, top, ff, shared)
    names = {"router": "router"}
    w = {"router": rnd(experts, width, dtype=BF16, seed=1, scale=4 * width ** -0.5)}
    for i, e in enumerate(list(range(experts)) + (["shared"] if shared else [])):
        p, size = (f"e{e}.", ff) if e != "shared" else ("shared.", shared)
        if e != "shared":
            names[f"gate_{e}"], names[f"up_{e}"], names[f"down_{e}"] = p + "gate", p + "up", p + "down"
        w[p + "gate"] = rnd(size, width, dtype=BF16, seed=200 + i, scale=2 * width ** -0.5)
        w[p + "up"] = rnd(size, width, dtype=BF16, seed=10 + i, scale=2 * width ** -0.5)
        w[p + "down"] = rnd(width, size, dtype=BF16, seed=100 + i, scale=size ** -0.5)
    shared_spec = None if not shared else PartSpec(
        "gated_mlp", {"hidden_size": width, "intermediate_size": shared, "activation": "clamped", "limit": 1.3, "name": "shared_expert"},
        {"gate": "shared.gate", "up": "shared.up", "down": "shared.down"})
    part = RoutedExperts(PartSpec("routed_experts", {
        "hidden_size": width, "intermediate_size": ff, "experts": experts, "top": top, "activation": "clamped", "limit": 0.8,
        "gated": True, "weights": "sigmoid", "weigh": "input", "shared": shared_spec}, names), dtype, DEV)
    part.load(w)
    x = rnd(tokens, width, dtype=dtype, seed=5)
    ctx = helpers.make_context(dtype, DEV, list(range(tokens)), [0] * tokens, [0, tokens])
    got = part.forward(x, ctx)
    want = plain.experts_ff(x.double().cpu(), {n: v.cpu() for n, v in w.items()}, "", mlp)
    rows = ((got.double().cpu() - want).abs().amax(-1) / want.abs().max()) <= TOL[dtype] * 2
    assert rows.float().mean().item() >= (1.0 if dtype == F32 else 0.97)
    # the weight joins the input, not the output: the two differ beyond any rounding here
    outside = plain.experts_ff(x.double().cpu(), {n: v.cpu() for n, v in w.items()}, "", dict(mlp, expert=dict(mlp["expert"], limit=50.0)))
    assert (outside - want).abs().max() > 0.05 * want.abs().max()


@pytest.mark.parametrize("dtype", DTYPES)
def test_block_with_norms_that_need_statistics(dtype):
    """The arrangement also runs with norms that cannot ride in its kernel (an RMS norm): u1 and u2 then come from
    the norms' own kernels over the joined stream."""
    import dataclasses

    from enginekernel_b200 import registry
    from enginekernel_b200.cache.store import SequenceCache
    from enginekernel_b200.config.kamosun import KamosunConfig
    from enginekernel_b200.engine.model import DecoderModel
    from enginekernel_b200.engine.runner import ModelRunner, StepEntry
    from enginekernel_b200.parts.spec import PartSpec
    cfg = models.SHAPES["flat"]
    spec = registry.model_spec_for(KamosunConfig.from_dict(cfg))
    rms = lambda s: PartSpec("rms_norm", {"size": cfg["width"], "eps": 1e-5}, {"gain": s.weights["gain"]})
    layers = [dataclasses.replace(l, norms={n: rms(s) for n, s in l.norms.items()}) for l in spec.layers]
    spec = dataclasses.replace(spec, layers=layers)
    model = DecoderModel(spec, dtype, DEV)
    w = models.make_tensors(cfg, 3)
    model.load({n: t.to(DEV) for n, t in w.items()})
    cache = SequenceCache(model.cache_entry_specs(), dtype, DEV, max_tokens=256, max_slots=2)
    runner = ModelRunner(model, cache)
    ids = models.random_prompts(cfg, [40], seed=2)[0]
    got = runner.step([StepEntry(cache.open(), ids, list(range(40)))])
    keep = plain.dynamic_tanh
    try:
        plain.dynamic_tanh = lambda x, ww, name: keep(x, ww, name) if name == "final.norm" else \
            plain.rms_unit(x, 1e-5) * ww[name].to(F64)
        want = plain.forward(cfg, w, ids)
    finally:
        plain.dynamic_tanh = keep
    assert helpers.rel_err(got, want) <= helpers.TOL["float32" if dtype == F32 else "bfloat16"]


# ===================================================================== one-mixer models
def _one_layer(mixer_entry, width, vocab, borrow=None):
    layers = [(mixer_entry, None)] if borrow is None else [(mixer_entry, None), (borrow, None)]
    return models.config(width, vocab, layers, residual_mult=1.3)


_QUIET = models.right(2, 16, 16, [0.0, 0.0])
ONE_LAYER = {
    # sharp attentions: scores spread over tens, so one key can hold nearly all the weight
    "chunk": _one_layer(models.attention(4, 2, 24, 40, models.rotation(16), 50, scale=1.0), 96, 600),
    "chunk_fast": _one_layer(models.attention(4, 2, 128, 128, models.rotation(128, 1e6), 100, scale=0.4), 128, 600),
    "chunk_small_values": _one_layer(models.attention(6, 1, 40, 12, models.rotation(10), 64, scale=0.5), 100, 600),
    "borrowed": _one_layer(models.attention(4, 2, 32, 32, models.rotation(32), 40, scale=0.8), 96, 600,
                           models.attention(2, 2, 32, 32, models.rotation(32), 90, kv_from=0, scale=0.8)),
    "capped": _one_layer(models.parallel(models.left(4, 2, 24, 40, models.rotation(16), 20.0, scale=1.0), _QUIET), 96, 600),
    "capped_fast": _one_layer(models.parallel(models.left(4, 4, 128, 128, models.rotation(128, 1e6), 30.0, scale=0.4), _QUIET), 128, 600),
    "memory": _one_layer(models.parallel(models.left(2, 1, 16, 16, None, 5.0), models.right(4, 24, 16, [0.99, 0.995, 1.0, 0.5])), 96, 83),
    "memory_wide": _one_layer(models.parallel(models.left(2, 1, 16, 16, None, 5.0), models.right(4, 128, 64, [0.999, 0.98, 1.0, 0.9])), 128, 83),
    "tall_values": _one_layer(models.parallel(models.left(2, 2, 48, 320, models.rotation(48), 20.0), models.right(2, 16, 300)), 64, 83),
}


@pytest.fixture(scope="module")
def one_layer_engines(tmp_path_factory):
    from enginekernel_b200 import Engine
    made = {}

    def get(tag, dtype):
        if (tag, dtype) not in made:
            cfg = ONE_LAYER[tag]
            w = models.make_tensors(cfg, 5)
            folder = models.write_folder(str(tmp_path_factory.mktemp("one_" + tag)), cfg, w)
            made[(tag, dtype)] = (Engine(folder, dtype, max_tokens=2048, max_batch=4), cfg, w)
        return made[(tag, dtype)]
    return get


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", list(ONE_LAYER))
def test_one_mixer_whole_then_token_by_token(one_layer_engines, tag, dtype):
    eng, cfg, w = one_layer_engines(tag, dtype)
    ids = models.random_prompts(cfg, [330], seed=2)[0]
    want = plain.forward(cfg, w, ids)
    assert helpers.rel_err(helpers.whole(eng, ids), want) <= helpers.TOL[dtype] * (1 if dtype == "float32" else 2)
    got = helpers.tail_one_by_one(eng, ids, 140)              # across page borders, chunks beginning among decoded tokens
    assert helpers.rel_err(got, want) <= helpers.TOL[dtype] * (1 if dtype == "float32" else 2)


def _best_key_token(cfg, w, last_token, last_pos, key_pos):
    """The vocabulary token whose key at ``key_pos`` scores highest against the query of ``last_token`` at ``last_pos``
    in some head of layer 0's attention (from the plain pieces)."""
    layer = cfg["layers"][0]
    pair = layer["type"] == "parallel"
    m, p = (layer["mixer"]["left"], "l0.mix.left.") if pair else (layer["mixer"], "l0.mix.")
    eps, v = cfg["norm"]["eps"], cfg["vocab"]
    h = plain.dynamic_tanh(w["embed"].double(), w, "l0.norm1")
    keys, _ = plain.make_keys_values(h, w, p, m, eps, torch.full((v,), key_pos), pair)
    q = plain.make_queries(h[last_token:last_token + 1], w, p, m, eps, torch.tensor([last_pos]), pair)[0]
    s = torch.einsum("hd,vhd->vh", q, keys.repeat_interleave(m["heads"] // m["kv_heads"], 1)) * m["scale"]
    s[:v // 2] = -1e9                                       # the prompts are drawn from the lower half
    return int(s.amax(-1).argmax())


@pytest.mark.parametrize("tag", ["chunk", "chunk_fast", "chunk_small_values", "borrowed", "capped", "capped_fast"])
def test_one_key_at_every_edge_decides_or_is_not_seen(one_layer_engines, tag):
    """The token whose key fits the last query best is put at the first places, just inside and just outside the
    last token's chunk, and on both sides of page borders, among 320 others: the last logits follow it where the
    plain rule sees it, in a prompt and when the last tokens are decoded alone."""
    eng, cfg, w = one_layer_engines(tag, "float32")
    layer, n = cfg["layers"][0], 320
    sizes = [l["mixer"]["mask"]["size"] for l in cfg["layers"] if l["type"] == "attention"]
    a = [t % (cfg["vocab"] // 2) for t in models.random_prompts(cfg, [n], seed=3)[0]]
    wa = plain.forward(cfg, w, a)[-1]
    runs = (helpers.whole, lambda e, ids: helpers.tail_one_by_one(e, ids, 3))
    ga = [run(eng, a)[-1] for run in runs]
    edges = {0, 1, 63, 64, 255, 256, n - 2}
    for size in sizes:
        lo = (n - 1) // size * size
        edges |= {lo - 1, lo, lo + 1}
    moved = {}
    for key_pos in sorted(edges & set(range(n - 1))):
        b = list(a)
        b[key_pos] = _best_key_token(cfg, w, a[-1], n - 1, key_pos)         # a token that is nowhere else
        wb = plain.forward(cfg, w, b)[-1]
        seen = any(plain.sees(n - 1, key_pos, s) for s in sizes) if sizes else True
        moved[key_pos] = (float((wa - wb).abs().max() / wa.abs().max()), seen)
        for run, base in zip(runs, ga):
            gb = run(eng, b)[-1]
            assert helpers.rel_err(gb, wb) <= helpers.TOL["float32"], key_pos
            assert (base - gb - (wa - wb).float()).abs().max().item() <= 1e-3 * float((wa - wb).abs().max()) + 2e-5 * float(wa.abs().max()), key_pos
    # the test's weights do what they are made for: a seen key moves the logits, an unseen one does not
    assert min(m for m, seen in moved.values() if seen) > 1e-3, moved
    if sizes:
        assert max([m for m, seen in moved.values() if not seen], default=0.0) < 1e-9, moved


@pytest.mark.parametrize("tag", ["memory", "memory_wide"])
@pytest.mark.parametrize("changed", [0, 63, 64, 300, 318])
def test_one_changed_token_moves_the_last_logits(one_layer_engines, tag, changed):
    """The same prompt with one token changed: what the state carries of it moves the logits at the end in the
    engine as in the plain model, in a prompt and when the last tokens are decoded alone."""
    eng, cfg, w = one_layer_engines(tag, "float32")
    a = models.random_prompts(cfg, [320], seed=3)[0]
    b = list(a)
    b[changed] = (a[changed] + 1) % cfg["vocab"]
    wa, wb = plain.forward(cfg, w, a)[-1], plain.forward(cfg, w, b)[-1]
    assert (wa - wb).abs().max() > 1e-4 * wa.abs().max()
    for run in (helpers.whole, lambda e, ids: helpers.tail_one_by_one(e, ids, 3)):
        ga, gb = run(eng, a)[-1], run(eng, b)[-1]
        assert (ga - gb - (wa - wb).float()).abs().max().item() <= 2e-2 * float((wa - wb).abs().max()) + 2e-5 * float(wa.abs().max())


# ===================================================================== whole models
TAGS = list(models.SHAPES)
SEEDS = {"early": 11, "flat": 12, "odd": 13, "wide": 14}
# in bfloat16 a router's score can round the other way than in 64-bit, and a row then takes another expert
ALLOWED = {"float32": 1.0, "bfloat16": 0.9}


@pytest.fixture(scope="module")
def weights():
    return {tag: models.make_tensors(cfg, SEEDS[tag]) for tag, cfg in models.SHAPES.items()}


@pytest.fixture(scope="module")
def engines(tmp_path_factory, weights):
    from enginekernel_b200 import Engine
    made = {}

    def get(tag, dtype):
        if (tag, dtype) not in made:
            folder = models.write_folder(str(tmp_path_factory.mktemp("kamosun_" + tag)), models.SHAPES[tag], weights[tag])
            made[(tag, dtype)] = Engine(folder, dtype, max_tokens=4096, max_batch=8)
        return made[(tag, dtype)]
    return get


def close(got, want, dtype, what=""):
    got, want = got.double().cpu(), want.double().cpu()
    err = (got - want).abs().amax(-1) / want.abs().max()
    limit = helpers.TOL[dtype] * (3 if dtype == "bfloat16" else 1)
    inside = (err <= limit).sum().item()
    assert inside >= ALLOWED[dtype] * err.numel() or err.numel() - inside <= (1 if dtype == "bfloat16" else 0), \
        f"{what} {dtype}: {inside} of {err.numel()} rows within {limit}, worst {err.max():.3e}"
    if dtype == "bfloat16" and err.numel() >= 3:
        assert err.median().item() <= helpers.TOL[dtype], f"{what}: median {err.median():.3e}"


_WANT = {}


def want_logits(weights, tag, ids):
    key = (tag, tuple(ids))
    if key not in _WANT:
        _WANT[key] = plain.forward(models.SHAPES[tag], weights[tag], ids)
    return _WANT[key]


def in_portions(engine, tokens, sizes):
    slot = engine.open_sequence()
    try:
        rows, at = [], 0
        for n in list(sizes) + [len(tokens)]:
            part = tokens[at:at + n]
            if not part:
                break
            rows.append(engine.step([(slot, part, list(range(len(part))))]).cpu())
            at += len(part)
        return torch.cat(rows, 0)
    finally:
        engine.close_sequence(slot)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", TAGS)
def test_whole_prompts(engines, weights, tag, dtype):
    eng = engines(tag, dtype)
    for j, n in enumerate((1, 2, 7, 33, 64, 65, 130, 260)):
        ids = models.random_prompts(models.SHAPES[tag], [n], seed=40 + j)[0]
        close(helpers.whole(eng, ids), want_logits(weights, tag, ids), dtype, f"{tag} length {n}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", TAGS)
def test_prompt_then_token_by_token(engines, weights, tag, dtype):
    eng = engines(tag, dtype)
    ids = models.random_prompts(models.SHAPES[tag], [150], seed=77)[0]
    got = helpers.tail_one_by_one(eng, ids, 80)               # every chunk of the shapes but one begins among decoded tokens
    close(got, want_logits(weights, tag, ids), dtype, tag)
    if dtype == "float32":
        assert helpers.rel_err(got, helpers.whole(eng, ids)) <= 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", TAGS)
def test_prompts_in_portions(engines, weights, tag, dtype):
    eng = engines(tag, dtype)
    ids = models.random_prompts(models.SHAPES[tag], [210], seed=78)[0]
    want = want_logits(weights, tag, ids)
    for sizes in ((2, 2, 2, 3, 17), (64, 64, 2), (63, 2, 65), (1, 127, 2), (129,)):
        close(in_portions(eng, ids, sizes), want, dtype, f"{tag} portions {sizes}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", TAGS)
def test_unequal_batches_and_reuse(engines, weights, tag, dtype):
    """Requests of unequal lengths start together and end at different steps; three such batches in a row
    through the same few slots, pages and states, then everything is free again."""
    eng = engines(tag, dtype)
    shapes = [((5, 9, 13), (3, 9, 1)), ((1, 70, 31, 16), (1, 64, 20, 16)), ((66, 2, 140), (65, 1, 100))]
    for j, (lens, heads) in enumerate(shapes):
        seqs = models.random_prompts(models.SHAPES[tag], lens, seed=200 + j)
        got = helpers.batch_then_steps(eng, seqs, heads)
        for ids, g in zip(seqs, got):
            close(g, want_logits(weights, tag, ids), dtype, f"{tag} batch {j} length {len(ids)}")
            if dtype == "float32":                       # what else is in the batch does not matter beyond rounding
                assert helpers.rel_err(g, helpers.whole(eng, ids)) <= 1e-5
    assert eng.cache.book.open_slots() == []
    assert eng.cache.free_tokens() == eng.cache.num_pages * 64


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["odd", "early"])
def test_first_tokens_one_by_one(engines, weights, tag, dtype):
    eng = engines(tag, dtype)
    ids = models.random_prompts(models.SHAPES[tag], [7], seed=5)[0]
    close(helpers.tail_one_by_one(eng, ids, tail=6), want_logits(weights, tag, ids), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["early", "flat"])
def test_long_decoding(engines, weights, tag, dtype):
    """Pages in front of the widest chunk go back while the sequence grows, and are used again."""
    eng = engines(tag, dtype)
    ids = models.random_prompts(models.SHAPES[tag], [300], seed=9)[0]
    close(helpers.tail_one_by_one(eng, ids, tail=290), want_logits(weights, tag, ids), dtype, tag)


def test_a_step_too_large_for_one_pass_is_cut(tmp_path, weights):
    """The engine's own cut of a large step: kept results of one piece do not leak into the next."""
    from enginekernel_b200 import Engine
    cfg = models.SHAPES["early"]
    eng = Engine(models.write_folder(str(tmp_path / "m"), cfg, weights["early"]), "float32", max_tokens=1024, max_batch=4)
    eng.runner.max_step_tokens = 50
    seqs = models.random_prompts(cfg, (70, 33), seed=6)
    slots = [eng.open_sequence() for _ in seqs]
    got = eng.step([(s, t, list(range(len(t)))) for s, t in zip(slots, seqs)]).cpu()
    close(got[:70], want_logits(weights, "early", seqs[0]), "float32")
    close(got[70:], want_logits(weights, "early", seqs[1]), "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["early", "wide"])
def test_greedy_generation_through_the_scheduler(tmp_path, tag, dtype):
    """``Engine.generate_all``: five requests of unequal lengths through two slots, so the scheduler forms
    several batches and the captured decode step runs on slots, states and pages used before."""
    from enginekernel_b200 import Engine
    cfg = models.SHAPES[tag]
    w = models.make_tensors(cfg, 21)
    folder = models.write_folder(str(tmp_path / "m"), cfg, w)
    eng = Engine(folder, dtype, max_tokens=2048, max_batch=2)
    prompts = models.random_prompts(cfg, [3, 70, 17, 64, 1], seed=8)
    got = eng.generate_all(prompts, 12)
    distinct = set()
    for ids, out in zip(prompts, got):
        assert len(out) == 12
        want = plain.greedy(cfg, w, ids, 12)
        distinct.update(want)
        if dtype == "float32":
            assert out == want
    assert len(distinct) > 3
    assert eng.cache.book.open_slots() == []
    eager = Engine(folder, dtype, max_tokens=2048, max_batch=2, use_graph=False)
    assert eager.generate_all(prompts, 12) == got             # without the captured graph: the same tokens


def test_unused_tensors_and_missing_ones(tmp_path):
    """A layer without feed-forward may still carry its second norm and gate; a file that lacks a tensor is refused
    by name, and so is one that holds keys for a layer that borrows them."""
    from enginekernel_b200 import Engine
    from enginekernel_b200.weights.checkpoint import WeightsError
    cfg = models.SHAPES["early"]
    w = models.make_tensors(cfg, 2)
    w["l1.norm2"] = torch.zeros(cfg["width"], dtype=BF16)
    w["l1.rg2.b"] = torch.zeros(cfg["width"], dtype=BF16)
    eng = Engine(models.write_folder(str(tmp_path / "a"), cfg, w), "float32", max_tokens=256, max_batch=2)
    ids = models.random_prompts(cfg, [20], seed=1)[0]
    assert helpers.rel_err(helpers.whole(eng, ids), plain.forward(cfg, w, ids)) <= helpers.TOL["float32"]
    for name in ("l0.dwa", "l2.rg1.b", "l0.norm1.alpha", "l0.mix.right.out", "l1.mix.k.norm", "l0.mlp.e3.up", "l2.mix.o.b"):
        less = dict(w)
        del less[name]
        with pytest.raises(WeightsError, match=name):
            Engine(models.write_folder(str(tmp_path / ("b" + name)), cfg, less), "float32", max_tokens=256, max_batch=2)
    with pytest.raises(WeightsError, match="l2.mix.k"):
        Engine(models.write_folder(str(tmp_path / "c"), cfg, dict(w, **{"l2.mix.k": w["l1.mix.k"].clone()})), "float32",
               max_tokens=256, max_batch=2)


def test_command_line_and_trace_replay(tmp_path):
    """``random-model`` writes a Kamosun folder from a configuration file, ``generate`` prints the plain model's
    greedy tokens for it, and ``bin/trace_run`` replays steps over the same folder."""
    import os
    import subprocess
    import sys

    import numpy as np
    from safetensors import safe_open
    from tests.test_cli_gpu import ROOT, run_cli
    cfg = models.SHAPES["flat"]
    config_file = tmp_path / "config.json"
    config_file.write_text(json.dumps(cfg))
    folder = tmp_path / "model"
    run_cli("random-model", "--config", str(config_file), "--seed", "5", "--out", str(folder))
    with safe_open(str(folder / "model.safetensors"), framework="pt", device="cpu") as f:
        w = {name: f.get_tensor(name) for name in f.keys()}
    assert {n: tuple(t.shape) for n, t in w.items()} == models.tensor_shapes(cfg)
    prompts = models.random_prompts(cfg, (3, 40), seed=4)
    ids = ";".join(",".join(str(t) for t in p) for p in prompts)
    out = run_cli("generate", "--model", str(folder), "--dtype", "float32", "--prompt-ids", ids, "--out-len", "5")
    rows = [json.loads(line) for line in out.strip().splitlines()]
    assert [r["tokens"] for r in rows] == [plain.greedy(cfg, w, p, 5) for p in prompts]

    steps = [{"step": 0, "entries": [{"id": "a", "tokens": prompts[1][:30], "want": [0, 29]},
                                     {"id": "b", "tokens": prompts[0][:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": prompts[1][30:31], "want": [0]},
                                     {"id": "b", "tokens": prompts[0][1:2], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": prompts[1][31:32], "want": [0]}], "end": ["a"]}]
    out_dir = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype",
                        "float32", "--out", str(out_dir), "--max-tokens", "128"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                       timeout=900)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    a, b = plain.forward(cfg, w, prompts[1][:32]), plain.forward(cfg, w, prompts[0][:2])
    want = {0: torch.stack([a[0], a[29]]), 1: torch.stack([a[30], b[1]]), 2: a[31:32]}
    for n, rows_wanted in want.items():
        got = torch.from_numpy(np.fromfile(str(out_dir / f"{n}.f32"), dtype="<f4").reshape(rows_wanted.shape))
        assert helpers.rel_err(got, rows_wanted) <= helpers.TOL["float32"], n
