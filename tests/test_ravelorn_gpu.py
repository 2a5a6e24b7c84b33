"""Ravelorn on the GPU against the plain implementation (tests/plain_ravelorn.py): each mechanism alone, then the
engine in every way of cutting and batching, in 32-bit and in bfloat16.

Tolerances are a fraction of the largest |logit| of the row compared.  float32: sums of a few hundred terms in
another order than the plain implementation's float64.  bfloat16: activations are rounded to 8 bits of mantissa
between kernels, a dozen roundings a layer, and a norm on a small result (a head of four values, a sum that nearly cancels)
multiplies its rounding: the plain implementation with its products' inputs and results rounded to bfloat16 is off by 0.1 in
single rows of these random models, by 0.02 in the median row.  So in bfloat16 the median row is held to a tight bound and
every row to a loose one; 32-bit is the sharp comparison.
"""
import json
import math
from types import SimpleNamespace

import pytest
import torch

import plain_ravelorn as P
from tiny_models import RAVELORN, prompt, write_ravelorn

pytestmark = pytest.mark.gpu

TOL = {"float32": 1e-4, "bfloat16": 3e-1}
MEDIAN = {"float32": 3e-5, "bfloat16": 3e-2}
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DEV = "cuda:0"


def rel_err(got, want):
    want = want.to(torch.float64)
    got = got.to(torch.float64).cpu()
    scale = want.abs().amax(dim=-1, keepdim=True).clamp_min(1e-30)
    return float(((got - want).abs() / scale).max())


def close(got, want, tol):
    want = want.double()
    got = got.double().cpu()
    return float((got - want).abs().max()) <= tol * max(1e-30, float(want.abs().max()))


def i32(xs):
    return torch.tensor(xs, dtype=torch.int32, device=DEV)


def cu_of(lens):
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    return cu


# ---- each mechanism alone -------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H", [20, 64, 131])
def test_learned_positions_join_the_embedding(dtype, H):
    """Rows of both tables added; a position or an id outside its table is recorded and gives zeros."""
    from rocml_b200 import kernels
    torch.manual_seed(H)
    table, pos = torch.randn(31, H).to(DT[dtype]), torch.randn(17, H).to(DT[dtype])
    ids, at = [3, 0, 30, 7, 31, 2], [0, 16, 5, 5, 1, 17]
    out = torch.full((6, H), 7.0, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    kernels.embedding_pos(i32(ids[:4]), table.to(DEV), out[:4], 1.0, i32(at[:4]), None, status=status, pos_table=pos.to(DEV))
    want = table.double()[ids[:4]] + pos.double()[at[:4]]
    assert close(out[:4], want, 1e-6) and int(status.item()) == 0
    kernels.embedding_pos(i32(ids[4:]), table.to(DEV), out[4:], 1.0, i32(at[4:]), None, status=status, pos_table=pos.to(DEV))
    assert float(out[4:].abs().sum()) == 0.0 and int(status.item()) != 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T, H, parts", [(5, 20, 2), (70, 64, 1), (300, 256, 3), (3, 131, 1), (9, 4096, 8)])
def test_layer_norm_with_partial_sums_and_gathered_rows(dtype, T, H, parts):
    from rocml_b200 import kernels
    torch.manual_seed(T + H)
    x, d = torch.randn(T, H) + 3.0, torch.randn(parts, T, H)
    w, b = 1 + 0.3 * torch.randn(H), torch.randn(H)
    resid = x.clone().to(DEV)
    out = torch.zeros((T, H), dtype=DT[dtype], device=DEV)
    kernels.add_layernorm(resid, d.to(DEV), w.to(DEV), b.to(DEV), 1e-5, out)
    r = x.double() + d.double().sum(0)
    assert close(out, P.layer_norm(r, w.double(), b.double(), 1e-5), 1e-2 if dtype == "bfloat16" else 3e-6)
    assert close(resid, r, 1e-6)
    rows = [T - 1, -1, 0]
    picked = torch.full((3, H), 7.0, dtype=DT[dtype], device=DEV)
    kernels.add_layernorm(resid, None, w.to(DEV), b.to(DEV), 1e-5, picked, rows=i32(rows), n_rows=3, write_back=False)
    want = P.layer_norm(r[[T - 1, 0]], w.double(), b.double(), 1e-5)
    assert close(picked[[0, 2]], want, 1e-2 if dtype == "bfloat16" else 3e-6) and float(picked[1].float().min()) == 7.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T, H, parts, layer, bias", [(70, 64, 1, True, True), (3, 131, 3, True, True), (300, 256, 2, False, False), (8, 2048, 6, True, True)])
def test_norm_of_a_result_and_its_addition(dtype, T, H, parts, layer, bias):
    """resid += m * norm(c * sum of partial sums), and the same with a weighted sum over a token's experts and its own row."""
    from rocml_b200 import kernels
    torch.manual_seed(T + H)
    x, d = torch.randn(T, H), torch.randn(parts, T, H) + 0.5
    w, b = 1 + 0.3 * torch.randn(H), torch.randn(H) if bias else None
    tol = 1e-2 if dtype == "bfloat16" else 3e-6

    def norm(r):
        b64 = b.double() if bias else 0.0
        return P.layer_norm(r, w.double(), b64, 2e-5) if layer else P.rms(r, 2e-5) * w.double() + b64
    resid = x.clone().to(DEV)
    out = torch.zeros((T, H), dtype=DT[dtype], device=DEV)
    kernels.out_norm(resid, d.to(DEV), w.to(DEV), None if b is None else b.to(DEV), 2e-5, 0.3, layer, out, scale=0.01)
    want = x.double() + 0.3 * norm(0.01 * d.double().sum(0))     # (a scale that brings the eps into play)
    assert close(resid, want, 3e-6) and close(out, want, tol)
    top, R = 3, 2 * T + 5
    rows = torch.randn(R, H)
    row_of = torch.randint(-1, R, (T, top), dtype=torch.int32)
    row_of[0] = -1
    wt, own = torch.rand(T, top), torch.rand(T)
    own[1] = 0.0
    resid = x.clone().to(DEV)
    kernels.out_norm(resid, rows.to(DEV), w.to(DEV), None if b is None else b.to(DEV), 2e-5, 0.3, layer, out, row_of=row_of.to(DEV),
                     weights=wt.to(DEV), top=top, self_weight=own.to(DEV), self_x=resid)
    s = own.double()[:, None] * x.double()
    for j in range(top):
        s = s + torch.where(row_of[:, j:j + 1] >= 0, wt.double()[:, j:j + 1] * rows.double()[row_of[:, j].clamp_min(0).long()], 0.0)
    assert close(resid, x.double() + 0.3 * norm(s), 5e-6)


def test_soft_cap():
    from rocml_b200 import kernels
    x = torch.linspace(-80, 80, 999, device=DEV)
    want = 7.0 * torch.tanh(x.double().cpu() * 0.5 / 7.0)
    kernels.softcap_(x, 7.0, 0.5)
    assert close(x, want, 1e-6)


DELTA_SIZES = [(4, 2, 8, 12, 3), (1, 1, 5, 7, 1), (3, 3, 36, 4, 6), (2, 1, 128, 128, 4), (3, 3, 136, 64, 3), (6, 3, 64, 64, 2), (2, 2, 30, 10, 9),
               (2, 1, 300, 20, 2)]


def delta_case(heads, kv, dim, vdim, taps, per_channel, total, seed):
    """Projection rows of sequences of the given lengths, and what the plain implementation makes of them."""
    torch.manual_seed(seed)
    kd, inner = kv * dim, heads * vdim
    offs = {"q": 3, "k": 3 + kd, "v": 3 + 2 * kd, "b": 3 + 2 * kd + inner, "a": 3 + 2 * kd + inner + heads}
    width = offs["a"] + (heads * dim if per_channel else heads) + 2
    conv = torch.randn(2 * kd + inner, taps)
    a_log, dt = torch.randn(heads) - 3.5, torch.randn(heads * dim if per_channel else heads)
    rows, want = [], []
    of = torch.arange(heads) // (heads // kv)
    for n in total:
        x = torch.randn(n, width)
        # one key far back that must still be found: an early token writes with a large value
        x[min(2, n - 1), offs["v"]:offs["v"] + inner] *= 6.0
        c = P.silu(P.causal_conv(x[:, offs["q"]:offs["q"] + 2 * kd + inner].double(), conv.double()))
        q = (P.unit(c[:, :kd].reshape(n, kv, dim)) * dim ** -0.5)[:, of]
        k = P.unit(c[:, kd:2 * kd].reshape(n, kv, dim))[:, of]
        v = c[:, 2 * kd:].reshape(n, heads, vdim)
        z = x[:, offs["a"]:width - 2].double()
        g = P.decay(z.reshape(n, heads, dim) if per_channel else z, a_log.double(), dt.double().reshape(heads, dim) if per_channel else dt.double())
        beta = torch.sigmoid(x[:, offs["b"]:offs["b"] + heads].double())
        o, S = P.delta_rule(q, k, v, beta, g)
        rows.append(x)
        want.append((q, k, v, beta, g, o.reshape(n, inner), S))
    return offs, conv, a_log, dt, rows, want


@pytest.mark.parametrize("sizes", DELTA_SIZES)
@pytest.mark.parametrize("per_channel", [False, True])
@pytest.mark.parametrize("chunks", [False, True])
def test_gated_delta_rule(sizes, per_channel, chunks):
    """Convolutions, unit norms, decays and the recurrence over several steps (prompts, pieces shorter than the taps, single
    tokens), two sequences side by side with a padding sequence, slots that others used before, from one result and from
    partial sums; token after token and four at a time."""
    from rocml_b200 import kernels
    heads, kv, dim, vdim, taps = sizes
    if chunks and kernels.delta_padded_dim(dim) is None:
        pytest.skip("more rows than the kernel for prompts takes")
    steps = [[70, 3], [1, 1], [2, 67], [1, 2], [33, 1]]
    slots, total = [2, 0], [sum(s[i] for s in steps) for i in range(2)]
    offs, conv, a_log, dt, rows, want = delta_case(heads, kv, dim, vdim, taps, per_channel, total, heads * dim + vdim)
    kd, inner = kv * dim, heads * vdim
    state = torch.full((3, heads, vdim, dim), 5.0, device=DEV)
    kept = torch.full((3, taps - 1, 2 * kd + inner), 5.0, device=DEV)
    state[slots] = 0.0
    kept[slots] = 0.0
    layout = kernels.DeltaRows(heads, kv, dim, vdim, per_channel)
    at = [0, 0]
    for step, lens in enumerate(steps):
        x = torch.cat([r[a:a + n] for r, a, n in zip(rows, at, lens)])
        proj = x.to(DEV) if step % 2 == 0 else torch.stack([0.5 * x, 0.25 * x, 0.25 * x]).to(DEV)
        T, cu = x.shape[0], i32(cu_of(lens) + [sum(lens)])
        seq = i32(slots + [-1])
        u = torch.full((T, layout.width), float("nan"), device=DEV)
        kernels.delta_prep(proj, T, offs["q"], offs["k"], offs["v"], offs["b"], heads, kv, dim, vdim, taps, conv.t().contiguous().to(DEV),
                           kept if taps > 1 else None, proj[..., offs["a"]:], dt.to(DEV), a_log.to(DEV), per_channel, 1e-6, dim ** -0.5,
                           seq, cu, 3, max(lens), u, layout)
        q, k, v, beta, g, o = (torch.cat([w[i][a:a + n] for w, a, n in zip(want, at, lens)]) for i in range(6))
        uq, uk, uv, ug, ub, ud = layout.offsets
        rep = heads // kv
        assert close(u[:, uq:uq + kd], q[:, ::rep].reshape(T, kd), 1e-5) and close(u[:, uk:uk + kd], k[:, ::rep].reshape(T, kd), 1e-5)
        assert close(u[:, uv:uv + inner], v.reshape(T, inner), 1e-5) and close(u[:, ub:ub + heads], beta, 1e-5)
        assert close(u[:, ug:ug + g[0].numel()], g.reshape(T, -1), 1e-5)
        assert close(u[:, ud:ud + kv], (q * k).sum(-1)[:, ::rep], 1e-5)
        out = torch.full((T, inner), float("nan"), device=DEV)
        if chunks and max(lens) > 1:
            dimp = kernels.delta_padded_dim(dim)
            work = [torch.full(shape, float("nan"), device=DEV)
                    for shape in ((heads, T, 3, dimp), (heads, T // 4 + 3, dimp + kernels.DELTA_CHUNK_NUMBERS))]
            kernels.delta_scan_chunks(u, T, layout, heads, kv, dim, vdim, per_channel, state, seq, cu, 3, max(lens), out, *work)
        else:
            kernels.delta_scan(u, T, layout, heads, kv, dim, vdim, per_channel, state, seq, cu, 3, out)
        assert close(out, o, 2e-5), (step, lens)
        at = [a + n for a, n in zip(at, lens)]
    for i, s in enumerate(slots):
        assert close(state[s].transpose(1, 2), want[i][6], 2e-5)
    assert float(state[1].min()) == 5.0 and (taps == 1 or float(kept[1].min()) == 5.0)


def test_a_cut_does_not_change_single_tokens_bits():
    """Token after token: one token a step gives the bits of all tokens in one step."""
    from rocml_b200 import kernels
    heads, kv, dim, vdim, taps = 4, 2, 20, 24, 4
    offs, conv, a_log, dt, rows, _ = delta_case(heads, kv, dim, vdim, taps, True, [15], 7)
    layout = kernels.DeltaRows(heads, kv, dim, vdim, True)
    outs = []
    for lens in ([15], [1] * 15, [4, 9, 2]):
        state = torch.zeros((1, heads, vdim, dim), device=DEV)
        kept = torch.zeros((1, taps - 1, conv.shape[0]), device=DEV)
        got, at = [], 0
        for n in lens:
            proj = rows[0][at:at + n].to(DEV)
            u = torch.zeros((n, layout.width), device=DEV)
            kernels.delta_prep(proj, n, offs["q"], offs["k"], offs["v"], offs["b"], heads, kv, dim, vdim, taps, conv.t().contiguous().to(DEV), kept,
                               proj[:, offs["a"]:], dt.to(DEV), a_log.to(DEV), True, 1e-6, dim ** -0.5, i32([0]), i32([0, n]), 1, n, u, layout)
            out = torch.zeros((n, heads * vdim), device=DEV)
            kernels.delta_scan(u, n, layout, heads, kv, dim, vdim, True, state, i32([0]), i32([0, n]), 1, out)
            got.append(out)
            at += n
        outs.append(torch.cat(got))
    assert torch.equal(outs[0], outs[1]) and torch.equal(outs[0], outs[2])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T, ranks, parts", [(3, (24, 16), 2), (20, (7, 130), 1), (8, (64, 64), 5)])
def test_narrow_products_for_few_tokens(dtype, T, ranks, parts):
    from rocml_b200 import kernels
    torch.manual_seed(T)
    n0, n1 = 150, 40
    x = torch.randn(T, ranks[0] + ranks[1] + 9)
    w0, w1 = torch.randn(n0, ranks[0]).to(DT[dtype]), torch.randn(n1, ranks[1]).to(DT[dtype])
    proj = torch.stack([x / parts] * parts).to(DEV)
    out = torch.zeros((T, n0 + n1), device=DEV)
    kernels.low_rank(proj, T, 2, w0.to(DEV), 4 + ranks[0], w1.to(DEV), out)
    want = torch.cat([x.double()[:, 2:2 + ranks[0]] @ w0.double().T, x.double()[:, 4 + ranks[0]:4 + sum(ranks)] @ w1.double().T], dim=1)
    assert close(out, want, 3e-6)
    only = torch.zeros((T, n1), device=DEV)
    kernels.low_rank(proj[0], T, 4 + ranks[0], w1.to(DEV), 0, None, only)
    assert close(only, want[:, n0:] / parts, 3e-6)


@pytest.mark.parametrize("E, identity, top", [(10, 2, 2), (5, 3, 5), (70, 9, 6), (3, 0, 1)])
def test_softmax_scores_correction_and_identity_experts(E, identity, top):
    """The choice follows score + correction, the weights are the scores; an identity choice has no row and joins the token's
    own weight; padding tokens choose nothing.  Then the weighted sum with the token's own row."""
    from rocml_b200 import kernels
    torch.manual_seed(E)
    T, H = 90, 36
    z, corr = 2 * torch.randn(T, E), 0.3 * torch.rand(E)
    slot = torch.zeros(T, dtype=torch.int32)
    slot[7] = -1
    ids, place = (torch.full((T, top), -9, dtype=torch.int32, device=DEV) for _ in range(2))
    weights, own = torch.zeros((T, top), device=DEV), torch.zeros(T, device=DEV)
    counts = torch.zeros(E, dtype=torch.int32, device=DEV)
    kernels.moe_route(z.to(DEV), corr.to(DEV), slot.to(DEV), T, top, ids, weights, place, counts, score="softmax", identity=identity,
                      self_weight=own)
    s = torch.softmax(z.double(), -1)
    order = torch.sort(s + corr.double(), dim=-1, descending=True)
    want, real = order.indices[:, :top], E - identity
    for t in range(T):
        got = ids[t].tolist()
        if t == 7:
            assert got == [-1] * top and float(own[t]) == 0.0
            continue
        assert got == [e if e < real else -1 for e in want[t].tolist()]
        assert abs(float(own[t]) - float(sum((s[t, e] for e in want[t].tolist() if e >= real), torch.tensor(0.0)))) < 1e-6
    live = [t for t in range(T) if t != 7]
    assert close(weights[live], torch.gather(s, 1, want)[live], 1e-5)
    real_ids = want[live][want[live] < real]
    assert counts.tolist() == [int((real_ids == e).sum()) if e < real else 0 for e in range(E)]
    # one launch for few tokens: the same choices, rows in whole tiles of their expert, the tokens' rows copied
    n = 13
    x = torch.randn(n, H).to(torch.bfloat16)
    tiles = n * top // 4 + min(real, n * top) + 1
    xs, row_of, group = torch.zeros((tiles * 4, H), dtype=torch.bfloat16, device=DEV), torch.full((n, top), -9, dtype=torch.int32, device=DEV), torch.full((tiles,), -9, dtype=torch.int32, device=DEV)
    w2, own2 = torch.zeros((n, top), device=DEV), torch.zeros(n, device=DEV)
    kernels.moe_route_few(z.to(DEV), corr.to(DEV), slot.to(DEV), n, E, top, x.to(DEV), xs, row_of, w2, 4, group, score="softmax",
                          identity=identity, self_weight=own2)
    assert torch.equal(w2, weights[:n]) and torch.equal(own2, own[:n])
    used = set()
    for t in range(n):
        for j in range(top):
            e, row = int(ids[t, j]), int(row_of[t, j])
            assert (row < 0) == (e < 0)
            if e >= 0:
                assert int(group[row // 4]) == e and row not in used and torch.equal(xs[row].cpu(), x[t])
                used.add(row)
    assert sorted(set(group.tolist())) == sorted({-1} | {e for e in ids[:n].flatten().tolist() if e >= 0})
    rows = torch.randn(20, H)
    row_of = torch.randint(-1, 20, (T, top), dtype=torch.int32)
    x = torch.randn(T, H).to(torch.bfloat16)
    out = torch.zeros((T, H), device=DEV)
    kernels.moe_combine(rows.to(DEV), row_of.to(DEV), weights, T, top, out, self_weight=own, self_x=x.to(DEV))
    ref = own.double().cpu()[:, None] * x.double()
    for j in range(top):
        ref = ref + torch.where(row_of[:, j:j + 1] >= 0, weights.double().cpu()[:, j:j + 1] * rows.double()[row_of[:, j].clamp_min(0).long()], 0.0)
    assert close(out, ref, 3e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nq, nkv, hd, vd, parts", [(4, 2, 16, 16, 1), (6, 1, 24, 12, 2), (8, 2, 128, 128, 1), (3, 3, 20, 28, 3)])
def test_unit_queries_and_keys_and_the_query_temperature(dtype, nq, nkv, hd, vd, parts):
    """No rotation; queries and keys over their root mean square, queries times the temperature of their position (positions
    around its steps), heads padded to one width, columns that are a part of wider rows."""
    from rocml_b200 import kernels
    torch.manual_seed(nq * hd)
    dt, T, eps = DT[dtype], 70, 1e-5
    hdp = -(-max(hd, vd) // 16) * 16
    width = (nq + nkv) * hd + nkv * vd
    full = torch.randn(parts, T, width + 16) if parts > 1 else torch.randn(T, width + 16).to(dt)
    pos = torch.arange(5, 5 + T, dtype=torch.int32)
    kc, vc = (torch.full((2, nkv, 64, hdp), 7.0, dtype=dt, device=DEV) for _ in range(2))
    q = torch.full((T, nq * hdp), 7.0, dtype=dt, device=DEV)
    kernels.qk_norm_rope_cache(full.to(DEV)[..., 8:8 + width], q, T, nq, nkv, hd, None, None, eps, None, 0, pos.to(DEV),
                               torch.zeros(T, dtype=torch.int32, device=DEV), i32([[1, 0]]), kc, vc, v_head_dim=vd, padded_head_dim=hdp,
                               post_norm=True, q_temp=(0.7, 16))
    x = (full.double().sum(0) if parts > 1 else full.double())[:, 8:8 + width]
    f = P.query_temperature(pos.tolist(), {"coef": 0.7, "every": 16})
    tol = 1e-2 if dtype == "bfloat16" else 2e-6
    q3 = q.reshape(T, nq, hdp)
    assert close(q3[..., :hd], P.rms(x[:, :nq * hd].reshape(T, nq, hd), eps) * f[:, None, None], tol)
    assert hd == hdp or float(q3[..., hd:].float().abs().max()) == 0.0

    def cached(c):
        return torch.stack([c[[1, 0][int(p) // 64], :, int(p) % 64] for p in pos])
    assert close(cached(kc)[..., :hd], P.rms(x[:, nq * hd:(nq + nkv) * hd].reshape(T, nkv, hd), eps), tol)
    assert close(cached(vc)[..., :vd], x[:, (nq + nkv) * hd:].reshape(T, nkv, vd), tol)


SINK_CASES = [
    # lens, q_lens, nq, nkv, hd, strided output
    ([5, 70, 129], [5, 70, 129], 4, 2, 16, False),
    ([200, 64, 1], [30, 1, 1], 6, 3, 48, True),
    ([700, 333, 150], [1, 1, 1], 8, 4, 64, True),
    ([300, 70], [300, 70], 8, 2, 128, True),
    ([1100, 65], [1, 1], 4, 4, 16, False),
    ([900, 200, 64, 2], [1, 1, 1, 1], 16, 4, 128, True),
    ([2500], [1], 4, 1, 256, False),
    ([513], [200], 4, 4, 64, True),
    ([260, 131], [130, 2], 4, 2, 256, False),
]


@pytest.mark.parametrize("case", range(len(SINK_CASES)))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_sink_for_every_head(case, dtype):
    """Every attention kernel (plain with and without the merge, the two for prompts, decode clustered and merged) with a sink per
    head: small, as large as the scores, far above them, far below.  A key hundreds of positions back is made to stand out
    for one head."""
    from rocml_b200 import kernels
    from rocml_b200.parts.attention import paged_attention
    from test_kernels_gpu import paged_case
    lens, q_lens, nq, nkv, hd, strided = SINK_CASES[case]
    dt = DT[dtype]
    ks, vs, qs, kc, vc, meta = paged_case(900 + case, lens, q_lens, nq, nkv, hd, dt)
    for b, n in enumerate(lens):
        if n > 40:
            ks[b][3, 0] = (qs[b][-1, 0] * 3.0).to(dt).float()
            kc[int(meta["table"][meta["seq_slot"][b], 0]), 0, 3] = ks[b][3, 0]
    sink = torch.tensor([0.0, 4.0, 9.0, -30.0])[torch.arange(nq) % 4]
    scale = 1.0 / math.sqrt(hd)
    want = []
    for q, k, v in zip(qs, ks, vs):
        n, ql = k.shape[0], q.shape[0]
        of = torch.arange(nq) // (nq // nkv)
        s = torch.einsum("ihd,jhd->hij", q.double(), k.double()[:, of]) * scale
        s = s.masked_fill(~(torch.arange(n)[None, :] <= torch.arange(n - ql, n)[:, None])[None], float("-inf"))
        e = torch.exp(s)
        a = e / (e.sum(-1, keepdim=True) + torch.exp(sink.double())[:, None, None])
        want.append(torch.einsum("hij,jhd->ihd", a, v.double()[:, of]))
    want = torch.cat(want)
    q = torch.cat(qs, 0).reshape(-1, nq * hd).to(dt).to(DEV)
    d = {k: v.to(DEV) for k, v in meta.items()}
    T = q.shape[0]
    positions = torch.cat([torch.arange(n - ql, n) for n, ql in zip(lens, q_lens)]).to(torch.int32).to(DEV)
    slot_of_token = torch.cat([torch.full((ql,), int(meta["seq_slot"][b])) for b, ql in enumerate(q_lens)]).to(torch.int32).to(DEV)
    batch = SimpleNamespace(is_decode=max(q_lens) == 1, n_tokens=T, n_seqs=len(lens), max_q_len=max(q_lens), max_kv_len=max(lens),
                            seq_slot=d["seq_slot"], cu_q=d["cu_q"], kv_len=d["kv_len"], positions=positions, slot_of_token=slot_of_token)
    whole = torch.full((T, nq * hd + (72 if strided else 0)), float("nan"), dtype=dt, device=DEV)
    out = whole[:, :nq * hd]
    kc, vc = kc.to(dt).to(DEV), vc.to(dt).to(DEV)
    paged_attention(q, out, batch, kc, vc, d["table"], nq, nkv, hd, scale, 0, sink=sink.to(DEV))
    tol = 3e-2 if dtype == "bfloat16" else 3e-5
    assert (out.cpu().double().reshape(want.shape) - want).abs().max().item() < tol
    if dtype == "bfloat16" and not batch.is_decode and hd in (64, 128, 256):         # the other kernel for prompts
        out.fill_(float("nan"))
        assert kernels.attention_prefill(q, out, kc, vc, d["table"], d["seq_slot"], d["cu_q"], d["kv_len"], len(lens), max(q_lens), nq, nkv,
                                         hd, scale, sink=sink.to(DEV))
        assert (out.cpu().double().reshape(want.shape) - want).abs().max().item() < tol


# ---- the engine -------------------------------------------------------------------------------------------------

class Folder:
    """A model folder with its plain implementation (logits kept per prompt)."""

    def __init__(self, folder):
        self.folder = folder
        self.cfg, self.w = P.load_folder(folder)
        self.kept = {}

    def __call__(self, ids):
        key = tuple(ids)
        if key not in self.kept:
            self.kept[key] = P.forward(self.cfg, self.w, list(ids))
        return self.kept[key]


@pytest.fixture(scope="module", params=sorted(RAVELORN))
def model(request, tmp_path_factory):
    name = request.param
    folder = str(tmp_path_factory.mktemp(f"ravelorn_{name}"))
    write_ravelorn(folder, RAVELORN[name], seed=40 + ord(name[-1]))
    return name, RAVELORN[name], Folder(folder)


def engine(folder, dtype, **kw):
    from rocml_b200 import Engine
    kw.setdefault("max_tokens", 1024)
    return Engine.from_folder(folder, dtype=dtype, **kw)


def assert_rows(got, want, dtype, what):
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} against {tuple(want.shape)}"
    assert bool(torch.isfinite(got).all()), what
    err = ((got.double().cpu() - want.double()).abs() / want.double().abs().amax(dim=-1, keepdim=True).clamp_min(1e-30)).amax(-1)
    assert float(err.max()) < TOL[dtype], f"{what}: off by {float(err.max()):.3g}"
    if len(err) >= 32:
        assert float(err.median()) < MEDIAN[dtype], f"{what}: the median row is off by {float(err.median()):.3g}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts(model, dtype):
    """Lengths around the pages' borders (64), the convolutions' taps, the recurrence's four tokens and its batches of sixteen,
    every place compared, the first tokens among them."""
    from rocml_b200 import StepEntry
    name, cfg, plain = model
    eng = engine(plain.folder, dtype)
    for n in (1, 2, 3, 4, 5, 9, 15, 16, 17, 18, 33, 63, 64, 65, 129, 257):
        ids = prompt(n, n, cfg["vocab"])
        slot = eng.new_sequence()
        got = eng.step([StepEntry(slot, ids, list(range(n)))])
        eng.release(slot)
        assert_rows(got, plain(ids), dtype, f"{name} {dtype} n={n}")
    eng.cache.check_invariants()


def test_every_mechanism_matters(model):
    """The plain implementation with one mechanism taken out or moved by one step is far from itself by many times the 32-bit
    tolerance, so the comparisons of this file would see it missing."""
    name, cfg, plain = model
    ids = prompt(5, 90, cfg["vocab"])
    want = plain(ids)

    def differs(w=None, c=None):
        return rel_err(P.forward(c or plain.cfg, w or plain.w, ids), want) > 30 * TOL["float32"]
    for suffix, value in ((".sink", -40.0), ("norm1.b", 0.0), ("norm2.b", 0.0), ("pos", 0.0), (".A_log", -20.0), (".dt_bias", 0.0),
                          ("mix.norm", 1.0), ("right.norm", 1.0), (".correction", 0.0)):
        w = {k: (torch.full_like(v, value) if k.endswith(suffix) else v) for k, v in plain.w.items()}
        if any(k.endswith(suffix) for k in w):
            assert differs(w) or (suffix == ".correction" and name == "RC"), suffix
    w = {k: (v.roll(1, 1) if k.endswith(".conv") and v.shape[1] > 1 else v) for k, v in plain.w.items()}
    assert differs(w), "conv"
    for path, value in ((("residual_mult",), 0.5 * cfg["residual_mult"]), (("logit_softcap",), 2.0 * cfg["logit_softcap"]),
                        (("layers", 0, "mixer", "left_scale"), 0.2), (("layers", 0, "mixer", "right_scale"), 0.2),
                        (("layers", 0, "mixer", "left", "q_temp", "coef"), 0.0), (("layers", 0, "mixer", "left", "scale"), 0.01)):
        other = json.loads(json.dumps(plain.cfg))
        at = other
        for p in path[:-1]:
            at = at[p]
        at[path[-1]] = value
        assert differs(c=other), path


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("graphs", [False, True])
def test_prompt_then_token_by_token(model, dtype, graphs):
    """The last tokens one by one (state, kept inputs and pages pass from the prompt's step to the single tokens), against the
    same positions of the whole prompt."""
    from rocml_b200 import StepEntry
    name, cfg, plain = model
    eng = engine(plain.folder, dtype, use_graphs=graphs)
    for n, tail in ((150, 80), (41, 40), (200, 3)):
        ids = prompt(300 + n, n, cfg["vocab"])
        want = plain(ids)
        slot = eng.new_sequence()
        head = n - tail
        got = [eng.step([StepEntry(slot, ids[:head], [head - 1])]).clone()]
        for t in range(head, n):
            got.append(eng.step([StepEntry(slot, [ids[t]], [0])]).clone())
        eng.release(slot)
        assert_rows(torch.cat(got, dim=0), want[head - 1:], dtype, f"{name} {dtype} n={n} graphs={graphs}")
    eng.cache.check_invariants()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decoding_from_the_very_first_token(model, dtype):
    from rocml_b200 import StepEntry
    name, cfg, plain = model
    n = 200
    ids = prompt(9, n, cfg["vocab"])
    eng = engine(plain.folder, dtype)
    slot = eng.new_sequence()
    got = [eng.step([StepEntry(slot, [ids[t]], [0])]).clone() for t in range(n)]
    eng.release(slot)
    assert_rows(torch.cat(got, dim=0), plain(ids), dtype, f"{name} {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("piece", [2, 5, 64, 100])
def test_prompts_in_pieces(model, dtype, piece):
    """Steps cut into pieces of 2 to 100 tokens (the engine's work space is that small; 2 is fewer than the taps of a
    convolution): two sequences side by side, every place wanted, then a few tokens one by one."""
    from rocml_b200 import StepEntry
    name, cfg, plain = model
    eng = engine(plain.folder, dtype, max_step_tokens=piece)
    lens = (140, 70) if piece > 2 else (67, 9)
    seqs = [prompt(700 + i, n + 4, cfg["vocab"]) for i, n in enumerate(lens)]
    slots = [eng.new_sequence() for _ in seqs]
    got = eng.step([StepEntry(s, ids[:-4], list(range(len(ids) - 4))) for s, ids in zip(slots, seqs)])
    rows, at = [], 0
    for ids in seqs:
        rows.append([got[at:at + len(ids) - 4].clone()])
        at += len(ids) - 4
    for k in range(4, 0, -1):
        out = eng.step([StepEntry(s, [ids[-k]], [0]) for s, ids in zip(slots, seqs)])
        for i in range(len(seqs)):
            rows[i].append(out[i:i + 1].clone())
    for i, ids in enumerate(seqs):
        assert_rows(torch.cat(rows[i], dim=0), plain(ids), dtype, f"{name} {dtype} piece={piece} seq {i}")
        eng.release(slots[i])
    eng.cache.check_invariants()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batches_against_each_alone_and_reuse(model, dtype):
    """Batches of unequal prompts, then one token each until the shorter ones end; later batches get the slots, pages and
    states that earlier ones gave back.  Every request is compared with the plain implementation of it alone, and in 32-bit
    the batched rows equal the rows of the request stepped alone in the same engine."""
    from rocml_b200 import StepEntry
    name, cfg, plain = model
    eng = engine(plain.folder, dtype, max_tokens=640)
    batches = [[(5, 8), (70, 3), (130, 12), (1, 5)], [(64, 4), (2, 9), (33, 1)], [(190, 6), (90, 2)]]
    for r, batch in enumerate(batches):
        seqs = []
        for j, (plen, ndec) in enumerate(batch):
            ids = prompt(1000 * r + j, plen + ndec, cfg["vocab"])
            seqs.append({"ids": ids, "plen": plen, "slot": eng.new_sequence(), "got": []})
        out = eng.step([StepEntry(s["slot"], s["ids"][:s["plen"]], [s["plen"] - 1]) for s in seqs])
        for i, s in enumerate(seqs):
            s["got"].append(out[i].clone())
            s["pos"] = s["plen"]
        live = list(seqs)
        while live:
            for s in [s for s in live if s["pos"] >= len(s["ids"])]:
                eng.release(s["slot"])
            live = [s for s in live if s["pos"] < len(s["ids"])]
            if not live:
                break
            out = eng.step([StepEntry(s["slot"], [s["ids"][s["pos"]]], [0]) for s in live])
            for i, s in enumerate(live):
                s["got"].append(out[i].clone())
                s["pos"] += 1
        for j, s in enumerate(seqs):
            got = torch.stack(s["got"])
            assert_rows(got, plain(s["ids"])[s["plen"] - 1:], dtype, f"{name} {dtype} batch {r} seq {j}")
            if dtype == "float32" and j == 2:
                slot = eng.new_sequence()
                alone = [eng.step([StepEntry(slot, s["ids"][:s["plen"]], [s["plen"] - 1])]).clone()]
                for t in range(s["plen"], len(s["ids"])):
                    alone.append(eng.step([StepEntry(slot, [s["ids"][t]], [0])]).clone())
                eng.release(slot)
                assert rel_err(got, torch.cat(alone).cpu()) < 1e-5
        eng.cache.check_invariants()
    assert eng.cache.slots.n_held == 0
    for g in eng.cache.kv_groups:
        assert g.pool.n_held == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_state_that_remembers_hundreds_of_tokens(tmp_path, dtype):
    """Decays close to one: the first three tokens still move the logits 500 tokens later (shown on the plain implementation), in a
    slot that another request used before; whole, and with the tail decoded."""
    from rocml_b200 import StepEntry
    cfg = RAVELORN["RA"]
    folder = write_ravelorn(str(tmp_path / "m"), cfg, seed=3, slow_decay=True)
    plain = Folder(folder)
    ids = prompt(21, 520, cfg["vocab"])
    want = plain(ids)
    other = plain([(t + 1) % cfg["vocab"] for t in ids[:3]] + ids[3:])
    assert rel_err(other[-1:], want[-1:]) > 10 * TOL["float32"]
    eng = engine(folder, dtype)
    slot = eng.new_sequence()
    eng.step([StepEntry(slot, prompt(22, 300, cfg["vocab"]), [])])
    eng.release(slot)
    slot = eng.new_sequence()
    got = [eng.step([StepEntry(slot, ids[:480], [479])]).clone()]
    for t in range(480, 520):
        got.append(eng.step([StepEntry(slot, [ids[t]], [0])]).clone())
    eng.release(slot)
    assert_rows(torch.cat(got), want[479:], dtype, f"{dtype} decoded tail")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(model, dtype):
    """A short prompt and 500 tokens one by one under CUDA graphs; the last 40 rows compared."""
    from rocml_b200 import StepEntry
    name, cfg, plain = model
    ids = prompt(77, 520, cfg["vocab"])
    eng = engine(plain.folder, dtype, max_tokens=1024)
    slot = eng.new_sequence()
    eng.step([StepEntry(slot, ids[:20], [])])
    got = []
    for t in range(20, 520):
        r = eng.step([StepEntry(slot, [ids[t]], [0] if t >= 480 else [])])
        if r is not None:
            got.append(r.clone())
    eng.release(slot)
    assert_rows(torch.cat(got), plain(ids)[480:], dtype, f"{name} {dtype}")
    eng.cache.check_invariants()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(model, dtype):
    """Engine.generate (its scheduler, sampler and run-ahead loop) against greedy decoding with the plain implementation,
    for prompts of unequal length in one batch; compared until the first step whose two best logits are closer than the
    tolerance."""
    from rocml_b200 import SamplingParams
    name, cfg, plain = model
    eng = engine(plain.folder, dtype)
    prompts = [prompt(50 + i, n, cfg["vocab"]) for i, n in enumerate((3, 70, 35))]
    outs = eng.generate(prompts, max_new_tokens=12, sampling=SamplingParams(temperature=0.0), ignore_eos=True)
    for ids, out in zip(prompts, outs):
        seq = list(ids)
        for tok in out.tokens:
            logits = P.forward(plain.cfg, plain.w, seq)[-1]
            top2 = torch.topk(logits, 2).values
            if float(top2[0] - top2[1]) < (1e-3 if dtype == "float32" else 0.3) * float(logits.abs().max()):
                break
            assert tok == int(logits.argmax()), f"{name} {dtype}: after {len(seq)} tokens"
            seq.append(tok)
    assert eng.cache.slots.n_held == 0


def test_trace_replay_and_command_line(model, tmp_path):
    """bin/trace_run on a folder of this architecture: a prompt in two steps and two decoded tokens, a second request
    beside it; the logits are the plain implementation's."""
    import os
    import subprocess
    import sys
    import numpy as np
    name, cfg, f = model
    a, b = prompt(1, 40, cfg["vocab"]), prompt(2, 9, cfg["vocab"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:38], "want": [0, 37]}, {"id": "b", "tokens": b[:7], "want": [6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[38:39], "want": [0]}, {"id": "b", "tokens": b[7:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[39:], "want": [0]}, {"id": "b", "tokens": b[8:], "want": [0]}], "end": ["a", "b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", f.folder, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = f(a), f(b)
    V = cfg["vocab"]
    got0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(-1, V))
    assert rel_err(got0, torch.stack([wa[0], wa[37], wb[6]])) < TOL["float32"]
    got2 = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4").reshape(-1, V))
    assert rel_err(got2, torch.stack([wa[39], wb[8]])) < TOL["float32"]
    r = subprocess.run([sys.executable, "-m", "rocml_b200", "generate", "--model", f.folder, "--prompt-ids", "1,2,3", "-n", "5"],
                       capture_output=True, text=True, timeout=600, cwd=root)
    assert r.returncode == 0, r.stderr[-2000:]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_far_back_that_stands_out(tmp_path, dtype):
    """One layer, whose attention looks (by weights made for it) for one token: the logits at the last places of a prompt depend on
    where that token stands hundreds of positions back, in prompts, across pieces and decoded."""
    from rocml_b200 import StepEntry
    cfg = json.loads(json.dumps(RAVELORN["RB"]))
    cfg["layers"] = cfg["layers"][2:3]
    folder = write_ravelorn(str(tmp_path / "m"), cfg, seed=5)
    from safetensors.torch import load_file, save_file
    w = load_file(f"{folder}/model.safetensors")
    # the query of token 77 is the key of token 78, every other token's query its own key
    e77, e78 = w["embed"][77].float(), w["embed"][78].float()
    wk = w["l0.mix.left.k"].float()
    wk = torch.cat([wk[128 * (h // 2):128 * (h // 2) + 128] for h in range(4)])
    w["l0.mix.left.q"] = (wk + torch.outer(wk @ (e78 - e77), e77 / (e77 @ e77))).to(torch.bfloat16)
    w["pos"] = w["pos"] * 0
    save_file({k: v.contiguous() for k, v in w.items()}, f"{folder}/model.safetensors")
    plain = Folder(folder)
    n, far = 420, 37
    ids = [t % 40 for t in prompt(3, n, cfg["vocab"])]
    ids[far], ids[n - 1], ids[n - 20] = 78, 77, 77
    want = plain(ids)
    moved = list(ids)
    moved[far] = 5
    assert rel_err(plain(moved)[-1:], want[-1:]) > 0.1
    eng = engine(folder, dtype)
    slot = eng.new_sequence()
    got = eng.step([StepEntry(slot, ids, [far, n - 20, n - 1])])
    eng.release(slot)
    assert_rows(got, want[[far, n - 20, n - 1]], dtype, f"{dtype} whole")
    slot = eng.new_sequence()
    eng.step([StepEntry(slot, ids[:130], [])])
    got = [eng.step([StepEntry(slot, ids[130:n - 20], [0])]).clone()]
    for t in range(n - 20, n):
        got.append(eng.step([StepEntry(slot, [ids[t]], [0])]).clone())
    eng.release(slot)
    assert_rows(torch.cat(got), torch.cat([want[130:131], want[n - 20:]]), dtype, f"{dtype} decoded")


def test_choices_that_follow_the_tokens(tmp_path):
    """Routers whose choices follow the tokens (32-bit): rows whose every router decides by more than rounding are compared,
    up to the sequence's first close call; those must be most."""
    from rocml_b200 import StepEntry
    for name in ("RA", "RB"):
        cfg = RAVELORN[name]
        plain = Folder(write_ravelorn(str(tmp_path / name), cfg, seed=11, fixed_routes=False))
        ids, gaps = prompt(8, 160, cfg["vocab"]), []
        want = P.forward(plain.cfg, plain.w, ids, gaps=gaps)
        margin = torch.stack(gaps).amin(0)
        close_call = (margin < 3e-6).nonzero()
        n = int(close_call[0]) if len(close_call) else len(ids)
        assert n > 80
        chosen = [P.route(torch.randn(50, cfg["width"]).double(), cfg["layers"][0]["mlp"]["router"], P.sub(plain.w, "l0.mlp."))[0]]
        assert len({tuple(sorted(r)) for r in chosen[0].tolist()}) > 5
        eng = engine(plain.folder, "float32")
        slot = eng.new_sequence()
        got = eng.step([StepEntry(slot, ids, list(range(n)))])
        assert_rows(got, want[:n], "float32", name)


def test_a_sequence_may_not_outgrow_the_position_table(tmp_path):
    from rocml_b200 import StepEntry
    from rocml_b200.errors import ContextOverflow
    cfg = json.loads(json.dumps(RAVELORN["RC"]))
    cfg["max_positions"] = 70
    eng = engine(write_ravelorn(str(tmp_path / "m"), cfg, seed=2), "float32")
    slot = eng.new_sequence()
    eng.step([StepEntry(slot, prompt(1, 69, 97), [])])
    eng.step([StepEntry(slot, [3], [0])])
    with pytest.raises(ContextOverflow):
        eng.step([StepEntry(slot, [3], [0])])


# ---- configurations drawn at random -----------------------------------------------------------------------------

def random_configuration(seed):
    from tiny_models import _rchan, _rdelta, _rleft, _rmoe, _rpar
    g = torch.Generator().manual_seed(3000 + seed)

    def pick(*xs):
        return xs[int(torch.randint(0, len(xs), (1,), generator=g))]

    def delta(ranks):
        kv = pick(1, 2, 3)
        return _rdelta(kv * pick(1, 2, 4), kv, pick(4, 8, 20, 32, 64, 100, 128), pick(4, 9, 24, 64, 80), pick(1, 2, 3, 4, 5, 8),
                       (pick(3, 8, 24, 40), pick(5, 16, 32)) if ranks else None)

    def moe():
        experts, identity = pick(1, 2, 5, 8, 12), pick(0, 1, 2, 4)
        return pick(None, _rmoe(experts, identity, min(pick(1, 2, 3, 6), experts + identity), pick(16, 24, 40, 64)))
    layers = []
    for i in range(pick(1, 2, 3, 4)):
        if pick(True, False):
            layers.append(_rchan(delta(True), moe()))
        else:
            kv = pick(1, 2, 3)
            left = _rleft(kv * pick(1, 2, 4), kv, pick(8, 16, 32, 64, 40, 128), pick(8, 32, 64, 48, 128), pick(0.1, 0.3, 0.7), (pick(0.0, 0.4, 1.0), pick(1, 7, 64, 1000)))
            layers.append(_rpar(left, delta(False), pick(1.0, 0.3, -0.8, 0.0), pick(0.5, 1.0, 1.7), moe()))
    return {"architecture": "Ravelorn", "vocab": pick(50, 101, 256), "width": pick(48, 64, 96, 136), "max_positions": pick(256, 300, 2000),
            "norm": {"eps": pick(1e-6, 1e-5)}, "residual_mult": pick(0.3, 0.6, 1.0), "logit_softcap": pick(2.0, 10.0, 50.0), "layers": layers}


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(tmp_path, seed):
    """A configuration drawn at random: a whole prompt, the same in pieces of 50 with a tail decoded under graphs, and two
    requests side by side, in 32-bit (sharp) and bfloat16."""
    from rocml_b200 import StepEntry
    cfg = random_configuration(seed)
    folder = str(tmp_path / "m")
    write_ravelorn(folder, cfg, seed)
    plain = Folder(folder)
    ids, other = prompt(seed, 210, cfg["vocab"]), prompt(seed + 50, 75, cfg["vocab"])
    for dtype in ("float32", "bfloat16"):
        eng = engine(folder, dtype)
        slot = eng.new_sequence()
        got = eng.step([StepEntry(slot, ids, list(range(210)))])
        eng.release(slot)
        assert_rows(got, plain(ids), dtype, f"seed {seed} {dtype} whole: {json.dumps(cfg)}")
        eng = engine(folder, dtype, max_step_tokens=50)
        a, b = eng.new_sequence(), eng.new_sequence()
        got = eng.step([StepEntry(a, ids[:180], [0, 179]), StepEntry(b, other[:60], [59])]).clone()
        assert_rows(got, torch.stack([plain(ids)[0], plain(ids)[179], plain(other)[59]]), dtype, f"seed {seed} {dtype} pieces")
        rows_a, rows_b = [], []
        for t in range(15):
            out = eng.step([StepEntry(a, [ids[180 + t]], [0]), StepEntry(b, [other[60 + t]], [0])])
            rows_a.append(out[0].clone())
            rows_b.append(out[1].clone())
        assert_rows(torch.stack(rows_a), plain(ids)[180:195], dtype, f"seed {seed} {dtype} decoded a")
        assert_rows(torch.stack(rows_b), plain(other)[60:75], dtype, f"seed {seed} {dtype} decoded b")
        eng.release(a)
        eng.release(b)
        eng.cache.check_invariants()
