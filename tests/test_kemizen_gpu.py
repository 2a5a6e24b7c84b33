"""Kemizen on the GPU against the plain implementation (tests/plain_kemizen.py): each mechanism alone, then the
engine in every way of cutting and batching, in 32-bit and in bfloat16.

Tolerances are a fraction of the largest |logit| of the row compared.  float32: sums of a few hundred terms in
another order than the plain implementation's float64.  bfloat16: activations are rounded to 8 bits of mantissa
between kernels, a dozen roundings a layer.  A norm on a small result (a difference of two maps that nearly cancels, a memory's read-out
whose terms cancel) multiplies its rounding in both: the plain implementation in 32-bit is itself off by 1e-4 and more in single rows of these
random models, by less than 1e-6 in the median row.  So the median row is held to a tight bound, nine rows of ten to a middle one and
every row to a loose one.
"""
import json
from types import SimpleNamespace

import pytest
import torch

import plain_kemizen as P
from tiny_models import KEMIZEN, prompt, write_kemizen

pytestmark = pytest.mark.gpu

TOL = {"float32": 1e-3, "bfloat16": 6e-1}
MOST = {"float32": 1e-4, "bfloat16": 1.5e-1}
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


# ---- attention: the soft cap in every kernel -----------------------------------------------------------------------------

def paged(k, v, n_pages, seed):
    """Keys and values [T, G, hd] in pages that lie in no order, beside pages full of garbage: (k cache, v cache, block table)."""
    T, G, hd = k.shape
    g = torch.Generator().manual_seed(seed)
    kc = torch.full((n_pages, G, 64, hd), 50.0).to(k.dtype)
    vc = torch.full((n_pages, G, 64, hd), 50.0).to(k.dtype)
    need = (T + 63) // 64
    pages = torch.randperm(n_pages, generator=g)[:need].tolist()
    for i, p in enumerate(pages):
        a, b = i * 64, min(T, i * 64 + 64)
        kc[p, :, :b - a] = k[a:b].transpose(0, 1)
        vc[p, :, :b - a] = v[a:b].transpose(0, 1)
    return kc.to(DEV), vc.to(DEV), i32([[-1] * need, pages])


def capped_case(nq, nkv, hd, T, window, cap, scale, dtype, seed, far=None):
    """Queries, keys, values and the plain result; the last query and key ``far`` positions back are made so that that score stands out."""
    torch.manual_seed(seed)
    q, k, v = (torch.randn(T, n, hd) for n in (nq, nkv, nkv))
    if far is not None:
        q[T - 1, 0] = 3.0 * k[T - 1 - far, 0]
    q, k, v = (x.to(DT[dtype]) for x in (q, k, v))
    of = torch.arange(nq) // (nq // nkv)
    s = P.capped(torch.einsum("ihd,jhd->hij", q.double(), k.double()[:, of]) * scale, cap)
    want = torch.einsum("hij,jhd->ihd", P.weights(s, list(range(T)), window), v.double()[:, of]).reshape(T, nq * hd)
    return q, k, v, want


@pytest.mark.parametrize("nq, nkv, hd", [(8, 1, 64), (4, 2, 128), (2, 2, 256), (6, 2, 48), (20, 1, 64)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cap, scale", [(2.0, 0.4), (30.0, 0.1), (50.0, 4.0)])
def test_soft_cap_in_every_attention_kernel(nq, nkv, hd, dtype, cap, scale):
    """Whole prompts, a piece behind a cache, and single tokens; scores far below, around and far above the cap; with a window, at whose
    edge one key stands out."""
    from rocml_b200 import kernels
    from rocml_b200.parts.attention import paged_attention
    tol = 2e-2 if dtype == "bfloat16" else 2e-5
    for T, window, far in ((150, 0, 140), (150, 70, 69), (150, 70, 70), (7, 0, 3)):
        q, k, v, want = capped_case(nq, nkv, hd, T, window, cap, scale, dtype, T + hd, far)
        kc, vc, table = paged(k, v, 7, T)
        for first in (0, T // 3, T - 1):
            n = T - first
            cu, kv, slot = i32([0, n]), i32([T]), i32([1])
            batch = SimpleNamespace(is_decode=n == 1, n_tokens=n, n_seqs=1, max_q_len=n, max_kv_len=T, seq_slot=slot, cu_q=cu, kv_len=kv,
                                    positions=i32(list(range(first, T))), slot_of_token=i32([1] * n))
            rows = q[first:].reshape(n, nq * hd).to(DEV)
            out = torch.zeros_like(rows)
            paged_attention(rows, out, batch, kc, vc, table, nq, nkv, hd, scale, window, softcap=cap)
            assert close(out, want[first:], tol), (T, window, first)
            if dtype == "bfloat16" and hd in (64, 128, 256) and n > 1:
                out2 = torch.zeros_like(rows)
                assert kernels.attention_prefill(rows, out2, kc, vc, table, slot, cu, kv, 1, n, nq, nkv, hd, scale, window, softcap=cap)
                assert close(out2, want[first:], tol), ("mma.sync", T, window, first)
                kernels.attention_generic(rows, out2, kc, vc, table, slot, cu, kv, 1, n, nq, nkv, hd, scale, window, softcap=cap)
                assert close(out2, want[first:], tol), ("plain", T, window, first)
    kernels.check_status(torch.device(DEV))


# ---- differential attention -------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("parts", [0, 3])
@pytest.mark.parametrize("heads, kv, dim, vdim, dims", [(3, 1, 64, 128, 64), (4, 2, 64, 128, 16), (2, 2, 64, 128, 0), (4, 2, 12, 20, 8),
                                                        (1, 1, 6, 40, 2), (2, 1, 32, 96, 32)])
def test_two_maps_a_head(dtype, parts, heads, kv, dim, vdim, dims):
    """Norm and rotation per map; a stored key is its two maps side by side; a query becomes two rows with zeros in the other's place."""
    from rocml_b200 import kernels
    torch.manual_seed(dim + heads + parts)
    T, eps = 9, 1e-5
    hdp = -(-max(2 * dim, vdim) // 16) * 16
    width = heads * 2 * dim + kv * (2 * dim + vdim)
    x = torch.randn(max(1, parts), T, width)
    proj = x if parts else x[0].to(DT[dtype])
    row = (x.sum(0) if parts else proj.float()).double()
    wq, wk = 1 + 0.3 * torch.randn(dim), 1 + 0.3 * torch.randn(dim)
    pos = [5, 6, 7, 64, 65, 3, 0, 200, 63]
    slots = [1, 1, 1, 0, 0, 2, -1, 2, 0]
    table = i32([[3, 0, -1, -1], [5, -1, -1, -1], [1, -1, -1, 2]])
    k_cache, v_cache = (torch.full((6, kv, 64, hdp), 9.0, dtype=DT[dtype], device=DEV) for _ in range(2))
    q = torch.full((T, 2 * heads * hdp), 9.0, dtype=DT[dtype], device=DEV)
    rot = {"base": 5000.0, "dims": dims, "scaling": {"factor": 4.0, "original": 100, "fast": 8.0, "slow": 1.0}}
    inv = mag = cs = None
    if dims:
        inv, mag = P.frequencies(rot)
        inv = inv.float().to(DEV)
        cs = kernels.rope_table(i32(pos), inv, T, mag)
    kernels.qk_norm_rope_cache(proj.to(DEV), q, T, 2 * heads, kv, dim, wq.to(DEV), wk.to(DEV), eps, inv, dims, i32(pos), i32(slots), table,
                               k_cache, v_cache, cos_sin=cs, v_head_dim=vdim, padded_head_dim=hdp, maps=2)

    def turned(y, n, w):
        y = P.rms(y.reshape(T, n, dim), eps) * w.double()
        return P.rotate(y, pos, rot) if dims else y
    qd, kd = heads * 2 * dim, kv * 2 * dim
    wantq, wantk = turned(row[:, :qd], 2 * heads, wq), turned(row[:, qd:qd + kd], 2 * kv, wk).reshape(T, kv, 2 * dim)
    wantv = row[:, qd + kd:].reshape(T, kv, vdim)
    tol = 1e-2 if dtype == "bfloat16" else 3e-5           # (a 32-bit angle of a few hundred)
    for t in range(T):
        got = q[t].reshape(heads, 2, hdp)
        if slots[t] < 0:
            assert bool((got == 9.0).all())
            continue
        for m in range(2):
            assert close(got[:, m, m * dim:(m + 1) * dim], wantq[t].reshape(heads, 2, dim)[:, m], tol)
            rest = torch.cat([got[:, m, :m * dim], got[:, m, (m + 1) * dim:]], dim=-1)
            assert float(rest.abs().sum()) == 0.0
        page = int(table[slots[t], pos[t] // 64])
        gk, gv = k_cache[page, :, pos[t] % 64], v_cache[page, :, pos[t] % 64]
        assert close(gk[:, :2 * dim], wantk[t], tol) and float(gk[:, 2 * dim:].abs().sum()) == 0.0
        assert close(gv[:, :vdim], wantv[t], tol) and float(gv[:, vdim:].abs().sum()) == 0.0
    untouched = 6 * 64 - sum(s >= 0 for s in slots)
    assert int((k_cache == 9.0).all(-1).all(1).sum()) == untouched


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads, hdp, vd, T", [(3, 128, 128, 40), (4, 48, 20, 9), (1, 16, 7, 5), (2, 512, 512, 3), (16, 64, 64, 300)])
def test_difference_of_two_maps(dtype, heads, hdp, vd, T):
    from rocml_b200 import kernels
    torch.manual_seed(T + vd)
    o = torch.randn(T, 2 * heads * hdp).to(DT[dtype])
    o[:, hdp:2 * hdp] = (o[:, :hdp].float() * 1.6).to(DT[dtype])          # a head whose maps agree but for a factor: a small difference
    out = torch.full((T, heads * vd + 4), 5.0, dtype=DT[dtype], device=DEV)
    slots = [0] * T
    slots[T // 2] = -1
    kernels.diff_heads(o.to(DEV), 0.6, 1e-5, 0.3, out[:, :heads * vd], heads, hdp, vd, i32(slots), T)
    x = o.double().reshape(T, heads, 2, hdp)[..., :vd]
    want = (P.rms(x[:, :, 0] - 0.6 * x[:, :, 1], 1e-5) * 0.3).reshape(T, heads * vd)
    keep = [t for t in range(T) if slots[t] >= 0]
    assert close(out[keep, :heads * vd], want[keep], 1e-2 if dtype == "bfloat16" else 1e-5)
    assert bool((out[:, heads * vd:] == 5.0).all()) and bool((out[T // 2] == 5.0).all())


# ---- short convolutions, the norm over whole projections ------------------------------------------------------------------------

@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("channels", [64, 30, 516])
@pytest.mark.parametrize("dtype, parts", [("bfloat16", 0), ("float32", 0), ("float32", 3)])
def test_causal_convolution_over_steps(taps, channels, dtype, parts):
    """Without an activation, with and without bias, over steps of one token to a hundred; slots that others used before."""
    from rocml_b200 import kernels
    torch.manual_seed(taps * channels)
    col0, width = 4, channels + 12
    w, bias = torch.randn(channels, taps), torch.randn(channels) if channels != 64 else None
    kept = torch.zeros(3, max(1, taps - 1), channels, device=DEV)
    steps = [[70, 3], [1, 1], [2, 101], [1, 2], [33, 1]]
    total = [sum(s[i] for s in steps) for i in range(2)]
    rows = [torch.randn(max(1, parts), n, width).to(DT[dtype]) for n in total]
    want = [P.causal_conv(r.double().sum(0)[:, col0:col0 + channels], w.double()) + (0 if bias is None else bias.double()) for r in rows]
    at = [0, 0]
    for step in steps:
        x = torch.cat([rows[i][:, at[i]:at[i] + n] for i, n in enumerate(step)], dim=1).contiguous().to(DEV)
        T = sum(step)
        out = torch.zeros(T, channels, device=DEV)
        kernels.causal_conv(x if parts else x[0], T, col0, channels, taps, w.to(DEV), None if bias is None else bias.to(DEV), "none",
                            kept if taps > 1 else None, i32([2, 0, -1]), i32(cu_of(step + [0])), 3, max(step), out)
        y = 0
        for i, n in enumerate(step):
            assert close(out[y:y + n], want[i][at[i]:at[i] + n], 2e-6), (step, i)
            at[i] += n
            y += n
    assert float(kept[1].abs().sum()) == 0.0


@pytest.mark.parametrize("dtype, parts", [("bfloat16", 0), ("float32", 0), ("float32", 2)])
@pytest.mark.parametrize("nq, nkv, hd, vd, dims", [(4, 2, 128, 128, 128), (2, 1, 64, 64, 16), (3, 3, 10, 7, 4), (6, 2, 20, 12, 12), (2, 2, 64, 64, 0)])
def test_norm_over_whole_projections(dtype, parts, nq, nkv, hd, vd, dims):
    """Queries and keys normalised over all their heads, rotated by halves, cached; the four-entries-a-thread path and the other."""
    from rocml_b200 import kernels
    torch.manual_seed(hd + nq)
    act = "bfloat16" if dtype == "bfloat16" else "float32"
    T, eps = 6, 1e-5
    hdp = -(-max(hd, vd) // 16) * 16
    qw, kw = nq * hd, nkv * hd
    x = torch.randn(max(1, parts), T, qw + kw + nkv * vd + 4)
    x = x if parts else x[0].to(DT[dtype])
    row = (x.sum(0) if parts else x.float()).double()
    wq, wk = 1 + 0.3 * torch.randn(qw), 1 + 0.3 * torch.randn(kw)
    pos, slots = [0, 63, 64, 5, 130, 2], [0, 0, 0, 1, 0, -1]
    table = i32([[4, 2, 0], [1, -1, -1]])
    kc, vc = (torch.full((5, nkv, 64, hdp), 9.0, dtype=DT[act], device=DEV) for _ in range(2))
    q = torch.zeros(T, nq * hdp, dtype=DT[act], device=DEV)
    rot = {"base": 700.0, "dims": dims}
    cs = kernels.rope_table(i32(pos), P.frequencies(rot)[0].float().to(DEV), T) if dims else None
    kernels.wide_norm_rope_cache(x.to(DEV), q, T, nq, nkv, hd, vd, hdp, wq.to(DEV), wk.to(DEV), eps, None, cs, dims, False, i32(pos), i32(slots),
                                 table, kc, vc)

    def turned(y, n):
        y = y.reshape(T, n, hd)
        return P.rotate(y, pos, rot) if dims else y
    wantq = turned(P.rms(row[:, :qw], eps) * wq.double(), nq)
    wantk = turned(P.rms(row[:, qw:qw + kw], eps) * wk.double(), nkv)
    wantv = row[:, qw + kw:qw + kw + nkv * vd].reshape(T, nkv, vd)
    tol = 1e-2 if act == "bfloat16" else 5e-6
    for t in range(T - 1):
        page = int(table[slots[t], pos[t] // 64])
        gk, gv = kc[page, :, pos[t] % 64], vc[page, :, pos[t] % 64]
        assert close(q[t].reshape(nq, hdp)[:, :hd], wantq[t], tol) and float(q[t].reshape(nq, hdp)[:, hd:].abs().sum()) == 0.0
        assert close(gk[:, :hd], wantk[t], tol) and close(gv[:, :vd], wantv[t], tol)
        assert float(gk[:, hd:].abs().sum()) == 0.0 and float(gv[:, vd:].abs().sum()) == 0.0


# ---- the matrix memory ----------------------------------------------------------------------------------------------------------

MEMORY_SIZES = [(2, 64, 32), (1, 256, 96), (3, 128, 64), (1, 192, 32), (4, 12, 20), (1, 9, 5), (2, 100, 70), (2, 64, 40)]


def memory_case(heads, dim, vdim, cap, total, parts, dtype, seed, forget=3.0):
    torch.manual_seed(seed)
    qk, vw = heads * dim, heads * vdim
    off = {"q": 8, "k": 8 + qk, "v": 8 + 2 * qk}
    width = -(-(8 + 2 * qk + vw) // 8) * 8
    rows, gates, want = [], [], []
    for n in total:
        x = torch.randn(max(1, parts), n, width).to(DT[dtype])
        z = torch.randn(2, n, 2 * heads + 1) * 2.0            # partial sums of the gates: [i | f | unused]
        z[0, :, heads:2 * heads] += forget
        z[0, min(3, n - 1), :heads] += 8.0                    # one early token that must still be found
        r, s = x.double().sum(0), z.double().sum(0)
        q = r[:, off["q"]:off["q"] + qk].reshape(n, heads, dim) * dim ** -0.5
        k = r[:, off["k"]:off["k"] + qk].reshape(n, heads, dim)
        v = r[:, off["v"]:off["v"] + vw].reshape(n, heads, vdim)
        i, f = P.capped(s[:, :heads], cap), P.log_sigmoid(P.capped(s[:, heads:2 * heads], cap))
        rows.append(x)
        gates.append(z)
        below = []
        o, last = P.mlstm_scan(q, k, v, i, f, below=below)
        want.append((o, torch.stack(below), last))
    return off, rows, gates, want


@pytest.mark.parametrize("sizes", MEMORY_SIZES)
@pytest.mark.parametrize("dtype, parts", [("bfloat16", 0), ("float32", 0), ("float32", 2)])
@pytest.mark.parametrize("cap, forget", [(15.0, 3.0), (90.0, -60.0), (3.0, 8.0)])
def test_matrix_memory_over_steps(sizes, dtype, parts, cap, forget):
    """The running maximum, the state, the sum of keys and the divisor over prompts, pieces and single tokens; two sequences side by
    side with a padding sequence; gates that forget slowly and ones whose exponents would overflow without the maximum."""
    from rocml_b200 import kernels
    heads, dim, vdim = sizes
    steps = [[70, 3], [1, 1], [2, 131], [1, 2], [64, 1], [1, 1]]
    total = [sum(s[i] for s in steps) for i in range(2)]
    off, rows, gates, want = memory_case(heads, dim, vdim, cap, total, parts, dtype, dim + heads, forget)
    S, n, m = torch.zeros(4, heads, dim, vdim, device=DEV), torch.zeros(4, heads, dim, device=DEV), torch.zeros(4, heads, 2, device=DEV)
    slots, at = [2, 0], [0, 0]
    got = [[], []]
    for step in steps:
        x = torch.cat([rows[i][:, at[i]:at[i] + k] for i, k in enumerate(step)], dim=1).contiguous().to(DEV)
        x = x if parts else x[0]
        z = torch.cat([gates[i][:, at[i]:at[i] + k] for i, k in enumerate(step)], dim=1).contiguous().to(DEV)
        T = sum(step)
        pos = i32([p for i, k in enumerate(step) for p in range(at[i], at[i] + k)])
        o = torch.zeros(T, heads * vdim, device=DEV)
        den = torch.zeros(T, heads, device=DEV)
        args = (i32(slots + [-1]), i32(cu_of(step + [0])))
        if max(step) == 1:
            kernels.mlstm_step(x, off["q"], off["k"], off["v"], z, 0, heads, cap, dim ** -0.5, 1e-6, heads, dim, vdim, S, n, m, *args, pos, 2, o, den)
        else:
            keep, add, em = (torch.zeros(heads, T, device=DEV) for _ in range(3))
            kernels.mlstm_gates(z, T, 0, heads, cap, heads, m, *args, pos, 3, max(step), keep, add, em)
            kernels.mlstm_blocks(x, T, off["q"], off["k"], off["v"], dim ** -0.5, 1e-6, heads, dim, vdim, keep, add, em, S, n, *args, 3, o, den)
        b = 0
        for i, k in enumerate(step):
            got[i].append((o[b:b + k].reshape(k, heads, vdim).cpu(), den[b:b + k].cpu()))
            at[i] += k
            b += k
    tol = 2e-5
    for i in range(2):
        o, below, (ws, wn, wm) = want[i]
        # apart, as the kernels give them: their quotient may divide by a product that nearly cancels
        assert close(torch.cat([g[1] for g in got[i]]), below, tol), i
        assert close(torch.cat([g[0] for g in got[i]]), o * below[..., None], tol), i
        assert close(S[slots[i]], ws, tol) and close(n[slots[i]], wn, tol)
        assert close(m[slots[i], :, (total[i] - 1) & 1], wm, 1e-5)
    assert float(S[1].abs().sum()) == 0.0 and float(S[3].abs().sum()) == 0.0


def test_which_memory_runs_on_the_tensor_cores():
    from rocml_b200 import kernels
    x = torch.zeros(4, 1024, dtype=torch.bfloat16, device=DEV)
    assert kernels.mlstm_chains(x, 0, 128, 256, 64, 32) and kernels.mlstm_chains(x, 8, 136, 264, 256, 96)
    assert not kernels.mlstm_chains(x, 4, 128, 256, 64, 32) and not kernels.mlstm_chains(x, 0, 128, 256, 64, 40)
    assert not kernels.mlstm_chains(x, 0, 128, 256, 100, 32) and not kernels.mlstm_chains(x.float(), 0, 128, 256, 64, 32)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_norm_of_divided_heads_and_gate(dtype):
    from rocml_b200 import kernels
    for heads, vd in ((3, 20), (1, 64), (2, 7)):
        torch.manual_seed(vd)
        T, W = 7, heads * vd
        o, gate, den, w = torch.randn(T, W), torch.randn(T, W + 3).to(DT[dtype]), torch.rand(T, heads) + 1e-3, 1 + 0.3 * torch.randn(W)
        out = torch.zeros(T, W, dtype=DT[dtype], device=DEV)
        kernels.group_norm_gate(o.to(DEV), gate.to(DEV), 3, w.to(DEV), 1e-3, heads, "sigmoid", out, i32([0] * T), T, divisor=den.to(DEV))
        want = P.rms(o.double().reshape(T, heads, vd) / den.double()[..., None], 1e-3).reshape(T, W) * w.double() * torch.sigmoid(gate.double()[:, 3:])
        assert close(out, want, 1e-2 if dtype == "bfloat16" else 1e-5), (heads, vd)


# ---- the recurrent block -----------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("blocks, part", [(2, 64), (3, 80), (1, 256), (4, 10), (1, 13), (2, 96)])
@pytest.mark.parametrize("w_dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rate", [-5.0, 0.5])
def test_gated_linear_recurrent_unit_over_steps(blocks, part, w_dtype, rate):
    """Gates, decay and state over prompts, pieces and single tokens, slow decays (where 1 - a^2 is a small difference) and fast ones; the
    state of a slot that is not in the step stays."""
    from rocml_b200 import kernels
    torch.manual_seed(blocks * part)
    width = blocks * part
    w = {"ra": torch.randn(blocks, part, part) * 0.3, "ri": torch.randn(blocks, part, part) * 0.3, "ra.b": torch.randn(blocks, part),
         "ri.b": torch.randn(blocks, part), "lam": torch.randn(width) + rate}
    w["ra"], w["ri"] = w["ra"].to(DT[w_dtype]), w["ri"].to(DT[w_dtype])
    w64 = {k: v.double() for k, v in w.items()}
    neg = (-8.0 * P.softplus(w64["lam"])).float().to(DEV)
    dev = [w["ra"].to(DEV), w["ri"].to(DEV), w["ra.b"].reshape(-1).to(DEV), w["ri.b"].reshape(-1).to(DEV), neg]
    steps = [[150, 3], [1, 1], [2, 65], [1, 2], [40, 1], [1, 1]]
    total = [sum(s[i] for s in steps) for i in range(2)]
    us = [torch.randn(n, width) for n in total]
    ys = [torch.randn(n, width + 5).to(DT[w_dtype]) for n in total]
    want = []
    for u, y in zip(us, ys):
        s, last = P.rglru_scan(*P.rglru_gates(u.double(), w64))
        want.append((s * P.gelu_tanh(y.double()[:, :width]) * 0.7, last))
    state = torch.zeros(4, width, device=DEV)
    state[3] = 4.0
    slots, at, got = [2, 0], [0, 0], [[], []]
    for step in steps:
        T = sum(step)
        u = torch.cat([us[i][at[i]:at[i] + n] for i, n in enumerate(step)]).to(DEV)
        y = torch.cat([ys[i][at[i]:at[i] + n] for i, n in enumerate(step)]).to(DEV)
        out = torch.zeros(T, width + 3, dtype=DT[w_dtype], device=DEV)[:, :width]
        if max(step) == 1:
            kernels.rglru_step(u, T, *dev, y[:, :width], 0.7, state, i32(slots), out)
        else:
            ax = torch.zeros(T, width, 2, device=DEV)
            kernels.rglru_gates(u, T, *dev, ax)
            kernels.rglru_scan(ax, T, y[:, :width], 0.7, state, i32(slots + [-1]), i32(cu_of(step + [0])), 3, out)
        b = 0
        for i, n in enumerate(step):
            got[i].append(out[b:b + n].cpu())
            at[i] += n
            b += n
    for i in range(2):
        assert close(torch.cat(got[i]), want[i][0], 1e-2 if w_dtype == "bfloat16" else 1e-5), i
        assert close(state[slots[i]], want[i][1], 1e-5), i
    assert float(state[1].abs().sum()) == 0.0 and bool((state[3] == 4.0).all())


def test_gates_on_the_tensor_cores_are_those_of_32_bit_numbers():
    """The inputs enter as three bfloat16 numbers each: the products of a width of 256 agree with FMA to 32-bit rounding."""
    from rocml_b200 import kernels
    torch.manual_seed(3)
    blocks, part, T = 3, 256, 130
    u = torch.randn(T, blocks * part, device=DEV) * torch.logspace(-2, 1, blocks * part, device=DEV)
    ra, ri = ((torch.randn(blocks, part, part, device=DEV) * 0.01).to(torch.bfloat16) for _ in range(2))
    zero, rate = torch.zeros(blocks * part, device=DEV), torch.full((blocks * part,), -0.3, device=DEV)
    tc, fma = torch.zeros(T, blocks * part, 2, device=DEV), torch.zeros(T, blocks * part, 2, device=DEV)
    kernels.rglru_gates(u, T, ra, ri, zero, zero, rate, tc)
    kernels.rglru_gates(u, T, ra.float(), ri.float(), zero, zero, rate, fma)
    w = {"ra": ra.cpu().double(), "ri": ri.cpu().double(), "ra.b": torch.zeros(blocks, part).double(), "ri.b": torch.zeros(blocks, part).double(),
         "lam": torch.log(torch.expm1(torch.full((blocks * part,), 0.3 / 8.0).double()))}
    want = torch.stack(P.rglru_gates(u.cpu().double(), w), dim=-1)
    size = torch.tensor([1.0, 0.0]).double() + torch.tensor([0.0, 1.0]).double() * u.cpu().double().abs()[..., None]
    err = [float(((x.cpu().double() - want) / size).abs().max()) for x in (tc, fma)]
    assert err[0] < 2e-6 and err[0] < 3 * err[1] + 2e-7, err


# ---- two results of one sublayer, the feed-forward ------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T, H, na, nb", [(5, 20, 1, 3), (9, 131, 2, 1), (300, 256, 1, 1), (3, 4096, 8, 4)])
def test_norms_of_two_results_and_their_sum(dtype, T, H, na, nb):
    from rocml_b200 import kernels
    torch.manual_seed(H)
    a, b, x = torch.randn(na, T, H) * 0.01, torch.randn(nb, T, H), torch.randn(T, H)
    wa, wb, w = (1 + 0.3 * torch.randn(H) for _ in range(3))
    v = 0.5 * (P.rms(a.double().sum(0), 1e-4) * wa.double() + P.rms(b.double().sum(0), 1e-4) * wb.double())
    dev = [t.to(DEV) for t in (a, b, wa, wb)]
    out_v = torch.zeros(T, H, device=DEV)
    kernels.pair_norm(*dev, 1e-4, 0.5, T, out_v=out_v)
    assert close(out_v, v, 3e-6)
    resid, out = x.clone().to(DEV), torch.zeros(T, H, dtype=DT[dtype], device=DEV)
    kernels.pair_norm(*dev, 1e-4, 0.5, T, resid=resid, weight=w.to(DEV), eps=1e-3, mult=0.4, out=out)
    want = x.double() + 0.4 * P.rms(v, 1e-3) * w.double()
    assert close(resid, want, 3e-6) and close(out, want, 1e-2 if dtype == "bfloat16" else 3e-6)


@pytest.mark.parametrize("kind", ["gelu", "gelu_tanh", "silu"])
def test_activations_alone_and_in_the_products_epilogue(kind):
    from rocml_b200 import kernels
    act = {"gelu": P.gelu_erf, "gelu_tanh": P.gelu_tanh, "silu": lambda z: z * torch.sigmoid(z)}[kind]
    torch.manual_seed(1)
    for shape, in_dt, out_dt in (((3, 5, 21), "float32", "float32"), ((1, 300, 64), "bfloat16", "bfloat16"), ((9, 7, 36), "float32", "bfloat16")):
        x = (torch.randn(shape) * 2).to(DT[in_dt])
        out = torch.zeros(shape[1:], dtype=DT[out_dt], device=DEV)
        kernels.unary_act(x.to(DEV) if shape[0] > 1 else x[0].to(DEV), out, kind)
        assert close(out, act(x.double().sum(0)), 1e-2 if out_dt == "bfloat16" else 2e-6), (shape, in_dt)
    for M, N, K, bias in ((300, 512, 192, False), (513, 320, 64, True), (257, 256, 1024, False)):
        x, w, b = (torch.randn(M, K) * 0.5).to(torch.bfloat16), (torch.randn(N, K) * 0.2).to(torch.bfloat16), torch.randn(N)
        out = torch.zeros(M, N, dtype=torch.bfloat16, device=DEV)
        assert kernels.gemm_tcgen05_act(x.to(DEV), w.to(DEV), out, kind, b.to(DEV) if bias else None)
        assert close(out, act(x.double() @ w.double().T + (b.double() if bias else 0)), 1e-2), (M, N, K)
    assert not kernels.gemm_tcgen05_act(x[:100].to(DEV), w.to(DEV), out[:100], kind)
    kernels.check_status(torch.device(DEV))


# ---- the engine, in every way of cutting and batching ----------------------------------------------------------------------------------

class Folder:
    """A model folder with the plain implementation beside it; whole sequences it has computed are kept."""

    def __init__(self, folder):
        self.folder = folder
        self.cfg, self.w = P.load_folder(folder)
        self.kept = {}

    def __call__(self, ids):
        key = tuple(ids)
        if key not in self.kept:
            self.kept[key] = P.forward(self.cfg, self.w, list(ids))
        return self.kept[key]


@pytest.fixture(scope="module", params=sorted(KEMIZEN))
def model(request, tmp_path_factory):
    name = request.param
    folder = str(tmp_path_factory.mktemp(f"kemizen_{name}"))
    write_kemizen(folder, KEMIZEN[name], seed=60 + ord(name[-1]))
    return name, KEMIZEN[name], Folder(folder)


def engine(folder, dtype, **kw):
    from rocml_b200 import Engine
    kw.setdefault("max_tokens", 1024)
    return Engine.from_folder(folder, dtype=dtype, **kw)


def assert_rows(got, want, dtype, what):
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} against {tuple(want.shape)}"
    assert bool(torch.isfinite(got).all()), what
    err = ((got.double().cpu() - want.double()).abs() / want.double().abs().amax(dim=-1, keepdim=True).clamp_min(1e-30)).amax(-1)
    assert float(err.max()) < TOL[dtype], f"{what}: off by {float(err.max()):.3g}"
    if len(err) >= 20:
        assert float(err.quantile(0.9)) < MOST[dtype], f"{what}: a tenth of the rows are off by {float(err.quantile(0.9)):.3g} or more"
        assert float(err.median()) < MEDIAN[dtype], f"{what}: the median row is off by {float(err.median()):.3g}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts(model, dtype):
    """Lengths around the pages' and the memory's blocks' borders (64), the convolutions' taps and the windows, every place compared, the
    first tokens among them."""
    from rocml_b200 import StepEntry
    name, cfg, plain = model
    eng = engine(plain.folder, dtype)
    for n in (1, 2, 3, 5, 8, 33, 50, 51, 63, 64, 65, 91, 129, 131, 257, 310):
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
    ids = prompt(5, 140, cfg["vocab"])
    want = plain(ids)

    def differs(w=None, c=None):
        return rel_err(P.forward(c or plain.cfg, w or plain.w, ids), want) > 30 * MOST["float32"]
    for suffix, value in ((".norm1", 0.0), (".norm2", 0.0), ("final.norm", 0.0), (".mix.norm", 1.0), (".mix.q.norm", 1.0), (".mix.k.norm", 1.0),
                          ("left.q.norm", 1.0), ("left.k.norm", 1.0), ("left.out", 1.0), ("right.out", 1.0), (".lq1", 0.0), (".lq2", 0.0),
                          (".mix.i.b", 0.0), (".mix.f.b", 0.0), ("left.q.b", 0.0), ("left.k.b", 0.0), ("left.v.b", 0.0), ("left.o.b", 0.0),
                          ("left.g", 0.0), ("right.y.b", 0.0), ("right.x.b", 0.0), ("conv.b", 0.0), ("ra.b", 0.0), ("ri.b", 0.0), (".lam", 1.0)):
        w = {k: (torch.full_like(v, value) if k.endswith(suffix) else v) for k, v in plain.w.items()}
        # (what multiplies a memory's keys alike cancels against its divisor unless that is the maximum's bound)
        assert any(k.endswith(suffix) for k in w) and (differs(w) or (suffix == ".mix.i.b" and name == "KC")), suffix
    w = {k: (v.roll(1, 1) if k.endswith(".conv") and v.shape[1] > 1 else v) for k, v in plain.w.items()}
    assert differs(w), "conv"
    paths = [(("embedding", "scale"), 0.5 * cfg["embedding"]["scale"])]
    for i, L in enumerate(cfg["layers"]):
        m = L["mixer"]
        if L["type"] == "attention":
            if m.get("mask"):
                if m["mask"]["size"] < len(ids):
                    paths.append((("layers", i, "mixer", "mask", "size"), m["mask"]["size"] + 1))
            if m.get("mask", {"size": 0})["size"] != 1:                 # (a window of one token leaves the scores no say)
                paths.append((("layers", i, "mixer", "scale"), 0.5 * m["scale"]))
                if m.get("softcap"):
                    paths.append((("layers", i, "mixer", "softcap"), 0.5 * m["softcap"]))
                if m["rot"].get("scaling"):
                    paths.append((("layers", i, "mixer", "rot", "scaling", "factor"), 1.0))
            paths.append((("layers", i, "mixer", "diff"), m["diff"] + 0.2))
        elif L["type"] == "mlstm":
            paths.append((("layers", i, "mixer", "gate_cap"), 0.4 * m["gate_cap"]))
        else:
            paths.append((("layers", i, "mixer", "left", "scale"), 0.3 * m["left"]["scale"]))
            paths.append((("layers", i, "mixer", "left", "rot", "base"), 1.5 * m["left"]["rot"]["base"]))
    for path, value in paths:
        other = json.loads(json.dumps(plain.cfg))
        at = other
        for p in path[:-1]:
            at = at[p]
        at[path[-1]] = value
        assert differs(c=other) or path[-1] in ("gate_cap", "softcap") and name == "KC", path


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("graphs", [False, True])
def test_prompt_then_token_by_token(model, dtype, graphs):
    """The last tokens one by one (states, kept inputs and pages pass from the prompt's step to the single tokens), against the
    same positions of the whole prompt; every window passes over decoded tokens."""
    from rocml_b200 import StepEntry
    name, cfg, plain = model
    eng = engine(plain.folder, dtype, use_graphs=graphs)
    for n, tail in ((150, 80), (41, 40), (200, 3), (330, 150)):
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
def test_prompts_and_single_tokens_in_one_step(model, dtype):
    """A step that brings one token for one sequence, two for another and a whole prompt for a third."""
    from rocml_b200 import StepEntry
    name, cfg, plain = model
    eng = engine(plain.folder, dtype)
    a, b, c = prompt(31, 81, cfg["vocab"]), prompt(32, 130, cfg["vocab"]), prompt(33, 65, cfg["vocab"])
    sa, sb, sc = eng.new_sequence(), eng.new_sequence(), eng.new_sequence()
    eng.step([StepEntry(sa, a[:80], []), StepEntry(sb, b[:128], [])])
    got = eng.step([StepEntry(sa, a[80:], [0]), StepEntry(sc, c, [0, 64]), StepEntry(sb, b[128:], [0, 1])])
    want = torch.stack([plain(a)[80], plain(c)[0], plain(c)[64], plain(b)[128], plain(b)[129]])
    assert_rows(got, want, dtype, f"{name} {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_states_that_remember_hundreds_of_tokens(tmp_path, dtype):
    """Gates and decays close to one, no attention that could look back: the first three tokens still move the logits 500 tokens later
    (shown on the plain implementation), in a slot that another request used before; whole, and with the tail decoded."""
    from rocml_b200 import StepEntry
    cfg = json.loads(json.dumps(KEMIZEN["KB"]))
    cfg["layers"] = [cfg["layers"][i] for i in (0, 2, 4)]
    folder = write_kemizen(str(tmp_path / "m"), cfg, seed=3, slow=True)
    from safetensors.torch import load_file, save_file
    w = load_file(f"{folder}/model.safetensors")
    w["l1.mix.left.v"], w["l1.mix.left.v.b"] = w["l1.mix.left.v"] * 0, w["l1.mix.left.v.b"] * 0
    save_file({k: v.contiguous() for k, v in w.items()}, f"{folder}/model.safetensors")
    plain = Folder(folder)
    ids = prompt(21, 520, cfg["vocab"])
    want = plain(ids)
    other = plain([(t + 1) % cfg["vocab"] for t in ids[:3]] + ids[3:])
    assert rel_err(other[-1:], want[-1:]) > 10 * MOST["float32"]
    eng = engine(folder, dtype)
    slot = eng.new_sequence()
    eng.step([StepEntry(slot, prompt(22, 301, cfg["vocab"]), [])])
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
        assert len(out.tokens) == 12
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
@pytest.mark.parametrize("far", [1, 129, 130])
@pytest.mark.parametrize("reader", [False, True])
def test_a_key_at_the_windows_edge(tmp_path, dtype, far, reader):
    """One attention layer (or one that reads its keys under a wider window than its own) whose weights are made so that one token looks for
    another: just inside the window of 130 the logits depend on it, just outside they do not; in prompts and decoding, across page borders."""
    from rocml_b200 import StepEntry
    from tiny_models import _kdiff, _krot
    rot = _krot(1e7, 16)
    layers = [_kdiff(4, 2, 64, 128, 1.0, 0.4, rot, None, size=130, softcap=30.0)]
    if reader:
        layers = [_kdiff(4, 2, 64, 128, 1.0, 0.4, rot, None, size=5, softcap=30.0),
                  _kdiff(4, 2, 64, 128, 1.0, 0.4, rot, None, size=130, softcap=30.0, kv_from=0)]
    cfg = {"architecture": "Kemizen", "vocab": 120, "width": 96, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6}, "layers": layers}
    folder = write_kemizen(str(tmp_path / "m"), cfg, seed=5)
    from safetensors.torch import load_file, save_file
    w = load_file(f"{folder}/model.safetensors")
    # the query of token 77 is the key of token 78, every other token's query its own key
    e77, e78 = w["embed"][77].float(), w["embed"][78].float()
    wk = w["l0.mix.k"].float().reshape(2, 2, 64, 96)[torch.arange(4) // 2].reshape(512, 96)
    last = f"l{len(layers) - 1}.mix.q"
    w[last] = (wk + torch.outer(wk @ (e78 - e77), e77 / (e77 @ e77))).to(torch.bfloat16)
    w[f"{last}.norm"] = w["l0.mix.k.norm"].clone()
    if reader:                     # the layer before leaves the stream as it is, so that the reader's queries see the embedding
        w["l0.norm1"] = torch.full_like(w["l0.norm1"], -1.0)
    save_file({k: v.contiguous() for k, v in w.items()}, f"{folder}/model.safetensors")
    plain = Folder(folder)
    n = 331
    ids = [t % 40 for t in prompt(3, n, cfg["vocab"])]
    for at in (180, n - 1):
        ids[at], ids[at - far] = 77, 78
    want = plain(ids)
    moved = list(ids)
    moved[n - 1 - far] = 5
    change = rel_err(plain(moved)[-1:], want[-1:])
    assert change > 0.1 if far < 130 else change < 1e-9
    places = [179, 180, 181, n - 1]
    eng = engine(folder, dtype)
    slot = eng.new_sequence()
    got = eng.step([StepEntry(slot, ids, places)])
    eng.release(slot)
    assert_rows(got, want[places], dtype, f"{dtype} whole")
    for head in (100, 315):
        slot = eng.new_sequence()
        eng.step([StepEntry(slot, ids[:head], [])])
        got = []
        if head < 200:
            got = [eng.step([StepEntry(slot, ids[head:250], [80])]).clone()]
        for t in range(max(head, 250), n):
            got.append(eng.step([StepEntry(slot, [ids[t]], [0])]).clone())
        eng.release(slot)
        rows = torch.cat([want[180:181], want[250:]]) if head < 200 else want[head:]
        assert_rows(torch.cat(got), rows, dtype, f"{dtype} decoded from {head}")


def test_pages_outside_every_readers_window_come_back(tmp_path):
    """The cache keeps what the reader with the widest window can see, and gives the rest back."""
    from rocml_b200 import StepEntry
    eng = engine(write_kemizen(str(tmp_path / "m"), KEMIZEN["KA"], seed=1), "bfloat16")
    group = [g for g in eng.cache.kv_groups if g.window is not None]
    assert len(group) == 1 and group[0].window == 90 and group[0].n_entries == 1
    slot = eng.new_sequence()
    eng.step([StepEntry(slot, prompt(1, 400, 211), [])])
    assert len(group[0].held_pages()) == 7 - (400 - 89) // 64
    for t in range(60):
        eng.step([StepEntry(slot, [t], [0])])
    assert len(group[0].held_pages()) == 8 - (460 - 89) // 64
    eng.release(slot)
    eng.cache.check_invariants()


# ---- configurations drawn at random -----------------------------------------------------------------------------

def random_configuration(seed):
    from tiny_models import _kdiff, _kmem, _kpar, _krot
    g = torch.Generator().manual_seed(9000 + seed)

    def pick(*xs):
        return xs[int(torch.randint(0, len(xs), (1,), generator=g))]

    def rot(dim):
        dims = min(dim, 2 * pick(1, 2, 4, 8, 16, 32))
        return _krot(pick(100.0, 10000.0, 1e6), dims - dims % 2, pick(None, (4.0, 128, 16.0, 1.0), (2.0, 2048, 32.0, 2.0)))
    layers, sources = [], {}
    for i in range(pick(2, 3, 4, 5)):
        kind, ff = pick("mlstm", "attention", "attention", "parallel"), pick(None, 24, 64, 130)
        if kind == "mlstm":
            layers.append(_kmem(pick(1, 2, 3), pick(8, 20, 64, 128), pick(4, 32, 50, 64), pick(1.0, 8.0, 15.0, 40.0), ff))
        elif kind == "parallel":
            kv, blocks = pick(1, 2, 3), pick(1, 2, 4)
            dim = pick(8, 12, 32, 64, 128)
            layers.append(_kpar(kv * pick(1, 2, 4), kv, dim, pick(8, 20, 64, 128), pick(0.1, 0.3), pick(1, 2, 3, 4, 6), rot(dim) | {"scaling": None},
                                blocks * pick(5, 16, 40, 64), blocks, pick(1, 2, 4, 5), ff))
            layers[-1]["mixer"]["left"]["rot"].pop("scaling")
        else:
            size, cap, diff, scale = pick(None, 1, 17, 64, 100, 400), pick(None, 2.0, 30.0), pick(0.1, 0.5, 0.8), pick(0.1, 0.4, 1.0)
            src = pick(None, *sources) if sources else None
            if src is None:
                kv, dim = pick(1, 2), pick(6, 16, 32, 64, 96)
                own = (kv * pick(1, 2, 4), kv, dim, pick(10, 32, 64, 128), rot(dim))
                sources[i] = own
            else:
                own = sources[src]
            layers.append(_kdiff(*own[:4], scale, diff, own[4], ff, size=size, softcap=cap, kv_from=src))
    return {"architecture": "Kemizen", "vocab": pick(50, 101, 256), "width": pick(48, 64, 96, 136), "embedding": {"scale": pick(0.7, 1.0, 4.0)},
            "norm": {"eps": pick(1e-6, 1e-5)}, "layers": layers}


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(tmp_path, seed):
    """A configuration drawn at random: a whole prompt, the same in pieces of 50 with a tail decoded under graphs, and two
    requests side by side, in 32-bit (sharp) and bfloat16."""
    from rocml_b200 import StepEntry
    cfg = random_configuration(seed)
    folder = str(tmp_path / "m")
    write_kemizen(folder, cfg, seed)
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
