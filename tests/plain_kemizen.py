"""A plain, slow implementation of the Kemizen decoder, for tests only.

Whole sequences, no cache, one function per mechanism, torch on the CPU in float32 or float64; it shares
no code with ``rocml_b200`` (the model folder is read with the ``safetensors`` package).  Notation: W is
stored [out, in] and applied as W x;  rms(x) = x / sqrt(mean(x^2) + eps).

    embedding       x = s_e E[id]
    layer           x += rms(mix(x)) (1 + w1);   x += rms(ff(x)) (1 + w2)
    mLSTM           q = Wq h / sqrt(dim), k = Wk h, v = Wv h;  a = cap tanh((Wi h + bi) / cap),
                    f = ln sigmoid(cap tanh((Wf h + bf) / cap)), both one a head;  m' = max(f + m, a);
                    S <- e^(f + m - m') S + e^(a - m') k v^T,  n <- the same with k alone;  m <- m'
                    o = S^T q / (max(|n . q|, e^(-m)) + 1e-6);   out = Wo (rms_head(o) * w * sigmoid(Wg h))
    attention       two maps of q and k a head over one v: q, k <- rms(.) w per head and map, then rotated (rotate half,
                    frequencies blended along a ramp, cosines and sines times 0.1 ln(factor) + 1);
                    s = cap tanh((q . k) scale / cap) over 0 <= i - j < size;  o = softmax(s1) v - lambda softmax(s2) v,
                    lambda = e^(lq1 . lk1) - e^(lq2 . lk2) + diff;  out = Wo (rms(o) (1 - diff)), rms per head
                    (a layer may use an earlier layer's keys and values with its own queries)
    side by side    (rms(left(h)) w_l + rms(right(h)) w_r) / 2
       left         attention: q, k, v = conv(W. h + b);  q, k <- rms(.) w over the whole projection;  rotated; causal softmax;
                    out = Wo (heads * sigmoid(Wg h)) + bo
       right        y = gelu_tanh(Wy h + by),  u = conv(Wx h + bx) + bc;  r = sigmoid(Ra u + ba), i = sigmoid(Ri u + bi), block
                    by block;  ln a = -8 r softplus(lam);  S <- a S + sqrt(1 - a^2) i u;  out = Wo (S * y)
    dense ff        Wdown gelu(Wup h), gelu with erf
    output          logits = Whead (rms(x) (1 + w_f))
"""
from __future__ import annotations

import json
import math
import os

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def log_sigmoid(z):
    return -softplus(-z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def capped(z, cap):
    return z if cap is None else cap * torch.tanh(z / cap)


def causal_conv(u, w, before=None):
    """u [T, C]; w [C, taps], the last column multiplies the current token; zeros (or ``before`` [taps - 1, C]) ahead."""
    taps = w.shape[1]
    first = torch.zeros((taps - 1, u.shape[1]), dtype=u.dtype) if before is None else before.to(u.dtype)
    padded = torch.cat([first, u], dim=0)
    return sum(padded[j: j + u.shape[0]] * w[:, j] for j in range(taps))


def frequencies(rot):
    """(the angles' factors [dims / 2], the factor on cosines and sines), in double precision."""
    n, base = rot["dims"], rot["base"]
    f = torch.tensor([base ** (-2.0 * i / n) for i in range(n // 2)], dtype=torch.float64)
    sc = rot.get("scaling")
    if sc is None:
        return f, 1.0

    def d(t):
        return n * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(d(sc["fast"])), 0), min(math.ceil(d(sc["slow"])), n - 1)
    ramp = torch.tensor([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(n // 2)], dtype=torch.float64)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, heads, dim]: entries i and i + dims / 2 of the first dims turn."""
    f, mag = frequencies(rot)
    a = torch.as_tensor(positions, dtype=torch.float64)[:, None] * f[None]
    c, s = (torch.cos(a) * mag).to(x.dtype)[:, None], (torch.sin(a) * mag).to(x.dtype)[:, None]
    h = rot["dims"] // 2
    u, v = x[..., :h], x[..., h: 2 * h]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * h:]], dim=-1)


def weights(scores, positions, size):
    """scores [H, T, T] -> softmax over the keys that each query sees."""
    p = torch.as_tensor(positions)
    back = p[:, None] - p[None, :]
    seen = (back >= 0) & (back < size) if size else back >= 0
    return torch.softmax(scores.masked_fill(~seen[None], float("-inf")), dim=-1)


def mlstm_scan(q, k, v, i, f, state=None, below=None):
    """q, k [T, H, dim] (q already scaled), v [T, H, vdim], i and f [T, H] log gates: (o [T, H, vdim], (S, n, m)).  ``below``: a list that
    receives every token's divisors [H]."""
    T, H, dim = q.shape
    if state is None:
        state = (torch.zeros((H, dim, v.shape[2]), dtype=q.dtype), torch.zeros((H, dim), dtype=q.dtype), torch.zeros(H, dtype=q.dtype))
    S, n, m = (x.clone() for x in state)
    o = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for t in range(T):
        m2 = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - m2), torch.exp(i[t] - m2)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m2
        d = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[t] = torch.einsum("hkv,hk->hv", S, q[t]) / d[:, None]
        if below is not None:
            below.append(d)
    return o, (S, n, m)


def mlstm(h, m, w, eps):
    T = h.shape[0]
    H, dim, vd, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w["q"].T).reshape(T, H, dim) * dim ** -0.5
    k = (h @ w["k"].T).reshape(T, H, dim)
    v = (h @ w["v"].T).reshape(T, H, vd)
    i = capped(h @ w["i"].T + w["i.b"], cap)
    f = log_sigmoid(capped(h @ w["f"].T + w["f.b"], cap))
    o, _ = mlstm_scan(q, k, v, i, f)
    return (rms(o, eps).reshape(T, H * vd) * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def diff_lambda(w, diff):
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def diff_keys(h, positions, m, w, eps):
    """(keys [T, G, 2, dim] after norm and rotation, values [T, G, vdim]) of a layer with projections of its own."""
    T, G, dim = h.shape[0], m["kv_heads"], m["dim"]
    k = rms((h @ w["k"].T).reshape(T, G * 2, dim), eps) * w["k.norm"]
    return rotate(k, positions, m["rot"]).reshape(T, G, 2, dim), (h @ w["v"].T).reshape(T, G, m["vdim"])


def diff_attention(h, positions, m, w, eps, kv):
    T = h.shape[0]
    H, G, dim = m["heads"], m["kv_heads"], m["dim"]
    q = rms((h @ w["q"].T).reshape(T, H * 2, dim), eps) * w["q.norm"]
    q = rotate(q, positions, m["rot"]).reshape(T, H, 2, dim)
    of = torch.arange(H) // (H // G)
    keys, v = kv[0][:, of], kv[1][:, of]
    a = []
    for p in range(2):
        s = capped(torch.einsum("ihd,jhd->hij", q[:, :, p], keys[:, :, p]) * m["scale"], m.get("softcap"))
        a.append(torch.einsum("hij,jhd->ihd", weights(s, positions, m["mask"]["size"] if m.get("mask") else None), v))
    o = a[0] - diff_lambda(w, m["diff"]) * a[1]
    return (rms(o, eps) * (1.0 - m["diff"])).reshape(T, -1) @ w["o"].T


def conv_attention(h, positions, m, w, eps):
    T = h.shape[0]
    H, G, dim, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ w[n].T + w[n + ".b"], w[n + ".conv"]) for n in "qkv")
    q = rotate((rms(q, eps) * w["q.norm"]).reshape(T, H, dim), positions, m["rot"])
    k = rotate((rms(k, eps) * w["k.norm"]).reshape(T, G, dim), positions, m["rot"])
    of = torch.arange(H) // (H // G)
    a = weights(torch.einsum("ihd,jhd->hij", q, k[:, of]) * m["scale"], positions, None)
    o = torch.einsum("hij,jhd->ihd", a, v.reshape(T, G, vd)[:, of]).reshape(T, H * vd)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T + w["o.b"]


def rglru_gates(u, w):
    """(decay a, gated input sqrt(1 - a^2) i u) of every token and channel."""
    T, width = u.shape
    n = w["ra"].shape[0]
    parts = u.reshape(T, n, width // n)
    r = torch.sigmoid(torch.einsum("tbi,boi->tbo", parts, w["ra"]) + w["ra.b"]).reshape(T, width)
    i = torch.sigmoid(torch.einsum("tbi,boi->tbo", parts, w["ri"]) + w["ri.b"]).reshape(T, width)
    log_a = -8.0 * r * softplus(w["lam"])
    return torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u


def rglru_scan(a, x, state=None):
    S = torch.zeros(a.shape[1], dtype=a.dtype) if state is None else state.clone()
    out = torch.zeros_like(a)
    for t in range(a.shape[0]):
        S = a[t] * S + x[t]
        out[t] = S
    return out, S


def griffin(h, m, w):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"]) + w["conv.b"]
    s, _ = rglru_scan(*rglru_gates(u, w))
    return (s * y) @ w["o"].T


def side_by_side(h, positions, m, w, eps):
    left = conv_attention(h, positions, m["left"], sub(w, "left."), eps)
    right = griffin(h, m["right"], sub(w, "right."))
    return (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"]) / 2.0


def dense_ff(h, w):
    return gelu_erf(h @ w["up"].T) @ w["down"].T


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def layer(x, positions, cfg, i, tensors, cached):
    """One layer on a whole sequence x [T, D]; ``cached``: layer -> its keys and values."""
    L = cfg["layers"][i]
    eps, m, p = cfg["norm"]["eps"], L["mixer"], f"l{i}."
    w = sub(tensors, p + "mix.")
    if L["type"] == "mlstm":
        y = mlstm(x, m, w, eps)
    elif L["type"] == "attention":
        if m.get("kv_from") is None:
            cached[i] = diff_keys(x, positions, m, w, eps)
        y = diff_attention(x, positions, m, w, eps, cached[i if m.get("kv_from") is None else m["kv_from"]])
    elif L["type"] == "parallel":
        y = side_by_side(x, positions, m, w, eps)
    else:
        raise ValueError(L["type"])
    x = x + rms(y, eps) * (1.0 + tensors[p + "norm1"])
    if L.get("mlp") is not None:
        x = x + rms(dense_ff(x, sub(tensors, p + "mlp.")), eps) * (1.0 + tensors[p + "norm2"])
    return x


def forward(cfg, tensors, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence; ``layers_out``: a list that receives the stream after every layer."""
    x = tensors["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    positions, cached = list(range(len(tokens))), {}
    for i in range(len(cfg["layers"])):
        x = layer(x, positions, cfg, i, tensors, cached)
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, cfg["norm"]["eps"]) * (1.0 + tensors["final.norm"])) @ tensors["head"].T


def load_folder(folder, dtype=torch.float64):
    from safetensors import safe_open
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    tensors = {}
    with safe_open(os.path.join(folder, "model.safetensors"), "pt") as f:
        for k in f.keys():
            t = f.get_tensor(k)
            tensors[k] = t.to(dtype) if t.is_floating_point() else t
    return cfg, tensors
