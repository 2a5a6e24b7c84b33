"""A plain, slow implementation of the Ravelorn decoder, for tests only.

Whole sequences, no cache, one function per mechanism, torch on the CPU in float32 or float64; it shares
no code with ``rocml_b200`` (the model folder is read with the ``safetensors`` package).  Notation: W is
stored [out, in] and applied as W x;  rms(x) = x / sqrt(mean(x^2) + eps);  unit(x) = x / sqrt(sum(x^2) + 1e-6);
ln(x) = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b.

    embedding       x_p = E[id_p] + P[p]
    layer           x += m * ln1(mix(x));   x += m * ln2(ff(x))
    delta rule      q, k, v <- silu(conv(W. h));  q <- unit(q) / sqrt(dim), k <- unit(k);  b = sigmoid(Wb h)
                    per head   g = exp(-exp(A) softplus(Wa h + c));      per channel   the same with Wa2 (Wa1 h), one a key channel
                    S <- g S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q
                    out = Wo (rms_head(o) * w * silu(Wg h))   or   ... * sigmoid(Wg2 (Wg1 h))
    attention       q, k <- rms per head;  q <- q (1 + coef ln(floor((p + 1) / every) + 1));  s = (q . k) scale
                    a_ij = e^s_ij / (e^sink + sum_j e^s_ij)
    side by side    left_scale * attention(h) + right_scale * delta(h)
    experts         s = softmax(Wr h);  the `top` largest of s + correction, weights s;  an expert is
                    Wdown (silu(Wgate h) * Wup h), one of the last `identity` places is h itself
    output          logits = cap * tanh(Whead ln_f(x) / cap)
"""
from __future__ import annotations

import json
import math
import os

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def layer_norm(x, w, b, eps):
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * w + b


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def causal_conv(u, taps_w, before=None):
    """u [T, C]; taps_w [C, taps], the last column multiplies the current token; zeros (or ``before``
    [taps - 1, C]) ahead of the first token."""
    taps = taps_w.shape[1]
    first = torch.zeros((taps - 1, u.shape[1]), dtype=u.dtype) if before is None else before.to(u.dtype)
    padded = torch.cat([first, u], dim=0)
    out = torch.zeros_like(u)
    for j in range(taps):
        out = out + padded[j: j + u.shape[0]] * taps_w[:, j]
    return out


def delta_rule(q, k, v, beta, g, state=None):
    """q, k [T, H, dim] (already one per head), v [T, H, vdim], beta [T, H], g [T, H] or [T, H, dim]: (o [T, H, vdim],
    the state [H, dim, vdim] after the last token)."""
    T, H, dim = q.shape
    if g.dim() == 2:
        g = g[:, :, None].expand(T, H, dim)
    S = torch.zeros((H, dim, v.shape[2]), dtype=q.dtype) if state is None else state.clone()
    o = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o, S


def decay(z, a_log, dt_bias):
    """z [T, H] or [T, H, dim], a_log [H], dt_bias of z's trailing shape."""
    rate = torch.exp(a_log)
    if z.dim() == 3:
        rate = rate[:, None]
    return torch.exp(-rate * softplus(z + dt_bias))


def delta_inputs(h, m, w, conv_before=None):
    """The recurrence's inputs: (q, k, v, beta) with q and k repeated for the heads that share them."""
    T = h.shape[0]
    H, G, dim, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    before = conv_before or {}

    def conv(n):
        return silu(causal_conv(h @ w[n].T, w[n + ".conv"], before.get(n)))
    of = torch.arange(H) // (H // G)
    q = unit(conv("q").reshape(T, G, dim)) * dim ** -0.5
    k = unit(conv("k").reshape(T, G, dim))
    v = conv("v").reshape(T, H, vd)
    return q[:, of], k[:, of], v, torch.sigmoid(h @ w["b"].T)


def delta_mixer(h, m, w, eps, per_channel):
    T = h.shape[0]
    H, dim, vd = m["heads"], m["dim"], m["vdim"]
    q, k, v, beta = delta_inputs(h, m, w)
    if per_channel:
        g = decay(((h @ w["a1"].T) @ w["a2"].T).reshape(T, H, dim), w["A_log"], w["dt_bias"].reshape(H, dim))
        gate = torch.sigmoid((h @ w["g1"].T) @ w["g2"].T)
    else:
        g = decay(h @ w["a"].T, w["A_log"], w["dt_bias"])
        gate = silu(h @ w["g"].T)
    o, _ = delta_rule(q, k, v, beta, g)
    o = rms(o, eps) * w["norm"] * gate.reshape(T, H, vd)
    return o.reshape(T, H * vd) @ w["o"].T


def query_temperature(positions, t):
    p = torch.as_tensor(positions, dtype=torch.float64)
    return 1.0 + t["coef"] * torch.log(torch.floor((p + 1.0) / t["every"]) + 1.0)


def sink_softmax(scores, positions, sink):
    """scores [H, T, T] -> causal weights whose denominator has the term e^sink_h too."""
    p = torch.as_tensor(positions)
    s = scores.masked_fill(~(p[None, :] <= p[:, None])[None], float("-inf"))
    top = torch.maximum(s.amax(dim=-1, keepdim=True), sink.reshape(-1, 1, 1))
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink.reshape(-1, 1, 1) - top))


def attention(h, positions, m, w, eps):
    T = h.shape[0]
    H, G, dim, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w["q"].T).reshape(T, H, dim), eps)
    k = rms((h @ w["k"].T).reshape(T, G, dim), eps)
    v = (h @ w["v"].T).reshape(T, G, vd)
    if m.get("q_temp") is not None:
        q = q * query_temperature(positions, m["q_temp"]).to(q.dtype)[:, None, None]
    of = torch.arange(H) // (H // G)
    a = sink_softmax(torch.einsum("ihd,jhd->hij", q, k[:, of]) * m["scale"], positions, w["sink"])
    return torch.einsum("hij,jhd->ihd", a, v[:, of]).reshape(T, H * vd) @ w["o"].T


def side_by_side(h, positions, m, w, eps):
    left = attention(h, positions, m["left"], sub(w, "left."), eps)
    right = delta_mixer(h, m["right"], sub(w, "right."), eps, per_channel=False)
    return m["left_scale"] * left + m["right_scale"] * right


def route(h, r, w):
    """(chosen [T, top], their weights, the smallest distance between a chosen and a passed-over choice score)."""
    s = torch.softmax(h @ w["router"].T, dim=-1)
    order = torch.sort(s + w["correction"], dim=-1, descending=True)
    ids = order.indices[:, : r["top"]]
    gap = order.values[:, r["top"] - 1] - order.values[:, r["top"]] if r["top"] < s.shape[1] else torch.ones(len(s), dtype=s.dtype)
    return ids, torch.gather(s, 1, ids), gap


def experts_ff(h, mlp, w, gaps=None):
    n = mlp["router"]["experts"]
    ids, weights, gap = route(h, mlp["router"], w)
    if gaps is not None:
        gaps.append(gap)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(ids[t].tolist(), weights[t]):
            y = h[t] if e >= n else w[f"e{e}.down"] @ (silu(w[f"e{e}.gate"] @ h[t]) * (w[f"e{e}.up"] @ h[t]))
            out[t] += wt * y
    return out


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def layer(x, positions, cfg, i, tensors, gaps=None):
    """One layer on a whole sequence x [T, D]."""
    L = cfg["layers"][i]
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    p = f"l{i}."
    w = sub(tensors, p + "mix.")
    if L["type"] == "channel_delta":
        y = delta_mixer(x, L["mixer"], w, eps, per_channel=True)
    elif L["type"] == "parallel":
        y = side_by_side(x, positions, L["mixer"], w, eps)
    else:
        raise ValueError(L["type"])
    x = x + m * layer_norm(y, tensors[p + "norm1"], tensors[p + "norm1.b"], eps)
    if L.get("mlp") is not None:
        y = experts_ff(x, L["mlp"], sub(tensors, p + "mlp."), gaps)
        x = x + m * layer_norm(y, tensors[p + "norm2"], tensors[p + "norm2.b"], eps)
    return x


def forward(cfg, tensors, tokens, layers_out=None, gaps=None):
    """Logits [T, vocab] of one whole sequence; ``layers_out``: a list that receives the stream after every layer;
    ``gaps``: one that receives every router's distances (see ``route``)."""
    x = tensors["embed"][torch.as_tensor(tokens)] + tensors["pos"][: len(tokens)]
    positions = list(range(len(tokens)))
    for i in range(len(cfg["layers"])):
        x = layer(x, positions, cfg, i, tensors, gaps)
        if layers_out is not None:
            layers_out.append(x)
    x = layer_norm(x, tensors["final.norm"], tensors["final.norm.b"], cfg["norm"]["eps"])
    z = x @ tensors["head"].T
    cap = cfg.get("logit_softcap")
    return z if cap is None else cap * torch.tanh(z / cap)


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
