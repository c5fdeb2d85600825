"""Fukatar restated plainly: one slow function per mechanism, float64 throughout, straight from the equations. Shares no
code with the package; the tests compare the package with this.

Notation: T tokens of one sequence at positions 0 .. T - 1 (or pos0 .. pos0 + T - 1 where a function takes ``pos0``);
W width; H heads, G key/value heads, D key size, V value size; weights are [out, in] and act as x @ W.T. ``p`` is a dict of
a part's tensors by their names under the part's prefix, ``m`` the part's entry of the config.
"""
import json
import math
import os

import torch

F = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def squared_relu(z):
    return torch.clamp(z, min=0.0) ** 2


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def embed(tokens, p, cfg):
    """Scaled token rows plus, for every token, a row of the table of token pairs: (previous * mul_prev + this * mul_cur)
    mod buckets, and the table's last row for the first token."""
    e = cfg.get("embedding") or {}
    x = p["embed"][torch.tensor(tokens)] * e.get("scale", 1.0)
    b = e.get("bigram")
    if b:
        rows = [b["buckets"] if i == 0 else (tokens[i - 1] * b["mul_prev"] + tokens[i] * b["mul_cur"]) % b["buckets"]
                for i in range(len(tokens))]
        x = x + p["bigram"][torch.tensor(rows)]
    return x


def token_shift(x, share, before=None):
    """x_t + (x_(t-1) - x_t) * share, element by element; ``before``: the vector ahead of the first (zeros at a start)."""
    prev = torch.cat([(torch.zeros_like(x[:1]) if before is None else before[None]), x[:-1]], 0)
    return x + (prev - x) * share


def frequencies(dims, base, scaling=None):
    """(angle per position of each pair, factor on sine and cosine), YaRN's interpolation where ``scaling`` asks for it."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def at(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(at(scaling["fast"])), 0), min(math.ceil(at(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def turn(x, pos, dims, freq, mag=1.0, pairs=False, back=False):
    """x [T, heads, D]: rotation of the first ``dims`` coordinates, coordinate i with i + dims/2, or 2i with 2i + 1 (``pairs``)."""
    a = pos.to(F)[:, None] * torch.tensor(freq, dtype=F)[None, :]
    c, s = (torch.cos(a) * mag)[:, None, :], (torch.sin(a) * mag)[:, None, :]
    if back:
        s = -s
    y = x.clone()
    if pairs:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        y[..., 0:dims:2], y[..., 1:dims:2] = u * c - v * s, v * c + u * s
    else:
        u, v = x[..., :dims // 2], x[..., dims // 2:dims]
        y[..., :dims // 2], y[..., dims // 2:dims] = u * c - v * s, v * c + u * s
    return y


def softmax_causal(s, sink=None):
    """Rows of scores [T, T] over the keys up to the diagonal; ``sink``: one more term of the denominator."""
    T = s.shape[0]
    s = torch.where(torch.arange(T)[None, :] <= torch.arange(T)[:, None], s, torch.full_like(s, -math.inf))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - top)
    return e / den


def attention_core(q, k, v, scale, cap=None, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        s = soft_cap((q[:, h] @ k[:, g].T) * scale, cap)
        out[:, h] = softmax_causal(s, None if sink is None else sink[h]) @ v[:, g]
    return out


def turned_value_attention(h, p, m, eps):
    """Grouped-query attention: q and k normed as whole projections before their rotation, values turned by their position
    before the sum and the sum turned back by the query's, a gate per head."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = (rms(h @ p["q"].T, eps) * p["q.norm"]).reshape(T, H, D)
    k = (rms(h @ p["k"].T, eps) * p["k.norm"]).reshape(T, G, D)
    v = (h @ p["v"].T).reshape(T, G, V)
    rot = m["rot"]
    f, mag = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    q, k = turn(q, pos, rot["dims"], f, mag), turn(k, pos, rot["dims"], f, mag)
    fv, _ = frequencies(V, rot["base"])
    o = attention_core(q, k, turn(v, pos, V, fv), m["scale"], m.get("softcap"))
    o = turn(o, pos, V, fv, back=True) * torch.sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(T, H * V) @ p["o"].T


def latent_sink_attention(h, p, m, eps):
    """Attention through one normed latent per token, without positions, with a sink per head."""
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    c = rms(h @ p["dkv"].T, eps) * p["dkv.norm"]
    q = (h @ p["q"].T).reshape(T, H, D)
    k = (c @ p["uk"].T).reshape(T, H, D)
    v = (c @ p["uv"].T).reshape(T, H, V)
    return attention_core(q, k, v, m["scale"], sink=p["sink"]).reshape(T, H * V) @ p["o"].T


def pairs_attention(h, p, m, eps):
    """Grouped-query attention, q and k rotated by neighbouring pairs and then divided by their root mean square."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q, k = (h @ p["q"].T).reshape(T, H, D), (h @ p["k"].T).reshape(T, G, D)
    v = (h @ p["v"].T).reshape(T, G, V)
    rot = m["rot"]
    f, mag = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    q, k = rms(turn(q, pos, rot["dims"], f, mag, pairs=True), eps), rms(turn(k, pos, rot["dims"], f, mag, pairs=True), eps)
    return attention_core(q, k, v, m["scale"], m.get("softcap")).reshape(T, H * V) @ p["o"].T


def conv_silu(u, w, before=None):
    """u [T, C], w [C, taps] (last column: the current token's); ``before``: the taps - 1 inputs ahead of them."""
    T, C = u.shape
    taps = w.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, C, dtype=F) if before is None else before, u], 0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + pad[j:j + T] * w[:, j]
    return silu(y), pad[T:]


def delta_rule(q, k, v, g, beta, S):
    """q, k [T, H, D], v [T, H, V], g, beta [T, H], S [H, D, V]: per token S <- g S, u = beta (v - S^T k), S <- S + k u^T,
    o = S^T q. -> (o [T, H, V], S)"""
    out = torch.zeros(*v.shape, dtype=F)
    for t in range(q.shape[0]):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def gated_delta(h, p, m, eps, state=None):
    """Short convolutions, unit keys and queries, one decay and one step size per head, the delta rule, a normed and gated
    output. -> (output, (S, the convolutions' memories))"""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    S, mem = (torch.zeros(H, D, V, dtype=F), {}) if state is None else state
    y, mem2 = {}, {}
    for n in ("q", "k", "v"):
        y[n], mem2[n] = conv_silu(h @ p[n].T, p[n + ".conv"], mem.get(n))
    grp = torch.arange(H) // (H // G)
    q = (unit(y["q"].reshape(T, G, D)) * D ** -0.5)[:, grp]
    k = unit(y["k"].reshape(T, G, D))[:, grp]
    beta = torch.sigmoid(h @ p["b"].T)
    g = torch.exp(-torch.exp(p["A_log"]) * softplus(h @ p["a"].T + p["dt_bias"]))
    o, S = delta_rule(q, k, y["v"].reshape(T, H, V), g, beta, S)
    o = rms(o, eps) * p["norm"] * silu(h @ p["g"].T).reshape(T, H, V)
    return o.reshape(T, H * V) @ p["o"].T, (S, mem2)


def sub(p, prefix):
    return {k[len(prefix):]: v for k, v in p.items() if k.startswith(prefix)}


def side_by_side(left, right, p, eps):
    """Half the sum of the two outputs, each over its root mean square first, times its weight."""
    return 0.5 * (rms(left, eps) * p["left.out"] + rms(right, eps) * p["right.out"])


def mixer(kind, a, p, m, eps):
    if kind == "attention":
        return turned_value_attention(a, p, m, eps)
    if kind == "latent_attention":
        return latent_sink_attention(a, p, m, eps)
    if kind == "parallel":
        left = pairs_attention(a, sub(p, "left."), m["left"], eps)
        right, _ = gated_delta(a, sub(p, "right."), m["right"], eps)
        return side_by_side(left, right, p, eps)
    raise ValueError(kind)


def read_model(folder):
    """(config.json as a dict, tensors by name) of a model folder."""
    from safetensors.torch import load_file

    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, load_file(os.path.join(folder, "model.safetensors"))


def forward(tokens, tensors, cfg, taps=None):
    """Logits [T, vocab] of one whole sequence. ``taps``: a list that receives the stream after every layer."""
    p = {k: v.to(F) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = embed(list(tokens), p, cfg)
    for i, lc in enumerate(cfg["layers"]):
        lp = sub(p, f"l{i}.")
        x = x + layer_norm(mixer(lc["type"], token_shift(x, lp["shift"]), sub(lp, "mix."), lc["mixer"], eps), lp["norm1"], eps)
        if lc.get("mlp"):
            x = x + layer_norm(squared_relu(x @ lp["mlp.up"].T) @ lp["mlp.down"].T, lp["norm2"], eps)
        if taps is not None:
            taps.append(x.clone())
    logits = layer_norm(x, p["final.norm"], eps) @ p["head"].T
    return soft_cap(logits, cfg.get("logit_softcap"))
