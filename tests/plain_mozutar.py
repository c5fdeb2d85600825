"""Mozutar restated plainly: one slow function per mechanism, float64 throughout, straight from the equations. Shares no
code with the package; the tests compare the package with this.

Notation: T tokens of one sequence at positions 0 .. T - 1; W width; H heads, G key/value heads, D key size, V value size;
weights are [out, in] and act as x @ W.T. ``p`` is a dict of a part's tensors by their names under the part's prefix, ``m``
the part's entry of the config.
"""
import json
import math
import os

import torch

F = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def silu(z):
    return z * torch.sigmoid(z)


def log_sigmoid(z):
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def rotate_halves(x, pos, dims, base):
    """x [T, heads, D]: coordinate i turned with coordinate i + dims / 2 (i below dims / 2) by pos * base^(-2i/dims)."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)
    a = pos.to(F)[:, None] * f[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def softmax_causal(s):
    T = s.shape[0]
    s = torch.where(torch.arange(T)[None, :] <= torch.arange(T)[:, None], s, torch.full_like(s, -math.inf))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def attention_core(q, k, v, scale, cap):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_causal(soft_cap((q[:, h] @ k[:, g].T) * scale, cap)) @ v[:, g]
    return out


def keys_as_values_attention(h, p, m, eps):
    """Grouped-query attention without a value projection: the values are the keys as projected, the keys that score are
    normed per head and rotated."""
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(T)
    k_raw = (h @ p["k"].T).reshape(T, G, D)
    q = rms((h @ p["q"].T).reshape(T, H, D), eps) * p["q.norm"]
    k = rms(k_raw, eps) * p["k.norm"]
    rot = m["rot"]
    q, k = rotate_halves(q, pos, rot["dims"], rot["base"]), rotate_halves(k, pos, rot["dims"], rot["base"])
    return attention_core(q, k, k_raw, m["scale"], m.get("softcap")).reshape(T, H * D) @ p["o"].T


def channel_decays(h, p, tau):
    """One decay per key channel and token: sigmoid(W_a2 (W_a1 h) + b)^(1/tau)."""
    return torch.exp(log_sigmoid((h @ p["a1"].T) @ p["a2"].T + p["a2.b"]) / tau)


def decayed_sums(q, k, v, a, S):
    """S <- diag(a_t) S + k_t v_t^T, o_t = S^T q_t; q, k, a [T, H, D], v [T, H, V], S [H, D, V]. -> (o [T, H, V], S)"""
    out = torch.zeros(*v.shape, dtype=F)
    for t in range(q.shape[0]):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def gated_linear_attention(h, p, m, eps, S=None):
    """-> (output, state)"""
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ p["q"].T).reshape(T, H, D) * D ** -0.5
    k, v = (h @ p["k"].T).reshape(T, H, D), (h @ p["v"].T).reshape(T, H, V)
    o, S = decayed_sums(q, k, v, channel_decays(h, p, m["tau"]).reshape(T, H, D), torch.zeros(H, D, V, dtype=F) if S is None else S)
    o = rms(o, eps) * p["norm"]
    return (o.reshape(T, H * V) * silu(h @ p["g"].T)) @ p["o"].T, S


def exponential_gates(h, p, cap):
    """-> (log input gate, log forget gate), each [T, H]."""
    i = soft_cap(h @ p["i"].T + p["i.b"], cap)
    f = log_sigmoid(soft_cap(h @ p["f"].T + p["f.b"], cap))
    return i, f


def matrix_memory(q, k, v, i, f, state=None):
    """The matrix memory with exponential gates kept in range by a running maximum: q, k [T, H, D], v [T, H, V], i, f [T, H].
    -> (o [T, H, V], (S [H, D, V], n [H, D], m [H])). The maximum starts at zero, not at minus infinity, so what is taken off
    the exponents (and the 1e-6 beside it) is part of the function."""
    T, H, D = q.shape
    V = v.shape[2]
    S, n, m = state if state is not None else (torch.zeros(H, D, V, dtype=F), torch.zeros(H, D, dtype=F), torch.zeros(H, dtype=F))
    out = torch.zeros(T, H, V, dtype=F)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        m = m_new
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return out, (S, n, m)


def mlstm(h, p, m, eps, state=None):
    """-> (output, state)"""
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ p["q"].T).reshape(T, H, D) * D ** -0.5
    k, v = (h @ p["k"].T).reshape(T, H, D), (h @ p["v"].T).reshape(T, H, V)
    i, f = exponential_gates(h, p, m["gate_cap"])
    o, state = matrix_memory(q, k, v, i, f, state)
    o = rms(o, eps).reshape(T, H * V) * p["norm"]
    return (o * torch.sigmoid(h @ p["g"].T)) @ p["o"].T, state


def sub(p, prefix):
    return {k[len(prefix):]: v for k, v in p.items() if k.startswith(prefix)}


def side_by_side(left, right, p, eps):
    """Half the sum of the two outputs, each over its root mean square first, times its weight."""
    return 0.5 * (rms(left, eps) * p["left.out"] + rms(right, eps) * p["right.out"])


def mixer(kind, a, p, m, eps):
    if kind == "mlstm":
        return mlstm(a, p, m, eps)[0]
    if kind == "parallel":
        left = keys_as_values_attention(a, sub(p, "left."), m["left"], eps)
        right, _ = gated_linear_attention(a, sub(p, "right."), m["right"], eps)
        return side_by_side(left, right, p, eps)
    raise ValueError(kind)


def gated_ff(h, p):
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def route(h, p, r):
    """For every token the chosen outputs of the router, best first, and their weights: [(numbers, weights)]. Scores are a
    softmax over experts and identity experts; the choice goes by score + correction among the best groups (group score: its
    largest choice score), the weights are the scores as they are."""
    z = h @ p["router"].T
    s = torch.exp(z - z.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    n = r["experts"] + r.get("identity", 0)
    groups = r.get("groups") or {"count": 1, "keep": 1}
    per = n // groups["count"]
    out = []
    for t in range(h.shape[0]):
        c = [float(s[t, e] + p["correction"][e]) for e in range(n)]
        best = sorted(range(groups["count"]), key=lambda g: -max(c[g * per:(g + 1) * per]))[:groups["keep"]]
        allowed = [e for e in range(n) if e // per in best]
        chosen = sorted(allowed, key=lambda e: -c[e])[:r["top"]]
        out.append((chosen, [float(s[t, e]) for e in chosen]))
    return out


def mixture(h, p, r):
    """The chosen experts' outputs times their scores; router outputs behind the experts pass the input on."""
    y = torch.zeros_like(h)
    for t, (chosen, weights) in enumerate(route(h, p, r)):
        for e, w in zip(chosen, weights):
            y[t] += w * (gated_ff(h[t:t + 1], sub(p, f"e{e}."))[0] if e < r["experts"] else h[t])
    return y


def feed_forward(h, p, mlp):
    return gated_ff(h, p) if mlp["kind"] == "dense" else mixture(h, p, mlp["router"])


def read_model(folder):
    """(config.json as a dict, tensors by name) of a model folder."""
    from safetensors.torch import load_file

    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, load_file(os.path.join(folder, "model.safetensors"))


def runs(cfg):
    """[(layer, pass number if the layer opens a pass of the loop, else None)] in running order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def take_in(x, x0, w, step):
    """What opens a pass of the loop: W [x; x0] + the pass's vector."""
    return torch.cat([x, x0], -1) @ w.T + step


def layer(x, lc, p, eps):
    y = mixer(lc["type"], layer_norm(x, p["norm1"], p["norm1.b"], eps), sub(p, "mix."), lc["mixer"], eps)
    x = x + layer_norm(y, p["norm1b"], p["norm1b.b"], eps) * p["ls1"]
    if lc.get("mlp"):
        y = feed_forward(layer_norm(x, p["norm2"], p["norm2.b"], eps), sub(p, "mlp."), lc["mlp"])
        x = x + layer_norm(y, p["norm2b"], p["norm2b.b"], eps) * p["ls2"]
    return x


def forward(tokens, tensors, cfg, taps=None):
    """Logits [T, vocab] of one whole sequence. ``taps``: a list that receives the stream after every layer run."""
    p = {k: v.to(F) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x0 = p["embed"][torch.tensor(list(tokens))] * (cfg.get("embedding") or {}).get("scale", 1.0)
    x = x0
    for i, t in runs(cfg):
        if t is not None:
            x = take_in(x, x0, p["loop.in"], p["loop.step"][t])
        x = layer(x, cfg["layers"][i], sub(p, f"l{i}."), eps)
        if taps is not None:
            taps.append(x.clone())
    return layer_norm(x, p["final.norm"], p["final.norm.b"], eps) @ p["embed"].T
