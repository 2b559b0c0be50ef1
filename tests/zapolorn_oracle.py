"""Plain, slow Zapolorn: one function per mechanism, token loops, no cache, any float dtype.  It imports nothing of the
framework: the tests compare the product path against it.

Weights are a flat dict name -> tensor ("l<i>.mix.q", "embed", ...), the configuration is the parsed config.json."""
import math

import torch


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotate_pairs(x, rot):
    """x [T, heads, d] at positions 0 .. T-1: coordinates (2i, 2i+1) turn by p base^(-2i/dims) / factor; the rest stays."""
    y, n = x.clone(), rot["dims"]
    slow = (rot.get("scaling") or {}).get("factor", 1.0)
    for i in range(n // 2):
        a = torch.arange(x.shape[0], dtype=torch.float64) * rot["base"] ** (-2 * i / n) / slow
        c, s = torch.cos(a).to(x.dtype).unsqueeze(1), torch.sin(a).to(x.dtype).unsqueeze(1)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def temperature(p, t):
    """Factor of the query at position p: grows with the logarithm of the number of begun blocks of `every` tokens."""
    return 1 + t["coef"] * math.log(math.floor((p + 1) / t["every"]) + 1)


def slope(h, H):
    return 2.0 ** (-8 * (h + 1) / H)


def visible(i, j, window):
    return 0 <= i - j and (window is None or i - j < window)


def softmax_with(extra, s):
    """exp(s) over its sum (last axis) and exp(extra), a score without a value (None: nothing is added)."""
    m = s.max(-1, keepdim=True).values
    if extra is not None:
        m = torch.maximum(m, extra.unsqueeze(-1))
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + (0 if extra is None else torch.exp(extra.unsqueeze(-1) - m)))


def projected_keys(h, W, p, c, eps):
    """Keys [T, G, d] (normed, rotated) and values [T, G, v]: what a cache holds."""
    T, G = h.shape[0], c["kv_heads"]
    k = rms_norm((h @ W[p + "k"].T).view(T, G, c["dim"]), W[p + "k.norm"], eps)
    if c.get("rot"):
        k = rotate_pairs(k, c["rot"])
    return k, (h @ W[p + "v"].T).view(T, G, c["vdim"])


def attend(q, k, v, scale, window=None, sink=None, slopes=None):
    """q [T, H, d], k [T, G, d], v [T, G, V] -> [T, H, V]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        j0 = next(j for j in range(max(0, i - (window or i + 1)), i + 1) if visible(i, j, window))
        s = torch.einsum("hd,jhd->hj", q[i], k[j0: i + 1]) * scale
        if slopes is not None:
            s = s - slopes.unsqueeze(1) * (i - torch.arange(j0, i + 1, dtype=q.dtype))
        out[i] = torch.einsum("hj,jhv->hv", softmax_with(sink, s), v[j0: i + 1])
    return out


def attention(h, W, p, c, eps, kv=None):
    """(output, (keys, values)); `kv`: another layer's keys and values instead of own ones."""
    T, H = h.shape[0], c["heads"]
    q = rms_norm((h @ W[p + "q"].T).view(T, H, c["dim"]), W[p + "q.norm"], eps)
    if c.get("rot"):
        q = rotate_pairs(q, c["rot"])
    kv = kv if kv is not None else projected_keys(h, W, p, c, eps)
    o = attend(q, *kv, c["scale"], c["mask"]["size"] if c.get("mask") else None, W[p + "sink"])
    o = o * sigmoid(h @ W[p + "g"].T).unsqueeze(-1)
    return o.reshape(T, -1) @ W[p + "o"].T, kv


def sloped_attention(h, W, p, c, eps):
    T, H = h.shape[0], c["heads"]
    q = rms_norm((h @ W[p + "q"].T).view(T, H, c["dim"]), W[p + "q.norm"], eps)
    q = q * torch.tensor([temperature(i, c["q_temp"]) for i in range(T)], dtype=h.dtype).view(T, 1, 1)
    k, v = projected_keys(h, W, p, c, eps)
    o = attend(q, k, v, c["scale"], slopes=torch.tensor([slope(x, H) for x in range(H)], dtype=h.dtype))
    return o.reshape(T, -1) @ W[p + "o"].T


def channel_decays(h, W, p, c):
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    return (sigmoid(z) ** (1 / c["tau"])).view(h.shape[0], c["heads"], c["dim"])


def decayed_sums(q, k, v, alpha):
    """S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t per head; q, k, alpha [T, H, d], v [T, H, V]."""
    T, H, d = q.shape
    S, out = torch.zeros(H, d, v.shape[2], dtype=q.dtype), torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = alpha[t].unsqueeze(-1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out[t] = torch.einsum("hd,hdv->hv", q[t], S)
    return out


def gated_linear_attention(h, W, p, c, eps):
    T, H, d = h.shape[0], c["heads"], c["dim"]
    q = (h @ W[p + "q"].T).view(T, H, d) * d ** -0.5
    k, v = (h @ W[p + "k"].T).view(T, H, d), (h @ W[p + "v"].T).view(T, H, c["vdim"])
    o = rms_norm(decayed_sums(q, k, v, channel_decays(h, W, p, c)), W[p + "norm"], eps)
    return (o.reshape(T, -1) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def side_by_side(h, W, p, c, eps):
    return c["left_scale"] * sloped_attention(h, W, p + "left.", c["left"], eps) \
        + c["right_scale"] * gated_linear_attention(h, W, p + "right.", c["right"], eps)


def swiglu_mlp(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def routed(h, W, p, top):
    """(weights, expert ids) [T, top]: the largest sigmoid scores as they are."""
    s = sigmoid(h @ W[p + "router"].T)
    ids = torch.argsort(-s, dim=-1, stable=True)[:, :top]
    return torch.gather(s, 1, ids), ids


def experts(h, W, p, mlp):
    w, ids = routed(h, W, p, mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for a, e in zip(w[t], ids[t].tolist()):
            out[t] += swiglu_mlp(a * h[t], W, f"{p}e{e}.")
    return out + swiglu_mlp(h, W, p + "shared.") if mlp.get("shared") else out


def forward(cfg, W, tokens, taps=None):
    """Logits [T, vocab] of one whole sequence; `taps` (a list) gets the residual stream after every layer."""
    eps, kvs = cfg["norm"]["eps"], {}
    x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, lc in enumerate(cfg["layers"]):
        p, c = f"l{i}.", lc["mixer"]
        if lc["type"] == "parallel":
            y = side_by_side(x, W, p + "mix.", c, eps)
        else:
            y, kvs[i] = attention(x, W, p + "mix.", c, eps, kvs[c["kv_from"]] if c.get("kv_from") is not None else None)
        x = x + rms_norm(y, W[p + "norm1"], eps)
        mlp = lc.get("mlp")
        if mlp:
            y = swiglu_mlp(x, W, p + "mlp.") if mlp["kind"] == "dense" else experts(x, W, p + "mlp.", mlp)
            x = x + rms_norm(y, W[p + "norm2"], eps)
        if taps is not None:
            taps.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T * cfg["logit_scale"]
