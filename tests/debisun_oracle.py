"""Plain, slow Debisun: one function per mechanism, token loops, no cache, any float dtype.  It imports nothing of the
framework: the tests compare the product path against it.

Weights are a flat dict name -> tensor ("l<i>.mix.q", "embed", ...), the configuration is the parsed config.json."""
import math

import torch


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return torch.where(z > 0, z * z, torch.zeros_like(z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def short_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j) with zeros before the start."""
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def distance_bucket(n, B, far):
    """Exact up to B/2, then logarithmic up to the distance `far`; everything beyond shares the last row."""
    half = B // 2
    if n < half:
        return n
    return min(B - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (B - half)))


def visible(i, j, chunk):
    return j <= i and i // chunk == j // chunk


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def weights_with_silent_sink(s):
    """exp(s) over one plus the sum of the visible ones (last axis; -inf = not visible)."""
    m = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def attention(h, W, p, c):
    T, H, G, D, V = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = short_conv(h @ W[p + "q"].T, W[p + "q.conv"]).view(T, H, D)
    k = short_conv(h @ W[p + "k"].T, W[p + "k.conv"]).view(T, G, D)
    v = short_conv(h @ W[p + "v"].T, W[p + "v.conv"]).view(T, G, V)
    rel, chunk = W[p + "rel"], c["mask"]["size"]
    B = rel.shape[0]
    bucket = torch.tensor([distance_bucket(n, B, c["bias_max"]) for n in range(min(T, chunk))])
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for i in range(T):
        seen = [j for j in range(i + 1) if visible(i, j, chunk)]
        near = bucket[[i - j for j in seen]]
        for x in range(H):
            g = x // (H // G)
            s = soft_cap((k[seen, g] * q[i, x]).sum(-1) * c["scale"], c["softcap"]) + rel[near, x]
            out[i, x] = (weights_with_silent_sink(s).unsqueeze(-1) * v[seen, g]).sum(0)
    return out.reshape(T, H * V) @ W[p + "o"].T


def relu_mlp(h, W, p):
    return relu_squared(h @ W[p + "up"].T) @ W[p + "down"].T


def routed(h, W, p, r):
    """(weights, expert ids) [T, top]: chosen by softmax score + correction, weighted by the score alone."""
    s = torch.softmax(h @ W[p + "router"].T, -1)
    ids = torch.argsort(-(s + W[p + "correction"]), dim=-1, stable=True)[:, : r["top"]]
    w = torch.gather(s, 1, ids)
    return w / (w.sum(-1, keepdim=True) + 1e-20) * r["scale"], ids


def experts(h, W, p, mlp):
    r = mlp["router"]
    w, ids = routed(h, W, p, r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for a, e in zip(w[t], ids[t].tolist()):
            out[t] += a * (h[t] if e >= r["experts"] else relu_mlp(h[t], W, f"{p}e{e}."))
    if mlp.get("shared"):
        out = out + sigmoid(h @ W[p + "shared.sg"].T) * relu_mlp(h, W, p + "shared.")
    return out


def token_side(x, e, W, p, eps):
    """Update from the token's own row e [T, dim] of this layer, gated by the residual stream."""
    y = (gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T
    return unit_rms(y, eps) * W[p + "side.norm"]


def forward(cfg, W, tokens, taps=None):
    """Logits [T, vocab] of one whole sequence; `taps` (a list) gets the residual stream after every layer."""
    eps, n = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    tokens = torch.as_tensor(tokens)
    x = W["embed"][tokens]
    norm = lambda x, name: layer_norm(x, W[name], W[name + ".b"], eps)
    for i, lc in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + W[p + "ls1"] * attention(norm(x, p + "norm1"), W, p + "mix.", lc["mixer"])
        mlp = lc.get("mlp")
        if mlp:
            h = norm(x, p + "norm2")
            x = x + W[p + "ls2"] * (relu_mlp(h, W, p + "mlp.") if mlp["kind"] == "dense" else experts(h, W, p + "mlp.", mlp))
        x = x + token_side(x, W["side.embed"][tokens][:, i * n: (i + 1) * n], W, p, eps)
        if taps is not None:
            taps.append(x)
    return norm(x, "final.norm") @ W["head"].T
