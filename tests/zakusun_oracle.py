"""Plain, slow Zakusun: one function per mechanism, token loops, no cache, any float dtype.  It imports nothing of the
framework: the tests compare the product path against it.

Weights are a flat dict name -> tensor ("l<i>.mix.q", "embed", ...), the configuration is the parsed config.json."""
import functools
import math

import torch


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def grouped_rms_norm(x, w, eps, groups):
    """Every part of the vector over its own root mean square."""
    n = x.shape[-1] // groups
    parts = [x[..., g * n: (g + 1) * n] for g in range(groups)]
    return torch.cat([p / torch.sqrt((p * p).mean(-1, keepdim=True) + eps) for p in parts], -1) * w


@functools.lru_cache(maxsize=4096)
def position_vector(p, width):
    v = torch.zeros(width, dtype=torch.float64)
    for i in range((width + 1) // 2):
        a = p * 10000.0 ** (-2 * i / width)
        v[2 * i] = math.sin(a)
        if 2 * i + 1 < width:
            v[2 * i + 1] = math.cos(a)
    return v


def embedding(tokens, W):
    x = W["embed"][torch.as_tensor(tokens)]
    return x + torch.stack([position_vector(p, x.shape[1]) for p in range(x.shape[0])]).to(x.dtype)


def input_convolution(h, w):
    """h + conv(h): every channel's own taps over the last inputs, the last tap on the token itself; w [width, taps]."""
    T, taps = h.shape[0], w.shape[1]
    out = h.clone()
    for back in range(min(taps, T)):                             # the input of `back` tokens before
        out[back:] += w[:, taps - 1 - back] * h[: T - back]
    return out


def softmax_with(sink, s):
    """exp(s) over its sum (last axis) and exp(sink), a score without a value; s [H, n], sink [H]."""
    m = torch.maximum(s.max(-1).values, sink).unsqueeze(-1)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink.unsqueeze(-1) - m))


def latents(h, W, p, eps):
    """[T, rank]: what a cache holds."""
    return rms_norm(h @ W[p + "dkv"].T, W[p + "dkv.norm"], eps)


def attend(q, k, v, scale, sink):
    """q, k [T, H, d], v [T, H, V] -> [T, H, V]: every token over itself and all before it."""
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=q.dtype)
    for i in range(q.shape[0]):
        s = torch.einsum("hd,jhd->hj", q[i], k[: i + 1]) * scale
        out[i] = torch.einsum("hj,jhv->hv", softmax_with(sink, s), v[: i + 1])
    return out


def latent_attention(h, W, p, c, eps):
    T, H = h.shape[0], c["heads"]
    lat = latents(h, W, p, eps)
    q, k = (h @ W[p + "q"].T).view(T, H, c["dim"]), (lat @ W[p + "uk"].T).view(T, H, c["dim"])
    o = attend(q, k, (lat @ W[p + "uv"].T).view(T, H, c["vdim"]), c["scale"], W[p + "sink"])
    return (o.reshape(T, -1) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def expert(h, W, p, limit):
    g = torch.clamp(h @ W[p + "gate"].T, max=limit)
    u = torch.clamp(h @ W[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ W[p + "down"].T


def routed(h, W, p, top):
    """(weights, expert ids) [T, top]: softmax over the largest logits alone."""
    z = h @ W[p + "router"].T + W[p + "router.b"]
    ids = torch.argsort(-z, dim=-1, stable=True)[:, :top]
    return torch.softmax(torch.gather(z, 1, ids), -1), ids


def experts(h, W, p, mlp):
    w, ids = routed(h, W, p, mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        share = (w * (ids == e)).sum(-1, keepdim=True)           # 0 for the tokens that did not choose it
        out += share * expert(h, W, f"{p}e{e}.", mlp["expert"]["limit"])
    return out


def depth_average(a, xs):
    return sum(a[j] * x for j, x in enumerate(xs))


def forward(cfg, W, tokens, taps=None):
    """Logits [T, vocab] of one whole sequence; `taps` (a list) gets the residual stream after every layer."""
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = embedding(tokens, W)
    xs = [x]
    for i, lc in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = input_convolution(grouped_rms_norm(x, W[p + "norm1"], eps, groups), W[p + "canon1"])
        x = x + latent_attention(h, W, p + "mix.", lc["mixer"], eps)
        if lc.get("mlp"):
            h = input_convolution(grouped_rms_norm(x, W[p + "norm2"], eps, groups), W[p + "canon2"])
            x = x + experts(h, W, p + "mlp.", lc["mlp"])
        xs.append(x)
        x = depth_average(W[p + "dwa"], xs)
        if taps is not None:
            taps.append(x)
    return grouped_rms_norm(x, W["final.norm"], eps, groups) @ W["embed"].T * cfg["logit_scale"]
