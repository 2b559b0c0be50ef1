"""Plain, slow Vabunex: one function per mechanism, token loops, no cache, any float dtype.  It imports nothing of the
framework: the tests compare the product path against it.

Weights are a flat dict name -> tensor ("l<i>.mix.q", "embed", ...), the configuration is the parsed config.json."""
import math

import torch


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_zero_centred(x, w, eps):
    return unit_rms(x, eps) * (1 + w)


def rotate_interleaved(x, pos, dims, base):
    """x [T, ..., D]: pairs (2i, 2i+1) of the first `dims` entries turned by pos * base^(-2i/dims)."""
    out = x.clone()
    for i in range(dims // 2):
        f = base ** (-2 * i / dims)
        for t in range(x.shape[0]):
            a = float(pos[t]) * f
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = u * c - v * s
            out[t, ..., 2 * i + 1] = v * c + u * s
    return out


def decay_scan(q, k, v, decay):
    """q, k [T, H, D], v [T, H, V], decay [H]: S = decay S + k v^T, o = S^T q."""
    T, H, D = q.shape
    S = q.new_zeros(H, D, v.shape[-1])
    out = []
    for t in range(T):
        S = decay.view(H, 1, 1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(-2)
        out.append((S * q[t].unsqueeze(-1)).sum(1))
    return torch.stack(out)


def wkv_scan(r, k, v, w, u):
    """o = (S + diag(u) k v^T)^T r, then S = diag(w) S + k v^T; w [T, H, D], u [H, D]."""
    T, H, D = r.shape
    S = r.new_zeros(H, D, v.shape[-1])
    out = []
    for t in range(T):
        kv = k[t].unsqueeze(-1) * v[t].unsqueeze(-2)
        out.append(((S + u.unsqueeze(-1) * kv) * r[t].unsqueeze(-1)).sum(1))
        S = w[t].unsqueeze(-1) * S + kv
    return torch.stack(out)


def lightning(h, W, p, c, eps):
    T, H, D, V = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = silu(h @ W[p + "q"].T).view(T, H, D)
    k = silu(h @ W[p + "k"].T).view(T, H, D)
    v = silu(h @ W[p + "v"].T).view(T, H, V)
    o = decay_scan(q, k, v, torch.tensor(c["decay"], dtype=h.dtype)).reshape(T, H * V)
    o = unit_rms(o, eps) * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def wkv(h, W, p, c, eps):
    T, H, D = h.shape[0], c["heads"], c["dim"]
    prev = torch.cat((torch.zeros_like(h[:1]), h[:-1]))
    mix = {s: h + (prev - h) * W[p + "mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ W[p + s].T).view(T, H, D) for s in "rkv")
    w = torch.exp(-torch.exp(torch.tanh(mix["w"] @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"])).view(T, H, D)
    o = unit_rms(wkv_scan(r, k, v, w, W[p + "u"].view(H, D)), eps).reshape(T, H * D)
    return (o * W[p + "norm"] * silu(mix["g"] @ W[p + "g"].T)) @ W[p + "o"].T


def latent_attention(h, W, p, c, eps):
    T, H, D, R, V, L = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    pos = torch.arange(T)
    cq = unit_rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (cq @ W[p + "uq"].T).view(T, H, D + R)
    kv = h @ W[p + "dkv"].T
    lat = unit_rms(kv[:, :L], eps) * W[p + "dkv.norm"]
    rot = c["rot"]
    kr = rotate_interleaved(kv[:, L:], pos, rot["dims"], rot["base"])
    qr = rotate_interleaved(q[..., D:], pos, rot["dims"], rot["base"])
    kn = (lat @ W[p + "uk"].T).view(T, H, D)
    v = (lat @ W[p + "uv"].T).view(T, H, V)
    sc = (torch.einsum("thd,shd->hts", q[..., :D], kn) + torch.einsum("thd,sd->hts", qr, kr)) * c["scale"]
    sc = sc.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    o = torch.einsum("hts,shd->thd", torch.softmax(sc, -1), v)
    o = o * torch.sigmoid(h @ W[p + "g"].T).unsqueeze(-1)
    return o.reshape(T, H * V) @ W[p + "o"].T


MIXERS = {"lightning": lightning, "wkv": wkv, "latent_attention": latent_attention}


def feed_forward(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def layer_runs(cfg):
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def forward(cfg, W, tokens, taps=None):
    """Logits [T, vocab] of one whole sequence; `taps` (a list) gets the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i in layer_runs(cfg):
        lc = cfg["layers"][i]
        h = norm_zero_centred(x, W[f"l{i}.norm1"], eps)
        d = MIXERS[lc["type"]](h, W, f"l{i}.mix.", lc["mixer"], eps)
        if lc.get("mlp"):
            d = d + feed_forward(h, W, f"l{i}.mlp.")
        x = x + d
        if taps is not None:
            taps.append(x)
    return norm_zero_centred(x, W["final.norm"], eps) @ W["head"].T
