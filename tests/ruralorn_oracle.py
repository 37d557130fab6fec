"""Plain, slow restatement of the Ruralorn decoder for the tests: one function per mechanism, one
sequence at a time, whole sequences only (no cache, no chunks), keys and values expanded per head, in
a chosen floating-point type. It shares no code with the package. Weights are a dict name -> tensor,
the configuration is the parsed ``config.json`` dict."""
import math

import torch


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotate_pairs(x, base, dims):
    """x [T, heads, d] at positions 0..T-1: neighbours (2i, 2i + 1) of the first ``dims`` turn by
    t * base^(-2i / dims)."""
    t = torch.arange(x.shape[0], dtype=torch.float64)[:, None]
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)],
                     dtype=torch.float64)
    c, s = torch.cos(t * f).to(x.dtype)[:, None], torch.sin(t * f).to(x.dtype)[:, None]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], -1)


def visible(T, size):
    """[T, T] bool: position i sees itself and the ``size - 1`` positions before it (None: all)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    ok = j <= i
    return ok if not size else ok & (i - j < size)


def attend(q, k, v, scale, ok):
    """q, k [T, H, d], v [T, H, e] -> [T, H, e]; softmax over the keys ``ok`` lets through."""
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    return torch.einsum("hij,jhe->ihe", torch.softmax(s.masked_fill(~ok, -math.inf), -1), v)


def latents(h, W, p, m, eps):
    """The normed latent [T, kv_rank] and the rotated key part [T, rot_dim] of every token."""
    y = h @ W[p + "dkv"].T
    r = m["kv_rank"]
    c = rms_norm(y[:, :r], W[p + "dkv.norm"], eps)
    return c, rotate_pairs(y[:, None, r:], m["rot"]["base"], m["rot"]["dims"])[:, 0]


def expand(c, kr, W, p, m):
    """Keys [T, H, dim + rot_dim] and values [T, H, vdim] from latents and the shared key part."""
    T, H = c.shape[0], m["heads"]
    k = (c @ W[p + "uk"].T).view(T, H, m["dim"])
    v = (c @ W[p + "uv"].T).view(T, H, m["vdim"])
    return torch.cat([k, kr[:, None].expand(T, H, -1)], -1), v


def queries(h, W, p, m):
    T, d = h.shape[0], m["dim"]
    q = (h @ W[p + "q"].T).view(T, m["heads"], d + m["rot_dim"])
    return torch.cat([q[..., :d], rotate_pairs(q[..., d:], m["rot"]["base"], m["rot"]["dims"])], -1)


def latent_attention(h, W, p, m, eps):
    k, v = expand(*latents(h, W, p, m, eps), W, p, m)
    o = attend(queries(h, W, p, m), k, v, m["scale"],
               visible(h.shape[0], (m.get("mask") or {}).get("size")))
    return (o.flatten(1) * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def gelu(x):
    return 0.5 * x * (1 + torch.erf(x / math.sqrt(2)))


def expert(h, W, p):
    return gelu(h @ W[p + "up"].T) @ W[p + "down"].T


def route(z, top):
    """Indices of the ``top`` largest scores and these scores (sigmoid of the router's output)."""
    s = torch.sigmoid(z)
    idx = torch.argsort(z, dim=-1, descending=True, stable=True)[:, :top]
    return idx, torch.gather(s, 1, idx)


def moe(h, W, p, f):
    idx, s = route(h @ W[p + "router"].T, f["router"]["top"])
    rows = []
    for t in range(h.shape[0]):
        y = expert(h[t], W, p + "shared.") if f.get("shared") else torch.zeros_like(h[t])
        for e, w in zip(idx[t].tolist(), s[t]):
            y = y + expert(w * h[t], W, p + f"e{e}.")
        rows.append(y)
    return torch.stack(rows)


def output(x, W, cfg):
    z = rms_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["head"].T * cfg["logit_scale"]
    return cfg["logit_softcap"] * torch.tanh(z / cfg["logit_softcap"])


def forward(cfg, W, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence; ``trace`` (a list) collects the residual after every
    layer."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens).long()] * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + latent_attention(rms_norm(x, W[p + "norm1"], eps), W, p + "mix.", L["mixer"], eps)
        if L.get("mlp"):
            x = x + moe(rms_norm(x, W[p + "norm2"], eps), W, p + "mlp.", L["mlp"])
        if trace is not None:
            trace.append(x)
    return output(x, W, cfg)
