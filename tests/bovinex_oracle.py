"""Plain, slow restatement of the Bovinex decoder for the tests: one function per mechanism, one
sequence at a time, whole sequences only (no cache, no chunks), in a chosen floating-point type.
It shares no code with the package. Weights are a dict name -> tensor, the configuration is the
parsed ``config.json`` dict."""
import math

import torch


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_one_plus(x, w, eps):
    return rms(x, eps) * (1 + w)


def rope_frequencies(rot):
    """Angular frequency of every rotated pair and the factor on cos / sin."""
    n, base = rot["dims"], rot["base"]
    freq = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return freq, 1.0

    def dim_of(turns):
        return n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(sc["fast"])), 0)
    hi = min(math.ceil(dim_of(sc["slow"])), n - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, rot):
    """x [T, heads, dim] at positions 0..T-1; dimension i pairs with i + dims/2."""
    freq, amp = rope_frequencies(rot)
    half = rot["dims"] // 2
    ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(
        freq, dtype=torch.float64)
    c = (amp * torch.cos(ang)).to(x.dtype)[:, None]
    s = (amp * torch.sin(ang)).to(x.dtype)[:, None]
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], -1)


def visible(T, mask):
    """[T, T] bool: may position i look at position j?"""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    ok = j <= i
    if mask:
        ok = ok & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
    return ok


def attention(h, W, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = h @ W[p + "q"].T + W[p + "q.b"]
    k = h @ W[p + "k"].T + W[p + "k.b"]
    v = h @ W[p + "v"].T + W[p + "v.b"]
    q = rms(q, eps) * W[p + "q.norm"]
    k = rms(k, eps) * W[p + "k.norm"]
    q = rotate(q.view(T, H, m["dim"]), m["rot"])
    k = rotate(k.view(T, G, m["dim"]), m["rot"])
    v = v.view(T, G, m["vdim"])
    ok = visible(T, m.get("mask"))
    heads = []
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * m["scale"]
        heads.append(torch.softmax(s.masked_fill(~ok, float("-inf")), -1) @ v[:, g])
    o = torch.cat(heads, -1) * torch.sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def gla_decay(h, W, p, m):
    """Per key channel decay in (0, 1): [T, heads, dim]."""
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    return torch.sigmoid(z).pow(1.0 / m["tau"]).view(h.shape[0], m["heads"], m["dim"])


def gla_recurrence(q, k, v, alpha):
    """q, k, alpha [T, H, d], v [T, H, e] -> o [T, H, e] and the final state [H, d, e]."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out), S


def gla(h, W, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q = (h @ W[p + "q"].T).view(T, H, m["dim"]) * m["dim"] ** -0.5
    k = (h @ W[p + "k"].T).view(T, H, m["dim"])
    v = (h @ W[p + "v"].T).view(T, H, m["vdim"])
    o, _ = gla_recurrence(q, k, v, gla_decay(h, W, p, m))
    o = (rms(o, eps) * W[p + "norm"]).reshape(T, -1)
    z = h @ W[p + "g"].T
    return (o * (z * torch.sigmoid(z))) @ W[p + "o"].T


def dense(h, W, p):
    return torch.relu(h @ W[p + "up"].T).square() @ W[p + "down"].T


def route(z, top):
    """Indices and weights of the chosen experts, by router logit."""
    val, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(val, -1)


def moe(h, W, p, cfg):
    idx, w = route(h @ W[p + "router"].T + W[p + "router.b"], cfg["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(idx[t].tolist(), w[t]):
            gate = W[p + f"e{e}.gate"] @ h[t]
            out[t] += a * (W[p + f"e{e}.down"]
                           @ (gate * torch.sigmoid(gate) * (W[p + f"e{e}.up"] @ h[t])))
    return out


def forward(cfg, W, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence; ``trace`` (a list) collects the residual after every
    layer."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens).long()] * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = norm_one_plus(x, W[p + "norm1"], eps)
        mix = {"attention": attention, "gla": gla}[L["type"]](h, W, p + "mix.", L["mixer"], eps)
        mlp = L.get("mlp")
        if mlp is None:
            ff = 0
        elif mlp["kind"] == "dense":
            ff = dense(h, W, p + "mlp.")
        else:
            ff = moe(h, W, p + "mlp.", mlp)
        x = x + (mix + ff)
        if trace is not None:
            trace.append(x)
    return norm_one_plus(x, W["final.norm"], eps) @ W["head"].T
