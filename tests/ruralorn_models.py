"""Small Ruralorn configurations and random weights for the tests."""
import copy
import math

import torch

from bovinex_models import build, error, tokens  # noqa: F401


def layer(heads=4, dim=24, rot=16, vdim=24, rank=40, window=20, base=10000.0, scale=None, mlp=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank,
             scale=scale or 1.1 / math.sqrt(dim + rot), rot=dict(dims=rot, base=base))
    if window:
        m["mask"] = dict(size=window)
    return dict(type="latent_attention", mixer=m, mlp=mlp)


def moe(experts=5, top=2, ff=40, shared=56):
    f = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if shared:
        f["shared"] = dict(ff=shared)
    return f


def config(layers, width=88, vocab=150, eps=1e-5, scale=3.0, logit_scale=0.5, cap=8.0):
    return dict(architecture="Ruralorn", vocab=vocab, width=width, norm=dict(eps=eps),
                embedding=dict(scale=scale), layers=layers, logit_scale=logit_scale,
                logit_softcap=cap)


def settled(cfg, dt):
    """For bf16: the configuration with every expert chosen (their weights still differ), so that no
    close call between two experts falls the other way after rounding."""
    if dt != "bf16":
        return cfg
    cfg = copy.deepcopy(cfg)
    for L in cfg["layers"]:
        if L["mlp"]:
            L["mlp"]["router"]["top"] = L["mlp"]["router"]["experts"]
    return cfg


def weights(cfg, seed=0, dtype=torch.bfloat16, gain=1.0):
    """Random tensors of every name the design has; linear weights keep the scale of their input,
    norms are not neutral."""
    g = torch.Generator().manual_seed(seed)
    W, out = cfg["width"], {}

    def lin(name, rows, cols, k=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * (k * gain / math.sqrt(cols))).to(dtype)

    def vec(name, n):
        out[name] = (1 + 0.2 * torch.randn(n, generator=g)).to(dtype)
    out["embed"] = (torch.randn(cfg["vocab"], W, generator=g) / cfg["embedding"]["scale"]).to(dtype)
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        H = m["heads"]
        vec(p + "norm1", W)
        lin(p + "mix.q", H * (m["dim"] + m["rot_dim"]), W, 1.5)
        lin(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], W, 1.5)
        vec(p + "mix.dkv.norm", m["kv_rank"])
        lin(p + "mix.uk", H * m["dim"], m["kv_rank"], 1.5)
        lin(p + "mix.uv", H * m["vdim"], m["kv_rank"], 1.5)
        lin(p + "mix.g", H * m["vdim"], W)
        lin(p + "mix.o", W, H * m["vdim"])
        if not f:
            continue
        vec(p + "norm2", W)
        lin(p + "mlp.router", f["router"]["experts"], W, 2.0)
        for x in range(f["router"]["experts"]):
            lin(p + f"mlp.e{x}.up", f["expert"]["ff"], W, 1.5)
            lin(p + f"mlp.e{x}.down", W, f["expert"]["ff"], 1.5)
        if f.get("shared"):
            lin(p + "mlp.shared.up", f["shared"]["ff"], W, 1.5)
            lin(p + "mlp.shared.down", W, f["shared"]["ff"], 1.5)
    vec("final.norm", W)
    lin("head", cfg["vocab"], W, 4.0)
    return out


# name -> configuration; between them: sizes on and off the grid of 8, few and many heads, dim != vdim,
# latents of every kernel width and beyond, head sizes too wide for expanded keys, layers with other
# windows, no window, no feed-forward, no shared expert, one expert, one / several / all chosen
ZOO = {
    "mixed": config([layer(6, 40, 24, 32, 72, window=20, mlp=moe(5, 2, 44)),
                     layer(3, 24, 8, 40, 56, window=7, base=500.0, mlp=moe(7, 1, 32, None)),
                     layer(6, 16, 32, 24, 104, window=33, mlp=None)], width=120, vocab=333),
    "plain": config([layer(2, 64, 64, 64, 128, window=None, mlp=moe(4, 4, 64, 24)),
                     layer(20, 32, 16, 16, 64, window=64, base=3e5, mlp=moe(1, 1, 48, 96))],
                    width=128, vocab=200, eps=1e-3, logit_scale=1.0, cap=5.0),
    "wide": config([layer(40, 128, 64, 128, 384, window=48, mlp=moe(6, 3, 56, 72)),
                    layer(12, 72, 40, 104, 512, window=130, mlp=moe(9, 2, 128, 136))],
                   width=192, vocab=257, logit_scale=2.0, cap=30.0),
    "odd": config([layer(3, 14, 6, 10, 27, window=9, mlp=moe(7, 3, 13, 21)),
                   layer(5, 13, 10, 19, 51, window=30, mlp=moe(3, 2, 9, 11))],
                  width=50, vocab=91, scale=1.0),
    "beyond": config([layer(2, 136, 72, 24, 88, window=40, mlp=moe(3, 1, 40, 40)),
                      layer(4, 24, 16, 136, 600, window=25, mlp=moe(2, 1, 24, 16))],
                     width=104, vocab=120),
}
