"""Small Bovinex configurations and random weights for the tests."""
import math

import torch

YARN = dict(factor=4.0, original=64, fast=8.0, slow=1.0)


def attn(heads=4, kv=2, dim=24, vdim=24, rot=None, base=10000.0, scaling=None, window=None,
         keep=0, scale=None, mlp=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale or 0.9 / math.sqrt(dim),
             rot=dict(dims=dim if rot is None else rot, base=base))
    if scaling:
        m["rot"]["scaling"] = scaling
    if window:
        m["mask"] = dict(size=window, keep_first=keep)
    return dict(type="attention", mixer=m, mlp=mlp)


def gla(heads=2, dim=16, vdim=24, tau=4.0, mlp=None):
    return dict(type="gla", mixer=dict(heads=heads, dim=dim, vdim=vdim, tau=tau), mlp=mlp)


def dense(ff=72):
    return dict(kind="dense", ff=ff)


def moe(experts=5, top=2, ff=40):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def config(layers, width=88, vocab=150, eps=1e-5, scale=3.0):
    return dict(architecture="Bovinex", vocab=vocab, width=width, norm=dict(eps=eps),
                embedding=dict(scale=scale), layers=layers)


def weights(cfg, seed=0, rank=12, dtype=torch.bfloat16, gain=1.0):
    """Random tensors of every name the design has; linear weights keep the scale of their
    input, norms and biases are not neutral."""
    g = torch.Generator().manual_seed(seed)
    W, out = cfg["width"], {}

    def lin(name, rows, cols, k=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * (k * gain / math.sqrt(cols))).to(dtype)

    def vec(name, n, mean=0.0, std=0.2):
        out[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)
    out["embed"] = (torch.randn(cfg["vocab"], W, generator=g) / cfg["embedding"]["scale"]).to(dtype)
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        vec(p + "norm1", W)
        H, d, e = m["heads"], m["dim"], m["vdim"]
        kv = m["kv_heads"] if L["type"] == "attention" else H
        for n, rows in (("q", H * d), ("k", kv * d), ("v", kv * e), ("g", H * e)):
            lin(p + "mix." + n, rows, W)
        lin(p + "mix.o", W, H * e)
        if L["type"] == "attention":
            for n, rows in (("q", H * d), ("k", kv * d), ("v", kv * e)):
                vec(p + f"mix.{n}.b", rows)
            vec(p + "mix.q.norm", H * d, 1.5)
            vec(p + "mix.k.norm", kv * d, 1.5)
        else:
            vec(p + "mix.norm", e, 1.0)
            lin(p + "mix.a1", rank, W)
            lin(p + "mix.a2", H * d, rank, 2.0)
            vec(p + "mix.a2.b", H * d, 1.0, 1.0)
        if f and f["kind"] == "dense":
            lin(p + "mlp.up", f["ff"], W)
            lin(p + "mlp.down", W, f["ff"])
        elif f:
            for x in range(f["router"]["experts"]):
                lin(p + f"mlp.e{x}.gate", f["expert"]["ff"], W)
                lin(p + f"mlp.e{x}.up", f["expert"]["ff"], W)
                lin(p + f"mlp.e{x}.down", W, f["expert"]["ff"])
            lin(p + "mlp.router", f["router"]["experts"], W, 2.0)
            vec(p + "mlp.router.b", f["router"]["experts"])
    vec("final.norm", W)
    lin("head", cfg["vocab"], W, 2.0)
    return out


# name -> configuration; between them: head sizes of every kernel width, dim != vdim, partial
# rotation, YaRN, one kv head, as many kv heads as heads, no window, no kept tokens, no feed-forward,
# one expert, all experts chosen, expert sizes off the 8-column grid
ZOO = {
    "mixed": config([attn(6, 3, 40, 24, rot=24, scaling=YARN, window=20, keep=3, mlp=dense(76)),
                     gla(3, 24, 40, mlp=moe(5, 2, 44)),
                     attn(6, 1, 40, 24, window=7, keep=1, mlp=moe(3, 1, 32)),
                     gla(3, 20, 28, tau=1.0, mlp=dense(40))], width=120, vocab=333),
    "plain": config([gla(1, 32, 32, mlp=None), attn(2, 2, 64, 64, window=None, mlp=dense(128)),
                     attn(8, 1, 32, 64, window=33, keep=0, scaling=YARN, mlp=None),
                     gla(4, 64, 20, tau=16.0, mlp=moe(4, 4, 64))], width=128, vocab=200, eps=1e-3),
    "wide": config([attn(4, 2, 128, 128, rot=64, window=48, keep=5, mlp=dense(256)),
                    gla(2, 128, 128, tau=8.0, mlp=moe(1, 1, 96)),
                    attn(3, 3, 72, 136, window=64, keep=8, mlp=moe(6, 3, 56)),
                    gla(1, 136, 72, tau=2.0, mlp=dense(64))], width=192, vocab=257),
    "odd": config([attn(3, 1, 14, 10, rot=6, window=9, keep=2, mlp=dense(27)),
                   gla(3, 7, 9, tau=3.0, mlp=moe(7, 3, 13)),
                   attn(2, 1, 200, 30, rot=40, window=12, keep=4, mlp=None)], width=50, vocab=91),
}


def build(cfg, W, dtype, batch, length, **kw):
    from easy_to_hard_b200.models.hybrid import HybridLM, hybrid_config
    model = HybridLM.from_tensors(hybrid_config(cfg), W, device="cuda", dtype=dtype)
    return model.make_engine(batch, length, use_graph=kw.pop("use_graph", False), **kw)


def tokens(cfg, n, seed=0):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def error(got, want, q=1.0):
    """Root mean square difference of logits over the vocabulary (means removed) relative to the
    spread of the expected logits, at the worst position (or at quantile ``q`` of them: in bf16 an
    expert whose logit ties with another's may swap)."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    e = d.pow(2).mean(-1).sqrt().flatten() / w.pow(2).mean().sqrt()
    return float(torch.quantile(e, q))
