"""Kernels of the Ruralorn decoder, one mechanism at a time, against the plain restatement."""
import math

import pytest
import torch

import ruralorn_models as M
import ruralorn_oracle as O

pytestmark = pytest.mark.gpu
DT = {"bf16": torch.bfloat16, "fp32": torch.float32}


def _ok():
    from easy_to_hard_b200.ops import _lib
    torch.cuda.synchronize()
    assert _lib.read_status() == 0


def _tol(dtype, fp32=2e-5, bf16=2e-2):
    return fp32 if dtype == torch.float32 else bf16


def _close(got, want, tol):
    d = (got.double().cpu() - want.double().cpu()).abs().max()
    s = max(1.0, float(want.abs().max()))
    assert float(d) <= tol * s, (float(d), s)


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("W", [64, 90, 1032])
def test_norm_with_outputs_that_carry_their_weight(dt, W):
    from easy_to_hard_b200.ops import hybrid as hy
    dtype = DT[dt]
    g = torch.Generator().manual_seed(W)
    n, top = 7, 3
    x, wt = torch.randn(n, W, generator=g), 1 + 0.3 * torch.randn(W, generator=g)
    y = torch.randn(n * top, W, generator=g).to(dtype)
    place = torch.randperm(n * top, generator=g).view(n, top).int()
    xd = x.cuda()
    out = torch.zeros(n, (W + 7) // 8 * 8, dtype=dtype, device="cuda")
    hy.stream_norm(xd, wt.cuda(), out, eps=1e-3, experts=(y.cuda(), place.cuda(), None))
    full = x.double() + y.double()[place.long()].sum(1)
    _close(xd, full, 1e-6)
    _close(out[:, :W], O.rms_norm(full, wt.double(), 1e-3), _tol(dtype, 1e-5, 1e-2))
    _ok()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("T", [1, 5, 64, 100, 300, 700])
@pytest.mark.parametrize("K,F,tail", [(72, 168, 24), (256, 512, 8), (50, 88, 0), (320, 768, 40)])
def test_projection_with_gelu(dt, T, K, F, tail):
    from easy_to_hard_b200.ops import gemm
    dtype = DT[dt]
    g = torch.Generator().manual_seed(T + K)
    kp = (K + 7) // 8 * 8
    w = torch.zeros(F + tail, kp, dtype=dtype, device="cuda")
    w[:, :K] = (torch.randn(F + tail, K, generator=g) * 2 / math.sqrt(K)).to(dtype)
    x = torch.zeros(T, kp, dtype=dtype, device="cuda")
    x[:, :K] = torch.randn(T, K, generator=g).to(dtype)
    out = torch.empty(T, F, dtype=dtype, device="cuda")
    tl = torch.empty(T, max(tail, 8), dtype=torch.float32, device="cuda")
    gemm.linear_packed(x[:, :K], w[:, :K], out, act="gelu", act_from=0, tail=tl if tail else None)
    y = x.double() @ w.double().T
    _close(out, O.gelu(y[:, :F]), _tol(dtype, 2e-6, 5e-3))
    if tail:
        _close(tl[:, :tail], y[:, F:], 1e-5)
        for bias in (None, torch.randn(tail, generator=g).cuda()):      # nothing but a tail
            gemm.linear_packed(x[:, :K], w[F:, :K], None, tail=tl, bias=bias)
            _close(tl[:, :tail], y[:, F:] + (0 if bias is None else bias), 1e-5)
    _ok()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("T", [1, 3, 90, 300])
def test_logits_are_scaled_and_capped(dt, T):
    from easy_to_hard_b200.ops import gemm
    g = torch.Generator().manual_seed(T)
    x = torch.randn(T, 96, generator=g).to(DT[dt]).cuda()
    w = torch.randn(136, 96, generator=g).to(DT[dt]).cuda()
    y = x.double() @ w.double().T
    for scale, cap in ((1.0, 0.0), (0.3, 0.0), (1.0, 4.0), (3.0, 20.0)):
        out = torch.empty(T, 136, device="cuda")
        gemm.linear_f32_out(x, w, out, scale=scale, softcap=cap)
        want = cap * torch.tanh(y * scale / cap) if cap else y * scale
        _close(out, want, 1e-5)
        assert not cap or float(want.abs().max()) > 0.9 * cap      # the cap is felt
    _ok()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("n,E,top,K,F", [(1, 4, 2, 64, 40), (33, 5, 3, 88, 72), (64, 8, 8, 128, 128),
                                         (300, 3, 1, 96, 136), (700, 9, 4, 64, 64), (6, 1, 1, 64, 24),
                                         (5, 300, 6, 64, 64), (900, 3, 2, 256, 192), (9, 6, 2, 50, 24)])
def test_sigmoid_routing_weighted_input_and_experts(dt, n, E, top, K, F):
    from easy_to_hard_b200.ops import gemm, hybrid as hy
    dtype = DT[dt]
    g = torch.Generator().manual_seed(n)
    z = torch.randn(n, E, generator=g)
    if E > 2 and top < E:
        z[:, 1] -= 100                                     # an expert that nobody chooses
    zp = torch.full((n, E + 3), 50.0, device="cuda")       # columns that are not experts
    zp[:, :E] = z
    Kp = (K + 7) // 8 * 8
    h, hg = (torch.zeros(r, Kp, dtype=dtype, device="cuda")[:, :K] for r in (n, n * top))
    h.copy_(torch.randn(n, K, generator=g))
    off = torch.zeros(E + 1, dtype=torch.int32, device="cuda")
    place, sel = (torch.zeros(n, top, dtype=torch.int32, device="cuda") for _ in range(2))
    w = torch.zeros(n, top, device="cuda")
    hy.moe_route(zp, E, top, h, hg, off, place, w, sel, score="sigmoid", weight_input=True)
    idx, want_w = O.route(z.double(), top)
    _close(w, want_w, 1e-6)
    o, pl = off.tolist(), place.cpu().long()
    assert o[0] == 0 and o[-1] == n * top
    assert [b - a for a, b in zip(o, o[1:])] == torch.bincount(idx.flatten(), minlength=E).tolist()
    assert sorted(pl.flatten().tolist()) == list(range(n * top))
    assert torch.equal(torch.bucketize(pl, off.cpu()[1:], right=True), idx)
    rows = hg[pl.cuda()]
    _close(rows, want_w[..., None] * h.double().cpu()[:, None], _tol(dtype, 1e-6, 5e-3))
    Fp = (F + 7) // 8 * 8
    up = torch.zeros(E * Fp, Kp, dtype=dtype, device="cuda")[:, :K]
    up.copy_(torch.randn(E * Fp, K, generator=g) * 2 / math.sqrt(K))
    a = torch.full((n * top, Fp), 7.0, dtype=dtype, device="cuda")
    gemm.grouped_linear(hg, up, a, off, E, n, act="gelu")
    for e in range(E):
        x = hg[o[e]: o[e + 1]].double()
        if len(x):
            _close(a[o[e]: o[e + 1]], O.gelu(x @ up[e * Fp: (e + 1) * Fp].double().T),
                   _tol(dtype, 1e-5, 1e-2))
    _ok()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("T", [1, 5, 64, 100, 300])
@pytest.mark.parametrize("H,K,F,step", [(3, 24, 40, 40), (5, 64, 96, 72), (2, 128, 512, 192),
                                        (40, 8, 24, 24), (4, 512, 128, 512)])
def test_one_product_per_head(dt, T, H, K, F, step):
    """Heads at a column step wider than the contraction; the columns between them are not zero."""
    from easy_to_hard_b200.ops import gemm
    dtype = DT[dt]
    g = torch.Generator().manual_seed(T + H)
    x = torch.randn(T, H * step + 8, generator=g).to(dtype).cuda()
    w = (torch.randn(H * F, K, generator=g) / math.sqrt(K)).to(dtype).cuda()
    want = torch.einsum("thk,hfk->thf", x[:, : H * step].double().view(T, H, step)[..., :K],
                        w.double().view(H, F, K))
    buf = torch.full((T, 16 + H * F), 3.0, dtype=dtype, device="cuda")
    out = buf[:, 8: 8 + H * F]
    gemm.batched_linear(x, w, out, batch=H, k=K, x_step=step, out_step=F)
    _close(out, want.flatten(1), _tol(dtype, 1e-5, 6e-3))
    gate = torch.randn(T, H * F, generator=g).to(dtype)
    out.copy_(gate)
    gemm.batched_linear(x, w, out, batch=H, k=K, x_step=step, out_step=F, gate=True)
    _close(out, want.flatten(1).cpu() * torch.sigmoid(gate.double()), _tol(dtype, 1e-5, 1e-2))
    assert bool((buf[:, :8] == 3).all()) and bool((buf[:, 8 + H * F:] == 3).all())
    _ok()


# ------------------------------------------------------------------ latent attention

class _Latent:
    """One latent attention layer's kernels on given projections of several sequences."""

    def __init__(self, L, dtype, slots, smax, seed=3, uk=None, uv=None, expand=True):
        from easy_to_hard_b200.models.hybrid import _pad_heads, hybrid_config, pad8
        from easy_to_hard_b200.ops import hybrid as hy
        self.hy, self.pad = hy, _pad_heads
        m = self.m = hybrid_config(M.config([L])).layers[0].mixer
        self.L, self.dtype, self.eps = L["mixer"], dtype, 1e-5
        H, r, rp = m.heads, m.kv_rank, pad8(m.kv_rank)
        g = torch.Generator().manual_seed(seed)
        self.W = {"dkv.norm": 1 + 0.2 * torch.randn(r, generator=g)}
        for n, d, t in (("uk", m.dim, uk), ("uv", m.vdim, uv)):
            t = torch.randn(H * d, r, generator=g) / math.sqrt(r) if t is None else t
            self.W[n] = t.to(dtype).float()
        kv = torch.zeros(H * (pad8(m.dim) + pad8(m.vdim)), rp)
        kv[:, :r] = torch.cat([_pad_heads(self.W["uk"], H, (m.dim,)),
                               _pad_heads(self.W["uv"], H, (m.vdim,))])
        ukt = kv[: H * pad8(m.dim)].view(H, -1, rp).transpose(1, 2).reshape(H * rp, -1)
        # columns: q head by head, latent and shared key part, gate head by head
        self.parts = ((H, (m.dim, m.rot_dim)), (1, (r, m.rot_dim)), (H, (m.vdim,)))
        self.offs, at = [], 0
        for h, sizes in self.parts:
            self.offs.append(at)
            at += h * sum(map(pad8, sizes))
        # whatever earlier sequences left in the cache must not matter
        self.cache = torch.full((slots, smax, rp + pad8(m.rot_dim)), 1e4, dtype=dtype, device="cuda")
        self.k = hy.LatentAttention(m, self.offs, self.cache, m.rot.table(
            smax, "cuda", pad8(m.rot_dim) // 2), kv.to("cuda", dtype), ukt.to("cuda", dtype)
            .contiguous(), _pad_heads(self.W["dkv.norm"], 1, (r,)).cuda(), self.eps)
        self.k.can_expand &= expand

    def pack(self, proj):
        """[n, H (dim + rot) | rank + rot | H vdim] -> the packed activation."""
        cols = proj.split([h * sum(s) for h, s in self.parts], 1)
        return torch.cat([self.pad(c.t().contiguous(), h, s) for c, (h, s) in
                          zip(cols, self.parts)]).t().contiguous().to("cuda", self.dtype)

    def heads(self, act):
        m = self.m
        x = act[:, self.offs[2]:].float().cpu().view(act.shape[0], m.heads, -1)
        assert not x[..., m.vdim:].any()
        return x[..., : m.vdim].flatten(1)

    def forward(self, entries):
        """entries: (slot, first position, projections); one launch sequence for all of them."""
        act = torch.cat([self.pack(p) for _, _, p in entries])
        lens = [len(p) for _, _, p in entries]
        pos = _i32([at + i for _, at, p in entries for i in range(len(p))])
        slot = _i32([s for s, _, p in entries for _ in range(len(p))])
        if max(lens) == 1:
            self.k.decode(act, pos, slot)
        else:
            assert lens == sorted(lens, reverse=True)
            ctx = self.hy.LatentContext(lens, [at for _, at, _ in entries],
                                        [s for s, _, _ in entries], self.m.window,
                                        self.k.can_expand, "cuda")
            self.k.prompt(act, pos, slot, _i32([sum(lens[:i]) for i in range(len(lens) + 1)]), ctx)
        return self.heads(act).split(lens)

    def run(self, proj, cuts, slot):
        return torch.cat([self.forward([(slot, a, proj[a:b])])[0] for a, b in zip(cuts, cuts[1:])])

    def expected(self, proj):
        """The oracle's mechanisms on given projections."""
        m, T, W = self.L, proj.shape[0], {n: w.double() for n, w in self.W.items()}
        H, d, r, e, k = (m[n] for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        rot = (m["rot"]["base"], m["rot"]["dims"])
        q, y, g = proj.double().split([H * (d + r), k + r, H * e], 1)
        q = q.view(T, H, d + r)
        q = torch.cat([q[..., :d], O.rotate_pairs(q[..., d:], *rot)], -1)
        c = O.rms_norm(y[:, :k], W["dkv.norm"], self.eps)
        keys, vals = O.expand(c, O.rotate_pairs(y[:, None, k:], *rot)[:, 0], W, "", m)
        o = O.attend(q, keys, vals, m["scale"], O.visible(T, (m.get("mask") or {}).get("size")))
        return o.flatten(1) * torch.sigmoid(g)

    def random(self, T, seed=5, k=1.0):
        n = sum(h * sum(s) for h, s in self.parts)
        g = torch.Generator().manual_seed(seed)
        return (k * torch.randn(T, n, generator=g)).to(self.dtype).float()


LAYERS = {
    "r72": M.layer(6, 40, 24, 32, 72, window=20),
    "r512": M.layer(16, 128, 64, 128, 512, window=140),
    "r512h40": M.layer(40, 64, 64, 64, 512, window=100),
    "r128full": M.layer(4, 64, 32, 64, 128, window=None),
    "r384": M.layer(24, 56, 48, 96, 384, window=64),
    "r27": M.layer(3, 14, 6, 10, 27, window=9),
    "r104": M.layer(17, 24, 8, 120, 104, window=150),
    "r600": M.layer(3, 40, 16, 24, 600, window=31),
    "wide": M.layer(2, 136, 72, 140, 200, window=70),
    "one": M.layer(1, 8, 2, 8, 8, window=130),
}


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("name", LAYERS)
def test_attention_prompts_portions_and_decoding(dt, name):
    dtype, T = DT[dt], 330
    a = _Latent(LAYERS[name], dtype, 3, 336)
    proj = a.random(T)
    want = a.expected(proj)
    for c in ([0, T], [0, 2, 37, 39, 168, 296, T], list(range(0, T, 30)),
              [0, 21] + list(range(22, 60)) + [300] + list(range(301, T + 1))):
        a.cache.fill_(1e4)
        _close(a.run(proj, c, 1), want[: c[-1]], _tol(dtype, 2e-5, 2.5e-2))
    _ok()


@pytest.mark.parametrize("name", ["r72", "r512", "r128full", "r104"])
def test_absorbed_and_expanded_keys_agree(name):
    """The same prompt through both kernels."""
    a, b = (_Latent(LAYERS[name], torch.bfloat16, 1, 200, expand=x) for x in (True, False))
    proj = a.random(200)
    assert a.k.can_expand and not b.k.can_expand
    x, y, want = a.run(proj, [0, 200], 0), b.run(proj, [0, 200], 0), a.expected(proj)
    _close(x, want, 2e-2)
    _close(y, want, 2e-2)
    assert torch.equal(a.cache, b.cache)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("name", ["r72", "r512", "r384", "r104"])
def test_window_edges_stand_out(dt, name):
    """One key at a time is made to dominate the scores of one query, through its rotated part at
    their distance or through its latent: just inside and just outside the window, and the query
    itself. The output then is that key's value, or does not contain it at all."""
    dtype, L = DT[dt], LAYERS[name]
    m = L["mixer"]
    win = m["mask"]["size"]
    T = win + 140
    i = T - 3
    H, d, r, e, k = (m[n] for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    base = a = _Latent(L, dtype, 2, T)
    freq = torch.tensor([m["rot"]["base"] ** (-2.0 * x / r) for x in range(r // 2)],
                        dtype=torch.float64)
    for j, seen in {i: True, i - 1: True, i - win + 1: True, i - win: False, i - win - 1: False,
                    0: False}.items():
        assert bool(O.visible(T, win)[i, j]) == seen
        for through in ("rotation", "latent"):
            g = torch.Generator().manual_seed(j)
            proj = base.random(T, 9, 0.2)
            q = proj[:, : H * (d + r)].view(T, H, d + r)
            c = proj[:, H * (d + r): H * (d + r) + k]
            kr = proj[:, H * (d + r) + k: H * (d + r) + k + r]
            c[j] = torch.randn(k, generator=g)
            if through == "rotation":
                v = torch.randn(r, generator=g)
                q[i, :, d:] = v
                u = torch.polar(torch.ones(r // 2, dtype=torch.float64), (i - j) * freq)
                z = torch.view_as_real(torch.view_as_complex(v.double().view(-1, 2)) * u).flatten()
                kr[j] = (z * 40 / (m["scale"] * (v * v).sum())).float()
            else:
                cn = O.rms_norm(c[j].double(), a.W["dkv.norm"].double(), a.eps)
                keys = (a.W["uk"].double() @ cn).view(H, d)
                q[i, :, :d] = (keys * 40 / (m["scale"] * keys.square().sum(1, keepdim=True))).float()
            proj = proj.to(dtype).float()
            want = a.expected(proj)
            val = a.W["uv"].double() @ O.rms_norm(proj[j, H * (d + r): H * (d + r) + k].double(),
                                                  a.W["dkv.norm"].double(), a.eps)
            share = want[i] / torch.sigmoid(proj[i, -H * e:].double())
            near = float((share - val).norm() / val.norm())
            assert near < 0.05 if seen else near > 0.5     # the test shows what it should
            for cuts in ([0, T], [0, i] + list(range(i + 1, T + 1)), [0, 3, i - 1, T],
                         [0, i - 30, T]):
                a.cache.fill_(1e4)
                got = a.run(proj, cuts, 0)
                _close(got[i:], want[i:], _tol(dtype, 1e-4, 3e-2))
    _ok()


@pytest.mark.parametrize("dt", DT)
def test_prompts_portions_and_decode_rows_in_one_launch(dt):
    """Whole prompts, continued ones and single tokens of unequal sequences together."""
    dtype = DT[dt]
    a = _Latent(LAYERS["r512"], dtype, 6, 400)
    seqs = {s: a.random(n, s) for s, n in {4: 360, 0: 240, 5: 130, 2: 61, 1: 70}.items()}
    want = {s: a.expected(p) for s, p in seqs.items()}
    plan = [[(4, 150), (2, 60), (0, 9), (5, 1)], [(0, 100), (1, 69), (5, 25), (4, 2)],
            [(5, 30), (4, 29), (0, 23), (2, 1)], [(4, 1), (0, 1), (5, 1), (1, 1)],
            [(4, 160), (0, 90), (5, 3)], [(5, 70), (4, 18), (0, 17)]]
    at = dict.fromkeys(seqs, 0)
    for step in plan:
        out = a.forward([(s, at[s], seqs[s][at[s]: at[s] + n]) for s, n in step])
        for (s, n), x in zip(step, out):
            _close(x, want[s][at[s]: at[s] + n], _tol(dtype, 2e-5, 2.5e-2))
            at[s] += n
    assert at == {s: len(p) for s, p in seqs.items()}
    assert bool((a.cache[3] == 1e4).all())                 # a slot that took no part
    _ok()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("splits", [1, 2, 4, 8])
def test_keys_split_over_a_cluster(dt, splits):
    """Any number of keys over any number of CTAs, fewer keys than CTAs included."""
    dtype = DT[dt]
    a = _Latent(LAYERS["r384"], dtype, 2, 80)
    a.k.splits = lambda n: splits if dtype == torch.bfloat16 else 1
    proj = a.random(75)
    want = a.expected(proj)
    _close(a.run(proj, list(range(76)), 1), want, _tol(dtype, 2e-5, 2.5e-2))
    _close(a.run(proj, [0, 3, 70, 72, 75], 0), want, _tol(dtype, 2e-5, 2.5e-2))
    _ok()
