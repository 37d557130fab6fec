"""Kernels of the hybrid decoders, one mechanism at a time, against the plain restatement."""
import math

import pytest
import torch

import bovinex_models as M
import bovinex_oracle as O

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


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("W", [64, 90, 1032])
def test_stream_norm(dt, W):
    from easy_to_hard_b200.ops import hybrid as hy
    dtype = DT[dt]
    g = torch.Generator().manual_seed(W)
    n, vocab, top = 7, 31, 3
    emb = torch.randn(vocab, W, generator=g).to(dtype)
    wt = 0.3 * torch.randn(W, generator=g)
    tok = torch.tensor([0, 30, 5, 5, 7, 1, 2], dtype=torch.int32)
    x = torch.zeros(n, W, device="cuda")
    out = torch.zeros(n, (W + 7) // 8 * 8, dtype=dtype, device="cuda")
    col = torch.tensor([9], dtype=torch.int32, device="cuda")
    pad = torch.arange(n, dtype=torch.int32, device="cuda")
    pos = torch.full((n,), -5, dtype=torch.int32, device="cuda")
    hy.stream_norm(x, wt.cuda(), out, eps=1e-3, offset=1.0, tokens=tok.cuda(), emb=emb.cuda(),
                   emb_scale=2.5, col=col, left_pad=pad, pos_out=pos)
    want = emb[tok.long()].float() * 2.5
    _close(x, want, 1e-6)
    _close(out[:, :W], O.norm_one_plus(want.double(), wt.double(), 1e-3), _tol(dtype, 1e-5, 1e-2))
    assert pos.tolist() == [9, 8, 7, 6, 5, 4, 3]
    # expert outputs of the layer before, then only some rows
    y = torch.randn(n * top, W, generator=g).to(dtype)
    place = torch.randperm(n * top, generator=g).view(n, top).int()
    w = torch.rand(n, top, generator=g)
    full = want + (w[..., None] * y.float()[place.long()]).sum(1)
    rows = torch.tensor([6, 2], dtype=torch.int32)
    hy.stream_norm(x, wt.cuda(), out, eps=1e-3, rows=rows.cuda(),
                   experts=(y.cuda(), place.cuda(), w.cuda()))
    _close(x, want, 1e-6)                                  # the stream itself is untouched
    _close(out[:2, :W], O.rms(full[[6, 2]].double(), 1e-3) * wt.double(), _tol(dtype, 1e-5, 1e-2))
    hy.stream_norm(x, wt.cuda(), out, eps=1e-3, offset=1.0,
                   experts=(y.cuda(), place.cuda(), w.cuda()))
    _close(x, full, 1e-5)
    _ok()


def test_token_ids_outside_the_table_are_reported():
    from easy_to_hard_b200.ops import _lib, hybrid as hy
    x = torch.zeros(2, 16, device="cuda")
    out = torch.zeros(2, 16, device="cuda")
    hy.stream_norm(x, torch.ones(16, device="cuda"), out, eps=1e-5,
                   tokens=torch.tensor([3, 99], dtype=torch.int32, device="cuda"),
                   emb=torch.ones(8, 16, device="cuda"))
    torch.cuda.synchronize()
    assert _lib.read_status() == 106


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("T", [1, 5, 64, 100, 300, 700])
@pytest.mark.parametrize("K,F,tail", [(72, 168, 24), (256, 512, 8), (50, 88, 0), (320, 768, 40)])
def test_packed_projection(dt, T, K, F, tail):
    """Bias, squared ReLU from a feature on, fp32 tail."""
    from easy_to_hard_b200.ops import gemm
    dtype = DT[dt]
    g = torch.Generator().manual_seed(T + K)
    kp = (K + 7) // 8 * 8
    w = torch.zeros(F + tail, kp, dtype=dtype, device="cuda")
    w[:, :K] = (torch.randn(F + tail, K, generator=g) / math.sqrt(K)).to(dtype)
    x = torch.zeros(T, kp, dtype=dtype, device="cuda")
    x[:, :K] = torch.randn(T, K, generator=g).to(dtype)
    b = torch.randn(F + tail, generator=g).cuda()
    act = F // 2 // 8 * 8
    out = torch.empty(T, F, dtype=dtype, device="cuda")
    tl = torch.empty(T, max(tail, 8), dtype=torch.float32, device="cuda")
    gemm.linear_packed(x[:, :K], w[:, :K], out, bias=b, act_from=act, tail=tl if tail else None)
    y = x.double() @ w.double().T + b.double()
    want = y[:, :F].clone()
    want[:, act:] = torch.relu(want[:, act:]).square()
    _close(out, want, _tol(dtype, 2e-6, 5e-3))
    if tail:
        _close(tl[:, :tail], y[:, F:], 1e-5)
    res = torch.randn(T, F, generator=g).cuda()
    want = res.double() + x.double() @ w[:F].double().T
    gemm.linear_residual_f32(x[:, :K], w[:F, :K], res)
    _close(res, want, 1e-5)
    _ok()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("n,E,top,K,F", [(1, 4, 2, 64, 40), (33, 5, 3, 88, 72), (64, 8, 8, 128, 128),
                                         (300, 3, 1, 96, 136), (700, 9, 4, 64, 64),
                                         (5, 300, 6, 64, 64), (900, 3, 2, 256, 192),
                                         (400, 3, 2, 512, 264)])
def test_routing_and_grouped_products(dt, n, E, top, K, F):
    from easy_to_hard_b200.ops import gemm, hybrid as hy
    dtype = DT[dt]
    g = torch.Generator().manual_seed(n)
    z = torch.randn(n, E, generator=g)
    if E > 2:
        z[:, 1] -= 100                                     # an expert that nobody chooses
    zp = torch.zeros(n, E + 3, device="cuda")
    zp[:, :E] = z
    h = torch.randn(n, K, generator=g).to(dtype).cuda()
    hg = torch.zeros(n * top, K, dtype=dtype, device="cuda")
    off = torch.zeros(E + 1, dtype=torch.int32, device="cuda")
    place, sel = (torch.zeros(n, top, dtype=torch.int32, device="cuda") for _ in range(2))
    w = torch.zeros(n, top, device="cuda")
    hy.moe_route(zp, E, top, h, hg, off, place, w, sel)
    idx, want_w = O.route(z.double(), top)
    _close(w, want_w, 1e-6)
    o = off.tolist()
    assert o[0] == 0 and o[-1] == n * top
    assert [b - a for a, b in zip(o, o[1:])] == torch.bincount(idx.flatten(), minlength=E).tolist()
    pl = place.cpu().long()
    assert sorted(pl.flatten().tolist()) == list(range(n * top))
    assert torch.equal(torch.bucketize(pl, off.cpu()[1:], right=True), idx)
    assert torch.equal(hg[pl.cuda()], h[:, None].expand(-1, top, -1))
    w1, w3 = ((torch.randn(E * F, K, generator=g) / math.sqrt(K)).to(dtype).cuda() for _ in "ab")
    w2 = (torch.randn(E * K, F, generator=g) / math.sqrt(F)).to(dtype).cuda()
    a = torch.full((n * top, F), 7.0, dtype=dtype, device="cuda")
    y = torch.empty(n * top, K, dtype=dtype, device="cuda")
    gemm.grouped_swiglu(hg, w1, w3, a, off, E, n)
    gemm.grouped_linear(a, w2, y, off, E, n)
    for e in range(E):
        rows = hg[o[e]: o[e + 1]].double()
        if len(rows):
            wa = torch.nn.functional.silu(rows @ w1[e * F: (e + 1) * F].double().T) * (
                rows @ w3[e * F: (e + 1) * F].double().T)
            _close(a[o[e]: o[e + 1]], wa, _tol(dtype, 1e-5, 2e-2))
            _close(y[o[e]: o[e + 1]], a[o[e]: o[e + 1]].double() @ w2[e * K: (e + 1) * K]
                   .double().T, _tol(dtype, 1e-5, 1e-2))
    _ok()


class _Attn:
    """One attention layer's kernels on given projections of several sequences."""

    def __init__(self, L, dtype, slots, smax, qn=None, kn=None, eps=1e-5):
        from easy_to_hard_b200.models.hybrid import hybrid_config
        from easy_to_hard_b200.ops import hybrid as hy
        m = self.m = hybrid_config(M.config([L])).layers[0].mixer
        p8 = lambda n: (n + 7) // 8 * 8  # noqa: E731
        self.offs, at = [], 0
        for n in (m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim, m.heads * m.vdim):
            self.offs.append(at)
            at += p8(n)
        self.ld, self.dtype = at, dtype
        # whatever earlier sequences left in the cache must not matter
        self.kc = torch.full((slots, m.kv_heads, smax, p8(m.dim)), 1e4, dtype=dtype, device="cuda")
        self.vc = torch.full((slots, m.kv_heads, smax, p8(m.vdim)), 1e4, dtype=dtype,
                             device="cuda")
        self.kc[..., m.dim:] = 0
        self.vc[..., m.vdim:] = 0
        self.k = hy.WindowAttention(m, self.offs, self.kc, self.vc, m.rot.table(smax, "cuda"),
                                    qn, kn, eps)

    def run(self, parts, slot):
        """parts: list of (position of the first token, projections [n, q | k | v | g]) that
        enter one after the other; single tokens go through the decode kernel."""
        m, outs = self.m, []
        for at, proj in parts:
            n = proj.shape[0]
            act = torch.zeros(n, self.ld, dtype=self.dtype, device="cuda")
            c = 0
            for o, w in zip(self.offs, (m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim,
                                        m.heads * m.vdim)):
                act[:, o: o + w] = proj[:, c: c + w].to(self.dtype)
                c += w
            pos = torch.arange(at, at + n, dtype=torch.int32, device="cuda")
            sl = torch.full((n,), slot, dtype=torch.int32, device="cuda")
            if n == 1:
                self.k.decode(act, pos, sl)
            else:
                self.k.prompt(act, pos, sl, torch.tensor([0, n], dtype=torch.int32,
                                                         device="cuda"), 1, n)
            outs.append(act[:, self.offs[3]: self.offs[3] + m.heads * m.vdim].float().cpu())
        return torch.cat(outs)


def _expected_attention(proj, L, eps, qn, kn):
    """The oracle's mechanisms on given projections."""
    m = L["mixer"]
    H, G, d, e, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], proj.shape[0]
    q, k, v, g = proj.double().split([H * d, G * d, G * e, H * e], 1)
    if qn is not None:
        q, k = O.rms(q, eps) * qn.double(), O.rms(k, eps) * kn.double()
    q, k, v = O.rotate(q.view(T, H, d), m["rot"]), O.rotate(k.view(T, G, d), m["rot"]), \
        v.view(T, G, e)
    ok = O.visible(T, m.get("mask"))
    out = []
    for a in range(H):
        s = (q[:, a] @ k[:, a // (H // G)].T * m["scale"]).masked_fill(~ok, float("-inf"))
        out.append(torch.softmax(s, -1) @ v[:, a // (H // G)])
    return torch.cat(out, -1) * torch.sigmoid(g)


LAYERS = {
    "d40v24": M.attn(6, 3, 40, 24, rot=24, scaling=M.YARN, window=20, keep=3),
    "d128": M.attn(8, 2, 128, 128, window=140, keep=5),
    "d128full": M.attn(4, 4, 128, 128, window=None),
    "d64v128": M.attn(8, 1, 64, 128, rot=32, window=64, keep=0),
    "d14": M.attn(3, 1, 14, 10, rot=6, window=9, keep=2),
    "d200": M.attn(2, 1, 200, 256, rot=40, window=100, keep=17),
    "d56v48": M.attn(6, 2, 56, 48, rot=56, window=150, keep=9),
    "d96v80": M.attn(4, 4, 96, 80, rot=48, scaling=M.YARN, window=31, keep=140),
    "mqa16": M.attn(16, 1, 72, 96, window=130, keep=129),
}


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("name", LAYERS)
def test_attention_prompts_portions_and_decoding(dt, name):
    dtype, L = DT[dt], LAYERS[name]
    m = L["mixer"]
    T = 330
    g = torch.Generator().manual_seed(5)
    nq, nk, nv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
    proj = torch.randn(T, nq + nk + nv + m["heads"] * m["vdim"], generator=g).to(dtype).float()
    qn = 1 + 0.3 * torch.randn(nq, generator=g)
    kn = 1 + 0.3 * torch.randn(nk, generator=g)
    want = _expected_attention(proj, L, 1e-5, qn, kn)
    cuts = {"whole": [0, T], "portions": [0, 2, 37, 39, 168, 296, T],
            "decode": [0, 21] + list(range(22, 60)) + [300] + list(range(301, T + 1))}
    for how, c in cuts.items():
        a = _Attn(L, dtype, 3, 336, qn.cuda(), kn.cuda())
        got = a.run([(lo, proj[lo:hi]) for lo, hi in zip(c, c[1:])], 1)
        _close(got, want, _tol(dtype, 2e-5, 2.5e-2))
        _ok()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("name", ["d40v24", "d128", "d64v128"])
def test_attention_edges_stand_out(dt, name):
    """One key at a time is made to dominate the scores of one query: just inside and just outside
    the window, the last kept token and the next one, the first token, the query itself. The
    output then is that key's value, or does not contain it at all."""
    dtype, L = DT[dt], LAYERS[name]
    m = L["mixer"]
    win, keep = m["mask"]["size"], m["mask"]["keep_first"]
    T = win + 128 + keep + 9
    g = torch.Generator().manual_seed(9)
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    i = T - 3
    cases = {i: True, i - 1: True, i - win + 1: True, i - win: False, i - win - 1: False,
             keep: False, keep + 1: False}
    if keep:
        cases.update({0: True, keep - 1: True})
    for j, seen in cases.items():
        assert bool(O.visible(T, m["mask"])[i, j]) == seen
        proj = 0.3 * torch.randn(T, H * d + G * d + G * e + H * e, generator=g)
        # the rotated query times the rotated key is large: aim the key at the query's direction
        # at their distance, by rotating back through the oracle
        qv = torch.randn(H, d, generator=g)
        for a in range(H):
            qv[a] = qv[a - a % (H // G)]                   # the heads of a group agree
        proj[i, : H * d] = qv.flatten()
        big = torch.zeros(T, G, d, dtype=torch.float64)
        big[i] = qv[:: H // G].double()
        rot = O.rotate(big, m["rot"])[i]
        inv = torch.zeros(T, G, d, dtype=torch.float64)
        inv[j] = rot
        freq, amp = O.rope_frequencies(m["rot"])
        half = len(freq)
        ang = j * torch.tensor(freq, dtype=torch.float64)
        u, v = inv[j][:, :half].clone(), inv[j][:, half:2 * half].clone()
        key = inv[j].clone()
        key[:, :half] = (u * torch.cos(ang) + v * torch.sin(ang)) / amp
        key[:, half:2 * half] = (v * torch.cos(ang) - u * torch.sin(ang)) / amp
        key *= 40 / (m["scale"] * (rot * rot).sum(-1, keepdim=True))
        proj[j, H * d: H * d + G * d] = key.float().flatten()
        proj[j, H * d + G * d: H * d + G * d + G * e] = 5.0
        proj = proj.to(dtype).float()
        want = _expected_attention(proj, L, 1e-5, None, None)
        share = (want[i] / torch.sigmoid(proj[i, -H * e:].double())).mean()
        assert (share > 4.5) == seen                       # the test shows what it should
        for c in ([0, T], [0, i] + list(range(i + 1, T + 1)), [0, 3, i - 1, T]):
            got = _Attn(L, dtype, 2, T).run([(a, proj[a:b]) for a, b in zip(c, c[1:])], 0)
            _close(got[i:], want[i:], _tol(dtype, 1e-4, 3e-2))
    _ok()


def test_attention_rows_of_unequal_sequences():
    """Prompts of several sequences in one launch, then one decode launch for all of them."""
    L = LAYERS["d128"]
    m = L["mixer"]
    g = torch.Generator().manual_seed(2)
    width = sum((m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"],
                 m["heads"] * m["vdim"]))
    lens = [1, 130, 7, 260, 128]
    a = _Attn(L, torch.bfloat16, 6, 272)
    projs = [torch.randn(n + 1, width, generator=g).bfloat16().float() for n in lens]
    slots = [4, 0, 5, 2, 1]

    def i32(x):
        return torch.tensor(x, dtype=torch.int32, device="cuda")
    for phase in ("prompt", "decode"):
        part = [p[:n] if phase == "prompt" else p[n:] for p, n in zip(projs, lens)]
        act = torch.cat(part).bfloat16().cuda()
        ld = [len(x) for x in part]
        pos = i32(sum(([*range(n)] if phase == "prompt" else [n] for n in lens), []))
        slot = i32(sum(([s] * n for s, n in zip(slots, ld)), []))
        if phase == "prompt":
            seg = [sum(ld[:i]) for i in range(len(ld) + 1)]
            a.k.prompt(act, pos, slot, i32(seg), len(ld), max(ld))
        else:
            a.k.decode(act, pos, slot)
        got = act[:, a.offs[3]:].float().cpu().split(ld)
        for x, p, n in zip(got, projs, lens):
            want = _expected_attention(p, L, 1e-5, None, None)
            _close(x, want[:n] if phase == "prompt" else want[n:], 2.5e-2)
    _ok()


class _Gla:
    def __init__(self, H, d, e, tau, rank, dtype, slots=3, seed=0, bias=1.0, spread=1.0):
        from easy_to_hard_b200.models.hybrid import GlaMixer
        from easy_to_hard_b200.ops import hybrid as hy
        g = torch.Generator().manual_seed(seed)
        self.m = GlaMixer(H, d, e, tau, rank)
        p8 = lambda n: (n + 7) // 8 * 8  # noqa: E731
        self.w = (H * d, H * d, H * e, H * e)
        self.offs, at = [], 0
        for n in self.w:
            self.offs.append(at)
            at += p8(n)
        self.ld, self.dtype = at, dtype
        self.a2 = (torch.randn(H * d, rank, generator=g) / math.sqrt(rank)).to(dtype)
        self.b2 = bias + spread * torch.randn(H * d, generator=g)
        self.norm = 1 + 0.2 * torch.randn(e, generator=g)
        # stale values of a slot's former owner
        self.state = torch.full((slots, H, d, (e + 3) // 4 * 4), 1e3, device="cuda")
        self.state[..., e:] = 0
        self.k = hy.GatedLinearAttention(self.m, self.offs, self.state, self.a2.cuda(),
                                         self.b2.cuda(), self.norm.cuda(), 1e-5)

    def run(self, parts, slot):
        outs = []
        for at, proj, a in parts:
            n = proj.shape[0]
            act = torch.zeros(n, self.ld, dtype=self.dtype, device="cuda")
            c = 0
            for o, w in zip(self.offs, self.w):
                act[:, o: o + w] = proj[:, c: c + w].to(self.dtype)
                c += w
            tail = torch.zeros(n, (self.m.rank + 7) // 8 * 8, device="cuda")
            tail[:, : self.m.rank] = a
            pos = torch.arange(at, at + n, dtype=torch.int32, device="cuda")
            sl = torch.full((n,), slot, dtype=torch.int32, device="cuda")
            if n == 1:
                self.k.decode(act, tail, pos, sl)
            else:
                self.k.prompt(act, tail, pos, sl, torch.tensor([0, n], dtype=torch.int32,
                                                               device="cuda"), 1, n)
            outs.append(act[:, self.offs[3]: self.offs[3] + self.w[3]].float().cpu())
        return torch.cat(outs)

    def expected(self, proj, a):
        m, T = self.m, proj.shape[0]
        q, k, v, g = proj.double().split(list(self.w), 1)
        z = a.double() @ self.a2.double().T + self.b2.double()
        al = torch.sigmoid(z).pow(1 / m.tau).view(T, m.heads, m.dim)
        o, S = O.gla_recurrence(q.view(T, m.heads, m.dim) * m.dim ** -0.5,
                                k.view(T, m.heads, m.dim), v.view(T, m.heads, m.vdim), al)
        o = (O.rms(o, 1e-5) * self.norm.double()).reshape(T, -1)
        return o * g * torch.sigmoid(g), S


GLA = {  # heads, dim, vdim, tau, rank, bias, spread of the decay logits
    "small": (3, 24, 40, 4.0, 12, 1.0, 1.0),
    "square": (2, 64, 64, 16.0, 16, 0.0, 1.0),
    "wide": (2, 128, 256, 8.0, 16, 2.0, 1.0),
    "odd": (3, 7, 9, 3.0, 5, 0.0, 1.0),
    "deep": (1, 256, 72, 2.0, 24, 1.0, 2.0),
    "forgets": (2, 64, 64, 1.0, 16, -20.0, 15.0),   # decays from about e^-60 to 1 in one step
    "half": (2, 48, 48, 8.0, 16, 0.0, 1.0),
    "tall": (2, 80, 136, 8.0, 5, 0.0, 1.0),         # decay rank off the vector width
    "flat": (1, 112, 40, 16.0, 20, 1.0, 1.0),
    "thin": (4, 16, 264, 4.0, 16, 0.0, 1.0),
    "edge": (2, 96, 64, 8.0, 16, -5.0, 0.5),        # around the steepest chunk of the fast form
    "keeps": (2, 128, 128, 16.0, 16, 30.0, 0.0),    # nothing decays: the sum over all tokens
}


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("name", GLA)
def test_gated_linear_attention(dt, name):
    dtype = DT[dt]
    H, d, e, tau, rank, bias, spread = GLA[name]
    T = 300
    g = torch.Generator().manual_seed(4)
    proj = torch.randn(T, 2 * H * d + 2 * H * e, generator=g).to(dtype).float()
    a = torch.randn(T, rank, generator=g)
    layer = _Gla(H, d, e, tau, rank, dtype, bias=bias, spread=spread)
    want, S = layer.expected(proj, a)
    for c in ([0, T], [0, 2, 37, 39, 168, 232, T], [0, 63] + list(range(64, 90)) + [T - 30]
              + list(range(T - 29, T + 1))):
        layer.state.fill_(1e3)
        layer.state[..., e:] = 0
        got = layer.run([(lo, proj[lo:hi], a[lo:hi]) for lo, hi in zip(c, c[1:])], 2)
        _close(got, want, _tol(dtype, 5e-5, 2.5e-2))
        st = layer.state[2][..., :e].double().cpu()
        assert float((st - S).abs().max()) <= _tol(dtype, 1e-5, 4e-3) * float(S.abs().max())
    _ok()


@pytest.mark.parametrize("dt", DT)
def test_a_far_token_is_still_in_the_state(dt):
    """One early token writes a value that nothing else writes; without decay it decides the output
    of the last token, through every kind of step."""
    dtype = DT[dt]
    H, d, e, T = 2, 64, 64, 400
    layer = _Gla(H, d, e, 16.0, 16, dtype, bias=30.0, spread=0.0)
    proj = 0.02 * torch.randn(T, 2 * H * (d + e), generator=torch.Generator().manual_seed(3))
    proj[5, H * d: 2 * H * d] = 1.0
    proj[5, 2 * H * d: 2 * H * d + H * e] = torch.linspace(-2, 2, e).repeat(H)
    proj[-1, : H * d] = 1.0
    proj[:, -H * e:] = 1.0
    proj = proj.to(dtype).float()
    want, _ = layer.expected(proj, torch.zeros(T, 16))
    assert float(want[-1].max()) > 1.0
    for c in ([0, T], [0, 6, T - 1, T], [0, 130, 140, T], [0, 2] + list(range(3, 12)) + [T]):
        got = layer.run([(lo, proj[lo:hi], torch.zeros(hi - lo, 16))
                         for lo, hi in zip(c, c[1:])], 0)
        _close(got[-1], want[-1], _tol(dtype, 5e-5, 2e-2))
    _ok()


def test_gla_segments_of_one_launch():
    H, d, e, rank = 2, 64, 96, 16
    layer = _Gla(H, d, e, 4.0, rank, torch.bfloat16, slots=6)
    g = torch.Generator().manual_seed(8)
    lens, slots = [5, 200, 1, 64, 129], [3, 0, 5, 1, 4]
    projs = [torch.randn(n, sum(layer.w), generator=g).bfloat16().float() for n in lens]
    As = [torch.randn(n, rank, generator=g) for n in lens]

    def i32(x):
        return torch.tensor(x, dtype=torch.int32, device="cuda")
    act, tail = torch.cat(projs).bfloat16().cuda(), torch.cat(As).cuda()
    seg = [sum(lens[:i]) for i in range(len(lens) + 1)]
    layer.k.prompt(act, tail, i32(sum(([*range(n)] for n in lens), [])),
                   i32(sum(([s] * n for s, n in zip(slots, lens)), [])), i32(seg), len(lens),
                   max(lens))
    got = act[:, layer.offs[3]:].float().cpu().split(lens)
    for x, p, a, s in zip(got, projs, As, slots):
        want, S = layer.expected(p, a)
        _close(x, want, 2.5e-2)
        _close(layer.state[s], S, 4e-3)
    assert float(layer.state[2][..., :e].min()) == 1e3     # a slot that took no part
    _ok()
