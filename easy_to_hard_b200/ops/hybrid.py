"""Front-ends of the hybrid decoders' kernels: fp32-residual norm, windowed attention over the slot
cache, latent attention, gated linear attention, expert routing. All of them take bf16 or fp32
activations; there is no CPU path."""
from __future__ import annotations

import ctypes as C
from typing import Optional

import numpy as np
import torch

from . import _lib, gemm
from ._lib import AttnWindowParams, FlashWindowArgs, GlaParams, LatentParams, StreamNormParams

N_SM = 148


def _is_bf16(t: torch.Tensor) -> int:
    assert t.dtype in (torch.bfloat16, torch.float32)
    return int(t.dtype == torch.bfloat16)


def stream_norm(x: torch.Tensor, weight: torch.Tensor, out: torch.Tensor, *, eps: float,
                offset: float = 0.0, tokens: Optional[torch.Tensor] = None,
                emb: Optional[torch.Tensor] = None, emb_scale: float = 1.0,
                experts: Optional[tuple] = None, rows: Optional[torch.Tensor] = None,
                col: Optional[torch.Tensor] = None, left_pad: Optional[torch.Tensor] = None,
                pos_out: Optional[torch.Tensor] = None) -> None:
    """out = rmsnorm(row) * (offset + weight) for the fp32 residual ``x`` [n, W].

    ``tokens`` starts the stream (x = emb[token] * emb_scale); ``experts`` = (y, place, weights)
    first adds the expert outputs of the layer before, weighted (or as they are: weights None), to x;
    ``rows`` normalises only
    these rows and leaves x alone. ``col`` / ``left_pad`` / ``pos_out``: positions of a decode
    step."""
    n, W = (rows if rows is not None else x).shape[0], x.shape[1]
    assert x.is_contiguous() and x.dtype == torch.float32 and weight.dtype == torch.float32
    assert out.stride(1) == 1 and out.shape[0] >= n
    p = StreamNormParams()
    p.x, p.W, p.x_rows = x.data_ptr(), W, x.shape[0]
    if tokens is not None:
        assert emb.dtype == out.dtype and tokens.dtype == torch.int32 and rows is None
        p.tokens, p.emb, p.lde = tokens.data_ptr(), emb.data_ptr(), emb.stride(0)
        p.vocab, p.emb_scale = emb.shape[0], emb_scale
    if experts is not None:
        y, place, w = experts
        assert y.dtype == out.dtype and place.dtype == torch.int32
        assert w is None or w.dtype == torch.float32
        p.y, p.ldy, p.y_rows = y.data_ptr(), y.stride(0), y.shape[0]
        p.place, p.ew, p.top = place.data_ptr(), _lib.ptr(w), place.shape[1]
    if rows is not None:
        p.rows = rows.data_ptr()
    if col is not None:
        p.col, p.left_pad, p.pos_out = col.data_ptr(), _lib.ptr(left_pad), pos_out.data_ptr()
    p.weight, p.offset, p.eps = weight.data_ptr(), offset, eps
    p.out, p.ldo = out.data_ptr(), out.stride(0)
    p.status = _lib.status_word(x.device).data_ptr()
    _lib.check(_lib.lib().e2h_stream_norm(C.byref(p), n, _is_bf16(out), _lib.stream()),
               "stream_norm")


def window_splits(n: int, heads: int, kv_heads: int, keys: int) -> int:
    """CTAs that share one (token, kv head) of ``attn_window``: enough to fill the SMs a few times
    over, while each still has some 64 keys."""
    per_g = heads // kv_heads
    ctas = n * kv_heads * -(-per_g // 8)
    s = 1
    while s < 8 and ctas * s * 2 <= N_SM * 4 and keys // (s * 2) >= 64:
        s *= 2
    return s


class WindowAttention:
    """Attention of one layer over the slot cache. ``act`` is the packed activation, ``offs`` the
    columns of q, k, v and the gate; ``qn`` / ``kn`` are the norm weights over the whole
    projections (or None)."""

    # shortest longest-segment for which the 128-query tensor-core tiles pay
    TENSOR_CORE_TOKENS = 24

    def __init__(self, mixer, offs, kcache, vcache, rot_table, qn, kn, eps: float):
        self.m, self.kc, self.vc = mixer, kcache, vcache
        self._held = (rot_table, qn, kn)     # the kernels keep raw addresses
        self.keys = kcache.shape[2] if not mixer.window else min(kcache.shape[2],
                                                                mixer.window + mixer.keep)
        p = self.p = AttnWindowParams()
        p.off_q, p.off_k, p.off_v, p.off_g = offs
        p.kc, p.vc = kcache.data_ptr(), vcache.data_ptr()
        p.slots, p.smax, p.dimp, p.vdimp = (kcache.shape[0], kcache.shape[2], kcache.shape[3],
                                            vcache.shape[3])
        p.H, p.G, p.dim, p.vdim = mixer.heads, mixer.kv_heads, mixer.dim, mixer.vdim
        assert rot_table.dtype == torch.float32 and rot_table.is_contiguous()
        assert rot_table.shape[0] >= p.smax and rot_table.shape[1] * 2 == mixer.rot.dims
        p.rot, p.rot_table = mixer.rot.dims, rot_table.data_ptr()
        p.scale, p.window, p.keep = mixer.scale, mixer.window, mixer.keep
        p.qn, p.kn, p.eps = _lib.ptr(qn), _lib.ptr(kn), eps
        p.status = _lib.status_word(kcache.device).data_ptr()

    def _bind(self, act, pos, slot):
        p = self.p
        assert act.dtype == self.kc.dtype and act.stride(1) == 1
        p.act, p.ld, p.n = act.data_ptr(), act.stride(0), act.shape[0]
        p.pos, p.slot = pos.data_ptr(), slot.data_ptr()
        return p

    def decode(self, act, pos, slot) -> None:
        """One token per sequence: norms, rotation, cache write, attention and gate."""
        p = self._bind(act, pos, slot)
        p.splits = window_splits(p.n, p.H, p.G, self.keys)
        _lib.check(_lib.lib().e2h_attn_window(C.byref(p), 1, _is_bf16(act), _lib.stream()),
                   "attn_window")

    def prep(self, act, pos, slot) -> None:
        p = self._bind(act, pos, slot)
        p.splits = 1
        _lib.check(_lib.lib().e2h_attn_prep(C.byref(p), _is_bf16(act), _lib.stream()),
                   "attn_prep")

    def prompt(self, act, pos, slot, seg, n_seg: int, seg_max: int) -> int:
        """Tokens seg[s] .. seg[s + 1] continue one sequence each. Returns the launches."""
        self.prep(act, pos, slot)
        self.attend(act, pos, slot, seg, n_seg, seg_max)
        return 2

    def attend(self, act, pos, slot, seg, n_seg: int, seg_max: int) -> None:
        """The second half of ``prompt``: attention and gate of tokens that are in the cache."""
        p = self._bind(act, pos, slot)
        if (act.dtype == torch.bfloat16 and seg_max >= self.TENSOR_CORE_TOKENS
                and p.dim % 8 == 0 and p.vdim % 8 == 0 and p.dim <= 128 and p.vdim <= 128):
            f = FlashWindowArgs()
            f.act, f.ld, f.off_q, f.q_head, f.off_g = p.act, p.ld, p.off_q, p.dim, p.off_g
            f.k, f.ld_k, f.v, f.ld_v = p.kc, p.dimp, p.vc, p.vdimp
            f.k_head, f.v_head = p.smax * p.dimp, p.smax * p.vdimp
            f.k_slot, f.v_slot = p.G * f.k_head, p.G * f.v_head
            f.rows, f.slots, f.smax = p.smax, p.slots, p.smax
            f.seg, f.n_seg, f.seg_max = seg.data_ptr(), n_seg, seg_max
            f.pos, f.slot, f.n = p.pos, p.slot, p.n
            f.H, f.G, f.dim, f.vdim = p.H, p.G, p.dim, p.vdim
            f.scale, f.window, f.keep, f.status = p.scale, p.window, p.keep, p.status
            _lib.check(_lib.lib().e2h_flash_window(C.byref(f), _lib.stream()), "flash_window")
        else:
            self.from_cache(act, pos, slot)

    def from_cache(self, act, pos, slot) -> None:
        """Attention of tokens that ``prep`` has put into the cache."""
        p = self._bind(act, pos, slot)
        p.splits = window_splits(p.n, p.H, p.G, self.keys)
        _lib.check(_lib.lib().e2h_attn_window(C.byref(p), 0, _is_bf16(act), _lib.stream()),
                   "attn_window")


class LatentContext:
    """What latent attention needs to know about the segments of a packed forward. Segments of at
    least ``LatentAttention.TENSOR_CORE_TOKENS`` tokens come first (``n_long`` tokens in
    ``n_long_seg`` segments, the longest of ``seg_max``): their keys and values are expanded per
    head, in a buffer of ``n_ctx`` rows that holds, segment after segment, the positions from the
    oldest one that any layer looks at to the newest. ``src`` / ``pos`` / ``slot`` describe these
    rows (token of this forward, or -1 for a position that the cache holds), ``shift`` [segments] is
    row - position."""

    def __init__(self, lengths, starts, slots, window: int, expand: bool, device):
        """Host lists per segment, in the order of the packed tokens: tokens, first position, cache
        slot. ``window``: the widest of the layers (0: unlimited)."""
        self.n_long = self.n_long_seg = self.seg_max = self.n_ctx = 0
        self.src = self.pos = self.slot = self.shift = None
        src, pos, slot, shift = [], [], [], []
        for n, p0, s in zip(lengths, starts, slots):
            lo = max(p0 - window + 1, 0) if window else 0
            if not expand or not LatentAttention.expands(n, p0 - lo):
                break
            shift.append(self.n_ctx - lo)
            src += [np.full(p0 - lo, -1), np.arange(self.n_long, self.n_long + n)]
            pos.append(np.arange(lo, p0 + n))
            slot.append(np.full(p0 + n - lo, s))
            self.n_long += n
            self.n_ctx += p0 + n - lo
            self.n_long_seg += 1
            self.seg_max = max(self.seg_max, n)
        if src:
            m = self.n_ctx
            d = np.concatenate(src + pos + slot + [shift]).astype(np.int32)
            self.src, self.pos, self.slot, self.shift = torch.from_numpy(d).to(device).split(
                [m, m, m, len(shift)])


class LatentAttention:
    """Latent attention of one layer over the slot cache (``[slots, positions, rank + rot]``).
    ``act`` is the packed activation: q head by head [dim | rot], [latent | shared key part], gate
    (columns ``offs`` = q, latent, gate). Head sizes are padded to multiples of 8 with zeros.
    ``w_kv`` [H * (dim + vdim), rank]: key and value expansion; ``w_uk_t`` [H * rank, dim]: the key
    expansion transposed per head, which absorbs it into the queries."""

    # shortest segment whose keys and values are expanded for the tensor-core prompt kernel, and how
    # many earlier positions per token it may bring along
    TENSOR_CORE_TOKENS, HISTORY = 24, 8

    def __init__(self, mixer, offs, cache, rot_table, w_kv, w_uk_t, norm, eps: float):
        self.m, self.cache = mixer, cache
        self._held = (rot_table, norm)           # the kernels keep raw addresses
        self.w_kv, self.w_uk_t = w_kv, w_uk_t
        p = self.p = LatentParams()
        p.off_q, p.off_c, self.off_g = offs
        self.dim, self.rot, self.vdim, self.rank = (
            -(-n // 8) * 8 for n in (mixer.dim, mixer.rot_dim, mixer.vdim, mixer.kv_rank))
        p.H, p.dim, p.rot, p.rank, p.rank_n = (mixer.heads, self.dim, self.rot, self.rank,
                                               mixer.kv_rank)
        p.cache, p.slots, p.smax = cache.data_ptr(), cache.shape[0], cache.shape[1]
        assert cache.shape[2] == self.rank + self.rot and cache.is_contiguous()
        assert rot_table.dtype == torch.float32 and rot_table.is_contiguous()
        assert rot_table.shape[0] >= p.smax and rot_table.shape[1] * 2 == self.rot
        assert norm.dtype == torch.float32 and norm.numel() == self.rank
        p.rot_table, p.norm, p.eps, p.scale = rot_table.data_ptr(), norm.data_ptr(), eps, mixer.scale
        p.window = mixer.window
        p.status = _lib.status_word(cache.device).data_ptr()
        bf = cache.dtype == torch.bfloat16
        # the kernel with the decode work fused in, and the tensor-core prompt kernel
        self.fused = bf and self.rank <= 512 and self.rank + self.rot <= 576
        self.can_expand = self.expandable(mixer, cache.dtype)

    @staticmethod
    def expandable(mixer, dtype) -> bool:
        return (dtype == torch.bfloat16 and mixer.dim <= 128 and mixer.rot_dim <= 64
                and mixer.vdim <= 128)

    @classmethod
    def expands(cls, tokens: int, history: int) -> bool:
        return tokens >= cls.TENSOR_CORE_TOKENS and history <= cls.HISTORY * tokens

    def _bind(self, act, pos, slot, n_long=0):
        p = self.p
        assert act.dtype == self.cache.dtype and act.stride(1) == 1
        p.act, p.ld, p.n, p.n_long = act.data_ptr(), act.stride(0), act.shape[0], n_long
        p.pos, p.slot = pos.data_ptr(), slot.data_ptr()
        return p

    def splits(self, n: int) -> int:
        """CTAs that share one token: enough to fill the SMs, each with some 64 keys at least."""
        if not self.fused:
            return 1
        keys = min(self.p.window or self.p.smax, self.p.smax)
        ctas = n * -(-self.p.H // (16 if self.p.H <= 16 else 32))
        s = 1
        while s < 8 and ctas * s * 2 <= N_SM and keys // (s * 2) >= 64:
            s *= 2
        return s

    def absorb(self, act, ql) -> None:
        """ql_h = W_uk,h^T q_h for every token of ``act``."""
        gemm.batched_linear(act[:, self.p.off_q:], self.w_uk_t, ql, batch=self.p.H, k=self.dim,
                            x_step=self.dim + self.rot, out_step=self.rank)

    def attend(self, act, ql, ol, pos, slot, n_long: int = 0, fused: bool = False) -> None:
        p = self._bind(act, pos, slot, n_long)
        p.ql, p.ol, p.splits = ql.data_ptr(), ol.data_ptr(), self.splits(p.n - n_long)
        _lib.check(_lib.lib().e2h_latent_attn(C.byref(p), int(fused), _is_bf16(act),
                                              _lib.stream()), "latent_attn")

    def values(self, act, ol) -> None:
        """gate columns = (W_uv,h ol_h) * sigmoid(gate)."""
        gemm.batched_linear(ol, self.w_kv[self.p.H * self.dim:], act[:, self.off_g:],
                            batch=self.p.H, k=self.rank, x_step=self.rank, out_step=self.vdim,
                            gate=True)

    def prep(self, act, pos, slot, ctx: LatentContext, rows=None) -> None:
        p = self._bind(act, pos, slot, ctx.n_long)
        p.n_ctx = ctx.n_ctx
        if rows is not None:
            p.ctx = rows.data_ptr()
            p.ctx_src, p.ctx_pos, p.ctx_slot = (t.data_ptr() for t in (ctx.src, ctx.pos, ctx.slot))
        _lib.check(_lib.lib().e2h_latent_prep(C.byref(p), _is_bf16(act), _lib.stream()),
                   "latent_prep")

    def expand(self, rows, kv) -> None:
        """Keys [H x dim] and values [H x vdim] of the context rows."""
        gemm.linear_rows(rows[:, : self.rank], self.w_kv, kv)

    def flash(self, act, pos, slot, seg, ctx: LatentContext, rows, kv) -> None:
        p = self._bind(act, pos, slot)
        f = FlashWindowArgs()
        f.act, f.ld, f.off_q, f.q_head, f.off_g = (p.act, p.ld, p.off_q, self.dim + self.rot,
                                                   self.off_g)
        f.k, f.ld_k, f.k_head, f.k_slot = kv.data_ptr(), kv.stride(0), self.dim, kv.numel()
        f.v, f.ld_v, f.v_head, f.v_slot = (kv[:, p.H * self.dim:].data_ptr(), kv.stride(0),
                                           self.vdim, kv.numel())
        f.k2, f.ld_k2 = rows[:, self.rank:].data_ptr(), rows.stride(0)
        f.rows, f.slots, f.smax, f.shift = kv.shape[0], 1, p.smax, ctx.shift.data_ptr()
        f.seg, f.n_seg, f.seg_max = seg.data_ptr(), ctx.n_long_seg, ctx.seg_max
        f.pos, f.slot, f.n = p.pos, p.slot, p.n
        f.H = f.G = p.H
        f.dim, f.dim2, f.vdim = self.dim, self.rot, self.vdim
        f.scale, f.window, f.keep, f.status = p.scale, p.window, 0, p.status
        _lib.check(_lib.lib().e2h_flash_window(C.byref(f), _lib.stream()), "flash_window")

    def _absorbed(self, act, n: int):
        return (torch.empty(n, self.p.H * self.rank, dtype=act.dtype, device=act.device)
                for _ in "qo")

    def decode(self, act, pos, slot, ql=None, ol=None) -> int:
        """One token per sequence. Returns the launches."""
        if ql is None:
            ql, ol = self._absorbed(act, act.shape[0])
        if not self.fused:
            self.prep(act, pos, slot, _NO_CONTEXT)
        self.absorb(act, ql)
        self.attend(act, ql, ol, pos, slot, fused=self.fused)
        self.values(act, ol)
        return 3 if self.fused else 4

    def prompt(self, act, pos, slot, seg, ctx: LatentContext) -> int:
        """Tokens seg[s] .. seg[s + 1] continue one sequence each. Returns the launches."""
        rows, k = None, 1
        if ctx.n_ctx:
            rows = torch.empty(ctx.n_ctx, self.rank + self.rot, dtype=act.dtype, device=act.device)
        self.prep(act, pos, slot, ctx, rows)
        if ctx.n_ctx:
            kv = torch.empty(ctx.n_ctx, self.w_kv.shape[0], dtype=act.dtype, device=act.device)
            self.expand(rows, kv)
            self.flash(act, pos, slot, seg, ctx, rows, kv)
            k += 2
        n = act.shape[0] - ctx.n_long
        if n:
            ql, ol = self._absorbed(act, n)
            rest = act[ctx.n_long:]
            self.absorb(rest, ql)
            self.attend(act, ql, ol, pos, slot, n_long=ctx.n_long)
            self.values(rest, ol)
            k += 3
        return k


_NO_CONTEXT = LatentContext((), (), (), 0, False, None)


class GatedLinearAttention:
    """Gated linear attention of one layer over the slot states."""

    # shortest longest-segment for which the chunked tensor-core form pays
    CHUNK_TOKENS = 48

    def __init__(self, mixer, offs, state, a2, a2_b, norm, eps: float):
        self.m, self.state, self.a2 = mixer, state, a2
        self._held = (a2_b, norm)            # the kernels keep raw addresses
        p = self.p = GlaParams()
        p.off_q, p.off_k, p.off_v, p.off_g = offs
        p.r, p.w2, p.ldw, p.b2 = a2.shape[1], a2.data_ptr(), a2.stride(0), a2_b.data_ptr()
        p.inv_tau, p.qscale, p.eps = 1.0 / mixer.tau, mixer.dim ** -0.5, eps
        p.norm, p.state = norm.data_ptr(), state.data_ptr()
        p.slots, p.H, p.dim, p.vdim, p.vp = (state.shape[0], mixer.heads, mixer.dim, mixer.vdim,
                                             state.shape[3])
        p.status = _lib.status_word(state.device).data_ptr()

    def _bind(self, act, tail, pos, slot):
        p = self.p
        assert act.dtype == self.a2.dtype and tail.dtype == torch.float32
        p.act, p.ld, p.n = act.data_ptr(), act.stride(0), act.shape[0]
        p.a, p.lda = tail.data_ptr(), tail.stride(0)
        p.pos, p.slot = pos.data_ptr(), slot.data_ptr()
        return p

    def decode(self, act, tail, pos, slot) -> None:
        p = self._bind(act, tail, pos, slot)
        s = 1
        while s < 8 and (p.n * p.H * s * 2 <= N_SM * 4 and p.vp // (s * 2) >= 32
                         or p.vp // s > 1024):
            s *= 2
        p.splits = s
        _lib.check(_lib.lib().e2h_gla_step(C.byref(p), _is_bf16(act), _lib.stream()), "gla_step")

    def prompt(self, act, tail, pos, slot, seg, n_seg: int, seg_max: int) -> int:
        """Tokens seg[s] .. seg[s + 1] continue one sequence each. Returns the launches."""
        p = self._bind(act, tail, pos, slot)
        n = p.n

        def buf(*shape, dtype=torch.float32):
            return torch.empty(*shape, dtype=dtype, device=act.device)
        o = buf(n, p.H * p.vdim)
        p.o = o.data_ptr()
        p.seg, p.n_seg, p.seg_max = seg.data_ptr(), n_seg, seg_max
        lib, bf, s = _lib.lib(), _is_bf16(act), _lib.stream()
        if (bf and seg_max >= self.CHUNK_TOKENS and p.dim % 16 == 0 and p.dim <= 128
                and p.vdim % 8 == 0 and p.r <= 128):
            p.chunks = n // 64 + n_seg + 1
            cq, ck = (buf(2, p.chunks, p.H, 64, p.dim, dtype=torch.bfloat16) for _ in "qk")
            ca = buf(2, p.chunks, p.H, 64, 64, dtype=torch.bfloat16)
            cg = buf(p.chunks, p.H, p.dim)
            p.cq, p.ck, p.ca, p.cg = (t.data_ptr() for t in (cq, ck, ca, cg))
            _lib.check(lib.e2h_gla_chunk(C.byref(p), s), "gla_chunk")
            _lib.check(lib.e2h_gla_out(C.byref(p), bf, s), "gla_out")
            return 3
        logdec = buf(n, p.H * p.dim)
        p.logdec = logdec.data_ptr()
        _lib.check(lib.e2h_gla_decay(C.byref(p), bf, s), "gla_decay")
        _lib.check(lib.e2h_gla_scan(C.byref(p), bf, s), "gla_scan")
        _lib.check(lib.e2h_gla_out(C.byref(p), bf, s), "gla_out")
        return 3


ROUTER_SCORES = {"softmax": 0, "sigmoid": 1}


def moe_route(logits: torch.Tensor, experts: int, top: int, h: torch.Tensor, hg: torch.Tensor,
              off: torch.Tensor, place: torch.Tensor, weights: torch.Tensor,
              sel: torch.Tensor, score: str = "softmax", weight_input: bool = False) -> int:
    """Top-``top`` routing of fp32 ``logits`` [n, >= experts]: ``weights`` / ``place`` [n, top]
    (softmax over the chosen logits or the ``sigmoid`` of each; row of ``hg`` that holds the token
    for that choice), ``off`` [experts + 1] (rows of every expert), ``hg`` [n * top, W] (h regrouped
    by expert, times its weight if ``weight_input``)."""
    n = h.shape[0]
    assert logits.dtype == torch.float32 and hg.dtype == h.dtype and hg.shape[0] >= n * top
    assert off.numel() > experts and sel.numel() >= n * top
    _lib.check(_lib.lib().e2h_moe_route(
        logits.data_ptr(), logits.stride(0), n, experts, top, ROUTER_SCORES[score],
        int(weight_input), h.data_ptr(), h.stride(0),
        h.shape[1], hg.data_ptr(), hg.stride(0), off.data_ptr(), place.data_ptr(),
        weights.data_ptr(), sel.data_ptr(), _is_bf16(h), _lib.stream()), "moe_route")
    return 1 if n * top <= 1024 and n <= 256 else 3
