"""Engine of the hybrid decoders (``models.hybrid``): one forward over a packed list of tokens that
serves prompts, portions of prompts, single decode steps and mixtures of them.

Tokens of all sequences lie one after the other (no padding); per-token positions and cache slots
live on the device, so that the same captured decode step serves rows of unequal length. In a packed
forward the longer pieces come first. Per layer, with the parallel block (mixer and feed-forward read
one norm):

    norm of the fp32 residual            (first adds the expert outputs of the layer before)
    w_in GEMM: q, k, v, gate, activated up projection; fp32 tail: decay input, router logits
    mixer, in place in the packed activation
        decode:  one kernel (norms, rotation, cache write, attention, gate) or (decay, state
                 update, output, norm, gate)
        prompts: attention over the slot cache, or the recurrence by segments
    w_out GEMM: residual += [gated heads, up] w_out^T
    experts: route + regroup, grouped SwiGLU GEMM, grouped down GEMM

A decode step is 4 kernels per dense layer and 7 per expert layer. A sequential block (the feed-forward
has a norm of its own) takes w_in without the feed-forward, then

    norm of the residual
    w_ff GEMM: activated up projection (dense, or the shared expert); fp32 tail: router logits
    w_down GEMM: residual += up w_down^T
    experts: route + regroup (rows weighted), grouped up GEMM + activation, grouped down GEMM

and latent attention is three kernels in a decode step (queries absorb the key expansion; norm,
rotation, cache write and attention over the latents; value expansion and gate), in prompts norm and
rotation, the expansion of keys and values, and flash attention.
"""
from __future__ import annotations

from typing import Dict, Hashable, List, Optional, Sequence, Tuple

import numpy as np
import torch

from ..ops import gemm, hybrid as hy
from .engine import GenerationEngine
from .hybrid import HybridLM, pad8
from .slot_cache import SlotCache

# most tokens of one packed forward: longer prompt batches are cut into portions
MAX_FORWARD_TOKENS = 32768


class _Scratch:
    """Activation buffers for up to ``n`` tokens."""

    def __init__(self, model: HybridLM, n: int):
        cfg, dev, dt = model.config, model.device, model.dtype

        def buf(rows, cols, dtype=dt):
            return torch.zeros(rows, max(cols, 8), dtype=dtype, device=dev)
        blocks = list(model.layers)
        self.n = n
        self.x = torch.empty(n, cfg.dim, dtype=torch.float32, device=dev)
        self.h = buf(n, pad8(cfg.dim))
        self._act = torch.empty(n * max([b.f_main for b in blocks] or [8]), dtype=dt, device=dev)
        self._ff = torch.empty(n * max([b.f_ff for b in blocks] or [8]), dtype=dt, device=dev)
        self._tail = torch.empty(n * max([max(b.n_tail, b.n_ff_tail) for b in blocks] + [8]),
                                 dtype=torch.float32, device=dev)
        moe = [b for b in blocks if b.layer.mlp is not None and b.layer.mlp.kind == "moe"]
        if moe:
            top = max(b.layer.mlp.top for b in moe)
            self.hg = buf(n * top, pad8(cfg.dim))
            self._ag = torch.empty(n * max(b.layer.mlp.top * b.ffp for b in moe), dtype=dt,
                                   device=dev)
            self.y = buf(n * top, pad8(cfg.dim))
            self.off = torch.zeros(max(b.layer.mlp.experts for b in moe) + 1, dtype=torch.int32,
                                   device=dev)
            self._place = torch.zeros(n * top, dtype=torch.int32, device=dev)
            self._ew = torch.zeros(n * top, dtype=torch.float32, device=dev)
            self.sel = torch.zeros(n * top, dtype=torch.int32, device=dev)

    def act(self, n, cols):
        return self._act[: n * cols].view(n, cols)

    def ff(self, n, cols):
        return self._ff[: n * cols].view(n, cols)

    def tail(self, n, cols):
        return self._tail[: n * cols].view(n, cols) if cols else None

    def ag(self, rows, cols):
        return self._ag[: rows * cols].view(rows, cols)

    def choice(self, n, top):
        return self._place[: n * top].view(n, top), self._ew[: n * top].view(n, top)


def _positions(lengths, starts, slots):
    """Position and cache slot of every packed token."""
    return (np.concatenate([np.arange(a, a + n) for n, a in zip(lengths, starts)]),
            np.repeat(slots, lengths))


class HybridEngine(GenerationEngine):
    def __init__(self, model: HybridLM, max_batch_size: int, max_seq_length: int,
                 reduce: str = "auto", use_graph: bool = True, use_pdl: bool = True):
        if reduce not in ("auto", "local"):
            raise ValueError("hybrid decoders run on one GPU: no tensor-parallel reduce")
        self._init_loop(model, model.device, max_batch_size, max_seq_length, use_graph, use_pdl)
        cfg, dev = model.config, self.dev
        self.vocab = cfg.vocab_size
        self.eps = cfg.norm_eps
        self.cache = SlotCache(cfg.layers, self.B, self.S, dev, model.dtype)
        tables: Dict[str, torch.Tensor] = {}
        self.mixers = []
        for blk, store in zip(model.layers, self.cache.layers):
            m = blk.layer.mixer
            if m.kind == "gla":
                self.mixers.append(hy.GatedLinearAttention(
                    m, (blk.off_q, blk.off_k, blk.off_v, blk.off_g), store[0], blk.a2, blk.a2_b,
                    blk.o_norm, self.eps))
                continue
            pairs = m.rot.dims // 2 if m.kind == "attention" else pad8(m.rot_dim) // 2
            key = repr((m.rot, pairs))
            if key not in tables:
                tables[key] = m.rot.table(self.S, dev, pairs).contiguous()
            if m.kind == "attention":
                self.mixers.append(hy.WindowAttention(
                    m, (blk.off_q, blk.off_k, blk.off_v, blk.off_g), *store, tables[key],
                    blk.q_norm, blk.k_norm, self.eps))
            else:
                self.mixers.append(hy.LatentAttention(
                    m, (blk.off_q, blk.off_c, blk.off_g), store[0], tables[key], blk.w_kv,
                    blk.w_uk_t, blk.c_norm, self.eps))
        lat = [x for x in self.mixers if isinstance(x, hy.LatentAttention)]
        self._latent = None
        if lat:     # how prompt segments are served: widest window, whether keys are expanded
            windows = [x.m.window for x in lat]
            self._latent = (0 if 0 in windows else max(windows), all(x.can_expand for x in lat))
            wide = max(x.p.H * x.rank for x in lat)
            self._absorbed = [torch.empty(self.B * wide, dtype=model.dtype, device=dev)
                              for _ in "qo"]
        self.slot = torch.zeros(self.B, dtype=torch.int32, device=dev)
        self.tok_pos = torch.zeros(self.B, dtype=torch.int32, device=dev)
        self.logits = torch.zeros(self.B, pad8(self.vocab), dtype=torch.float32, device=dev)
        self.hf = torch.zeros(self.B, pad8(cfg.dim), dtype=model.dtype, device=dev)
        self._scratch = _Scratch(model, self.B)
        self._rows: List[Hashable] = []
        self.layer_trace: Optional[list] = None    # a list collects the residual after each layer

    # ------------------------------------------------------------------ forward
    def _forward(self, w: _Scratch, n: int, tokens, pos, slot, *, seg=None, ctx=None, rows=None,
                 decode_counters: bool = False, hf=None, logits=None) -> None:
        """Runs ``n`` packed tokens through all layers. ``seg`` = (device offsets, segments,
        longest segment), or None when every token is the next one of its own sequence; ``ctx``: the
        segments' ``LatentContext``. ``rows`` (int32, None: all) are the tokens whose ``logits`` are
        computed."""
        m, cfg = self.model, self.model.config
        W = cfg.dim
        x, h = w.x[:n], w.h[:n]
        pending = None
        start = dict(tokens=tokens, emb=m.embed, emb_scale=cfg.embed_scale)
        if decode_counters:
            start.update(col=self.pos, left_pad=self.left_pad, pos_out=pos)
        for blk, mix in zip(m.layers, self.mixers):
            f = blk.layer.mlp
            hy.stream_norm(x, blk.norm1, h, eps=self.eps, offset=cfg.norm_offset,
                           experts=pending, **start)
            if self.layer_trace is not None and not start:
                self.layer_trace.append(x.clone())
            start, pending = {}, None
            act = w.act(n, blk.f_main)
            tail = w.tail(n, blk.n_tail)
            hw = h[:, :W]
            dense = dict(act=blk.act) if blk.act else {}
            self._count(1 + gemm.linear_packed(
                hw, blk.mat("w_in"), act, bias=blk.b_in, tail=tail,
                **(dict(dense, act_from=blk.off_u) if cfg.parallel and dense else {})))
            kind = blk.layer.mixer.kind
            if kind == "latent":
                if seg is None:
                    self._count(mix.decode(act, pos, slot, *self._absorbed_rows(mix, n)))
                else:
                    self._count(mix.prompt(act, pos, slot, seg[0], ctx))
            elif kind == "attention":
                if seg is None:
                    mix.decode(act, pos, slot)
                    self._count(1)
                else:
                    self._count(mix.prompt(act, pos, slot, *seg))
            elif seg is None:
                mix.decode(act, tail, pos, slot)
                self._count(1)
            else:
                self._count(mix.prompt(act, tail, pos, slot, *seg))
            gemm.linear_residual_f32(act[:, blk.off_g:], blk.mat("w_out"), x)
            self._count(1)
            if not cfg.parallel and f is not None:
                hy.stream_norm(x, blk.norm2, h, eps=self.eps, offset=cfg.norm_offset)
                tail = w.tail(n, blk.n_ff_tail)
                up = w.ff(n, blk.f_ff) if dense else None
                self._count(1 + gemm.linear_packed(hw, blk.mat("w_ff"), up, bias=blk.b_ff,
                                                   tail=tail, act_from=0, **dense))
                if dense:
                    gemm.linear_residual_f32(up, blk.mat("w_down"), x)
                    self._count(1)
            if f is not None and f.kind == "moe":
                pending = self._experts(w, blk, n, hw, tail)
        if rows is None:
            rows_n = n
        else:
            rows_n = rows.shape[0]
        if rows_n:
            hy.stream_norm(x, m.norm, hf[:rows_n], eps=self.eps, offset=cfg.norm_offset,
                           experts=pending, rows=rows, **start)
            gemm.linear_f32_out(hf[:rows_n, :W], m.head_w[:, :W], logits[:rows_n],
                                scale=cfg.logit_scale, softcap=cfg.logit_softcap)
            self._count(2)
        if self.layer_trace is not None:
            last = x.clone()
            if pending is not None and rows is not None:   # not yet added to the residual
                y, place, ew = pending
                y = y.float()[place.long()][..., :W]
                last += (y if ew is None else y * ew[..., None]).sum(1)
            self.layer_trace.append(last)

    def _experts(self, w: _Scratch, blk, n: int, hw, tail):
        f, W = blk.layer.mlp, self.model.config.dim
        place, ew = w.choice(n, f.top)
        k = hy.moe_route(tail[:, blk.off_r:], f.experts, f.top, hw, w.hg[: n * f.top, :W], w.off,
                         place, ew, w.sel, score=f.score, weight_input=f.weight_input)
        hg, ag, y = w.hg[: n * f.top, :W], w.ag(n * f.top, blk.ffp), w.y[: n * f.top, :W]
        if f.gated:
            gemm.grouped_swiglu(hg, blk.mat("e_gate"), blk.mat("e_up"), ag, w.off, f.experts, n)
        else:
            gemm.grouped_linear(hg, blk.mat("e_up"), ag, w.off, f.experts, n, act=f.act)
        gemm.grouped_linear(ag, blk.mat("e_down"), y, w.off, f.experts, n)
        self._count(k + 2)
        return y, place, None if f.weight_input else ew

    def _absorbed_rows(self, mix, n: int):
        """Absorbed queries and attended latents of ``n`` decode tokens."""
        if n > self.B:
            return ()
        cols = mix.p.H * mix.rank
        return (t[: n * cols].view(n, cols) for t in self._absorbed)

    def _upload(self, *parts):
        """int32 host sequences as slices of one device tensor."""
        host = np.concatenate([np.asarray(p, dtype=np.int32) for p in parts])
        return torch.from_numpy(host).to(self.dev).split([len(p) for p in parts])

    def _context(self, lengths, starts, slots) -> Optional[hy.LatentContext]:
        if self._latent is None:
            return None
        window, expand = self._latent
        return hy.LatentContext(lengths, starts, slots, window, expand, self.dev)

    # ------------------------------------------------------------------ steps over sequences
    def open(self, key: Hashable) -> None:
        """Starts a sequence (takes a cache slot)."""
        self.cache.open(key)

    def close(self, key: Hashable) -> None:
        """Ends a sequence; its slot goes to the next one that opens."""
        self.cache.close(key)

    @torch.no_grad()
    def step(self, entries: Sequence[Tuple[Hashable, Sequence[int], Sequence[int]]]
             ) -> torch.Tensor:
        """Runs the next tokens of open sequences. ``entries``: (key, token ids, places among
        these tokens whose logits are wanted). Returns the wanted logits, fp32 [wanted, vocab], in
        the order of the entries and places."""
        toks, seg = [], [0]
        first: Dict[int, int] = {}       # entry -> its first packed token
        starts, slots = [], []
        keys = [k for k, _, _ in entries]
        if len(set(keys)) != len(keys):
            raise ValueError("a sequence may appear once per step")
        if sum(len(t) for _, t, _ in entries) > MAX_FORWARD_TOKENS:
            return self._step_portions(entries)
        for i in sorted(range(len(entries)), key=lambda i: -len(entries[i][1])):
            key, ids, want = entries[i]
            if any(not 0 <= int(j) < len(ids) for j in want):
                raise ValueError("a wanted place lies outside the tokens of its entry")
            if not len(ids):
                continue
            at = self.cache.extend(key, len(ids))
            first[i] = len(toks)
            starts.append(at)
            slots.append(self.cache.slot(key))
            toks += [int(t) for t in ids]
            seg.append(len(toks))
        rows = [first[i] + int(j) for i, (_, _, want) in enumerate(entries) for j in want]
        n = len(toks)
        out = torch.empty(len(rows), self.vocab, dtype=torch.float32, device=self.dev)
        if n == 0:
            return out
        if min(toks) < 0 or max(toks) >= self.vocab:
            raise ValueError("token id outside the vocabulary")
        lengths = [b - a for a, b in zip(seg, seg[1:])]
        alone = max(lengths) == 1
        t_d, p_d, s_d, seg_d, rows_d = self._upload(
            toks, *_positions(lengths, starts, slots), seg, rows)
        w = self._scratch if n <= self.B else _Scratch(self.model, n)
        hf = torch.zeros(len(rows), pad8(self.cfg.dim), dtype=self.model.dtype, device=self.dev)
        logits = torch.empty(len(rows), pad8(self.vocab), dtype=torch.float32, device=self.dev)
        self._forward(w, n, t_d, p_d, s_d, rows=rows_d,
                      seg=None if alone else (seg_d, len(lengths), max(lengths)),
                      ctx=None if alone else self._context(lengths, starts, slots),
                      hf=hf, logits=logits)
        out.copy_(logits[:, : self.vocab])
        return out

    def _step_portions(self, entries):
        """A step too large for one forward: its tokens in portions, in order."""
        got: Dict[int, List[torch.Tensor]] = {}
        batch, room = [], MAX_FORWARD_TOKENS

        def flush():
            nonlocal batch, room
            if batch:
                res = self.step([(k, ids, want) for _, k, ids, want in batch])
                at = 0
                for i, _, _, want in batch:
                    got.setdefault(i, []).append(res[at: at + len(want)])
                    at += len(want)
            batch, room = [], MAX_FORWARD_TOKENS
        order: Dict[int, List[int]] = {}
        for i, (key, ids, want) in enumerate(entries):
            at = 0
            order[i] = []
            while at < len(ids):
                take = min(room, len(ids) - at)
                here = [j for j, p in enumerate(want) if at <= p < at + take]
                order[i] += here
                batch.append((i, key, ids[at: at + take], [want[j] - at for j in here]))
                at += take
                room -= take
                if room == 0:
                    flush()
        flush()
        out = []
        for i in range(len(entries)):
            if order[i]:
                res = torch.cat(got[i])
                back = torch.empty_like(res)
                back[torch.tensor(order[i], device=res.device)] = res
                out.append(back)
        return torch.cat(out) if out else torch.empty(0, self.vocab, device=self.dev)

    # ------------------------------------------------------------------ generation loop
    def _open_rows(self, B: int) -> None:
        self._close_rows()
        for b in range(B):
            key = ("row", b)
            self.cache.open(key)
            self._rows.append(key)
        self.slot[:B] = torch.tensor([self.cache.slot(k) for k in self._rows], dtype=torch.int32)

    def _close_rows(self) -> None:
        while self._rows:
            self.cache.close(self._rows.pop())

    def _decode_step(self, B, temperature, top_k, eos_id):
        self._forward(self._scratch, B, self.next_tok[:B], self.tok_pos[:B], self.slot[:B],
                      decode_counters=True, hf=self.hf, logits=self.logits)
        self._sample(self.logits[:B], B, temperature, top_k, eos_id)
        self._count(1)

    @torch.no_grad()
    def prefill(self, prompt: torch.Tensor, left_pad_mask_pos: Optional[torch.Tensor],
                temperature: float, top_k: Optional[int], seed: int, eos_id: int):
        """prompt [B, T], left padded: the pads are dropped, every row's tokens enter at position
        0, and the first new token goes to ``seq[:, T]``."""
        B, T = prompt.shape
        if not self._rows:
            self._open_rows(B)
        ids = prompt.to(device=self.dev, dtype=torch.int32)
        self._begin(prompt, left_pad_mask_pos, seed)
        pads = [0] * B if left_pad_mask_pos is None else \
            [min(int(p), T - 1) for p in left_pad_mask_pos.tolist()]
        self.left_pad[:B] = torch.tensor(pads, dtype=torch.int32)
        self.launches_per_step = 0
        slots = self.slot[:B].tolist()
        done = [0] * B
        while True:
            # next packed forward: whole rows while they fit, else a portion of one
            pick, room = [], MAX_FORWARD_TOKENS
            for b in range(B):
                left = T - pads[b] - done[b]
                if left > 0 and room > 0:
                    take = min(left, room)
                    pick.append((b, done[b], take))
                    done[b] += take
                    room -= take
            if not pick:
                break
            self._prefill_part(ids, T, pads, slots, pick)
        self.pos.fill_(T - 1)
        self._sample(self.logits[:B], B, temperature, top_k, eos_id)
        self.prefill_launches = self.launches_per_step + 1

    def _prefill_part(self, ids, T, pads, slots, pick):
        seg, cell, rows, fin = [0], [], [], []
        pick = sorted(pick, key=lambda p: -p[2])
        for b, at, take in pick:
            lo = b * T + pads[b] + at
            cell.append(np.arange(lo, lo + take))
            seg.append(seg[-1] + take)
            if at + take == T - pads[b]:
                rows.append(seg[-1] - 1)
                fin.append(b)
        n = seg[-1]
        lengths, starts = [t for _, _, t in pick], [a for _, a, _ in pick]
        slots = [slots[b] for b, _, _ in pick]
        ctx = self._context(lengths, starts, slots)
        cell, pos, slot, seg_d, rows_d, fin_d = self._upload(
            np.concatenate(cell), *_positions(lengths, starts, slots), seg, rows, fin)
        tokens = ids.reshape(-1)[cell.long()]
        w = self._scratch if n <= self.B else _Scratch(self.model, n)
        whole = fin == list(range(ids.shape[0]))
        logits = self.logits if whole else torch.empty_like(self.logits)
        self._forward(w, n, tokens, pos, slot, seg=(seg_d, len(lengths), max(lengths)), ctx=ctx,
                      rows=rows_d, hf=self.hf, logits=logits)
        if not whole and fin:
            self.logits[fin_d.long()] = logits[: len(fin)]
