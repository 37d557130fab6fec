"""Device time of every kernel of a hybrid-decoder layer against its roofline, beside the like
kernels of the LLaMA path at equal size.

    python bench/hybrid_kernel_bench.py [--model bovinex|ruralorn] [--size 4k] [--batch 64]
                                        [--context 1024] [--prompt 8x2048]

Beside Bovinex: the LLaMA path; beside Ruralorn: the Bovinex layers of attention + experts.

Each kernel is timed alone with CUDA events, L2 flushed before every launch (a 512 MB write),
median of the launches. The roofline time is the larger of algorithmic bytes over the measured copy
bandwidth and algorithmic FLOPs over the measured GEMM rate (MEASURED_PEAKS.json, or its stated
fallback)."""
from __future__ import annotations

import argparse
import json
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "bench"))

import torch  # noqa: E402

from hybrid_shapes import (bovinex_attention_model, bovinex_model, llama_model,  # noqa: E402
                           ruralorn_model)


def peaks():
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as fh:
            d = json.load(fh)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12
    except OSError:
        return 6.65e12, 1.59e15


FLUSH = None


def time_us(fn, reps=12):
    global FLUSH
    if FLUSH is None:
        FLUSH = torch.empty(512 << 20, dtype=torch.uint8, device="cuda")
    for _ in range(3):
        fn()
    out = []
    for _ in range(reps):
        FLUSH.fill_(1)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        out.append(a.elapsed_time(b) * 1e3)
    out.sort()
    return out[len(out) // 2]


def row(name, us, nbytes, flops=0.0):
    bw, fl = peaks()
    floor = max(nbytes / bw, flops / fl) * 1e6
    kind = "HBM" if nbytes / bw >= flops / fl else "tensor"
    print(f"| {name} | {us:.1f} | {floor:.1f} | {kind} | {floor / us:.2f} |", flush=True)


def head(title):
    print(f"\n### {title}\n\n| kernel | us | roofline us | bound | fraction of measured |\n"
          "|---|---|---|---|---|")


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def bovinex(size, batch, context, prompts, plen, attention_only=False):
    from easy_to_hard_b200.models.hybrid_engine import _Scratch
    from easy_to_hard_b200.ops import gemm, hybrid as hy
    layers = 1 if attention_only else 4
    model = bovinex_attention_model(size, 1) if attention_only else bovinex_model(size, 4)
    n_max = prompts * plen
    eng = model.make_engine(max(batch, prompts), max(context + 8, plen), use_graph=False)
    cfg, W = model.config, model.config.dim
    for phase, n in (("decode", batch), ("prompt", n_max)):
        head(f"Bovinex {size}, {phase}: " + (f"{batch} sequences at position {context}"
                                             if phase == "decode" else
                                             f"{prompts} prompts of {plen} tokens"))
        w = _Scratch(model, n)
        w.x.normal_()
        if phase == "decode":
            pos, slot, seg = i32([context] * n), i32(list(range(n))), None
        else:
            pos = i32(list(range(plen)) * prompts)
            slot = i32([b for b in range(prompts) for _ in range(plen)])
            seg = (i32([b * plen for b in range(prompts + 1)]), prompts, plen)
        h = w.h[:n]
        hy.stream_norm(w.x, model.layers[0].norm1, h, eps=1e-5, offset=1.0)
        row("residual norm", time_us(lambda: hy.stream_norm(
            w.x, model.layers[0].norm1, h, eps=1e-5, offset=1.0)), n * W * 6)
        for li in range(layers):
            blk, mix, m, f = (model.layers[li], eng.mixers[li], model.layers[li].layer.mixer,
                              model.layers[li].layer.mlp)
            tag = f"{m.kind}+{f.kind}"
            act = w.act(n, blk.f_main)
            tail = w.tail(n, blk.n_tail) if blk.n_tail else None
            F = blk.w_in.shape[0]
            args = dict(bias=blk.b_in, tail=tail,
                        act_from=blk.off_u if f.kind == "dense" else None)
            run_in = lambda: gemm.linear_packed(h[:, :W], blk.mat("w_in"), act, **args)  # noqa
            run_in()
            row(f"{tag}: w_in GEMM ({F} x {W})", time_us(run_in), (F * W + n * W + n * F) * 2,
                2.0 * n * F * W)
            if li in (0, 1):
                if m.kind == "attention":
                    kv = m.kv_heads * (m.dim + m.vdim) * 2
                    io = n * (m.heads * (m.dim + 2 * m.vdim) * 2 + kv)
                    if phase == "decode":
                        keys = min(context + 1, m.window + m.keep)
                        row("attention decode (norms, rotation, cache write, gate)",
                            time_us(lambda: mix.decode(act, pos, slot)), io + n * keys * kv,
                            2.0 * n * keys * m.heads * (m.dim + m.vdim))
                    else:
                        vis = sum(min(i + 1, m.window + m.keep) for i in range(plen)) * prompts
                        row("attention prep (norms, rotation, cache write)",
                            time_us(lambda: mix.prep(act, pos, slot)),
                            n * (2 * m.heads * m.dim * 2 + 2 * kv))
                        row("attention (windowed flash, gate)", time_us(
                            lambda: mix.attend(act, pos, slot, *seg)), io,
                            2.0 * vis * m.heads * (m.dim + m.vdim))
                else:
                    st = m.heads * m.dim * m.vdim * 4
                    io = n * (2 * m.heads * m.dim + 3 * m.heads * m.vdim) * 2
                    if phase == "decode":
                        row("gla decode (decay, state, norm, gate)",
                            time_us(lambda: mix.decode(act, tail, pos, slot)), io + n * 2 * st)
                    else:
                        # recurrent form of the chunked algorithm, one product each
                        fl = 2.0 * n * m.heads * (2 * m.dim * m.vdim + 64 * (m.dim + m.vdim))
                        row("gla prompt (decay, chunks, norm, gate)",
                            time_us(lambda: mix.prompt(act, tail, pos, slot, *seg)),
                            io + prompts * 2 * st, fl)
            K = blk.f_main - blk.off_g
            row(f"{tag}: w_out GEMM + fp32 residual ({W} x {K})",
                time_us(lambda: gemm.linear_residual_f32(act[:, blk.off_g:], blk.mat("w_out"),
                                                         w.x[:n])),
                (W * K + n * K) * 2 + n * W * 8, 2.0 * n * W * K)
            if f.kind == "moe" and li == layers // 3:
                top, E = f.top, f.experts
                place, ew = w.choice(n, top)
                hg, ag, y = w.hg[: n * top, :W], w.ag(n * top, blk.ffp), w.y[: n * top, :W]
                tail[:, blk.off_r:].normal_()
                rt = lambda: hy.moe_route(tail[:, blk.off_r:], E, top, h[:, :W], hg,  # noqa: E731
                                          w.off, place, ew, w.sel)
                row("expert routing + regrouping", time_us(rt), n * W * 2 * (1 + top))
                rt()
                live = min(E, n * top)
                row(f"expert gate/up + SwiGLU ({E} x 2 x {blk.ffp} x {W})", time_us(
                    lambda: gemm.grouped_swiglu(hg, blk.mat("e_gate"), blk.mat("e_up"), ag, w.off,
                                                E, n)),
                    (2 * live * blk.ffp * W + n * top * (W + blk.ffp)) * 2,
                    4.0 * n * top * blk.ffp * W)
                row(f"expert down ({E} x {W} x {blk.ffp})", time_us(
                    lambda: gemm.grouped_linear(ag, blk.mat("e_down"), y, w.off, E, n)),
                    (live * blk.ffp * W + n * top * (W + blk.ffp)) * 2,
                    2.0 * n * top * blk.ffp * W)
                row("residual norm + expert outputs", time_us(lambda: hy.stream_norm(
                    w.x, model.layers[0].norm1, h, eps=1e-5, offset=1.0,
                    experts=(y, place, ew))), n * W * (10 + 2 * top))
        del w
    from easy_to_hard_b200.ops import _lib
    assert _lib.read_status() == 0


def ruralorn(size, batch, context, prompts, plen):
    from easy_to_hard_b200.models.hybrid_engine import _Scratch
    from easy_to_hard_b200.ops import gemm, hybrid as hy
    model = ruralorn_model(size, 1)
    eng = model.make_engine(max(batch, prompts), max(context + 8, plen), use_graph=False)
    W, blk, mix = model.config.dim, model.layers[0], eng.mixers[0]
    m, f = blk.layer.mixer, blk.layer.mlp
    H, d, r, e, k = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
    for phase, n in (("decode", batch), ("prompt", prompts * plen)):
        head(f"Ruralorn {size}, {phase}: " + (f"{batch} sequences at position {context}"
                                              if phase == "decode" else
                                              f"{prompts} prompts of {plen} tokens"))
        w = _Scratch(model, n)
        w.x.normal_()
        h = w.h[:n, :W]
        norm = lambda **kw: hy.stream_norm(w.x, blk.norm1, w.h[:n], eps=1e-5, **kw)  # noqa: E731
        norm()
        row("residual norm", time_us(norm), n * W * 6)
        act, F = w.act(n, blk.f_main), blk.f_main
        run = lambda: gemm.linear_packed(h, blk.mat("w_in"), act)  # noqa: E731
        run()
        row(f"w_in GEMM: q, latent, gate ({F} x {W})", time_us(run), (F * W + n * W + n * F) * 2,
            2.0 * n * F * W)
        if phase == "decode":
            pos, slot = i32([context] * n), i32(list(range(n)))
            ql, ol = eng._absorbed_rows(mix, n)
            run = lambda: mix.absorb(act, ql)  # noqa: E731
            run()
            row(f"absorbed queries ({H} x {k} x {d})", time_us(run),
                (H * k * d + n * H * (d + k)) * 2, 2.0 * n * H * k * d)
            keys = min(context + 1, m.window or context + 1)
            row("attention decode (norm, rotation, cache write)", time_us(
                lambda: mix.attend(act, ql, ol, pos, slot, fused=True)),
                n * (keys * (k + r) + H * (2 * k + r) + k + r) * 2, 2.0 * n * keys * H * (2 * k + r))
            row(f"value expansion + gate ({H} x {e} x {k})", time_us(lambda: mix.values(act, ol)),
                (H * k * e + n * H * (k + 2 * e)) * 2, 2.0 * n * H * k * e)
        else:
            pos = i32(list(range(plen)) * prompts)
            slot = i32([b for b in range(prompts) for _ in range(plen)])
            seg = i32([b * plen for b in range(prompts + 1)])
            ctx = eng._context([plen] * prompts, [0] * prompts, list(range(prompts)))
            bf = dict(dtype=torch.bfloat16, device="cuda")
            rows, kv = torch.empty(n, k + r, **bf), torch.empty(n, blk.w_kv.shape[0], **bf)
            row("attention prep (norm, rotation, cache write)", time_us(
                lambda: mix.prep(act, pos, slot, ctx, rows)), n * (3 * (k + r) + 2 * H * r) * 2)
            row(f"key and value expansion ({H * (d + e)} x {k})", time_us(
                lambda: mix.expand(rows, kv)), (H * (d + e) * k + n * (H * (d + e) + k)) * 2,
                2.0 * n * H * (d + e) * k)
            vis = sum(min(i + 1, m.window or plen) for i in range(plen)) * prompts
            row("attention (windowed flash, gate)", time_us(
                lambda: mix.flash(act, pos, slot, seg, ctx, rows, kv)),
                n * (H * (d + r + 2 * e) + H * (d + e) + r) * 2, 2.0 * vis * H * (d + r + e))
        K = blk.f_main - blk.off_g
        row(f"w_out GEMM + fp32 residual ({W} x {K})", time_us(
            lambda: gemm.linear_residual_f32(act[:, blk.off_g:], blk.mat("w_out"), w.x[:n])),
            (W * K + n * K) * 2 + n * W * 8, 2.0 * n * W * K)
        up, tail, top, E = w.ff(n, blk.f_ff), w.tail(n, blk.n_ff_tail), f.top, f.experts
        F = blk.w_ff.shape[0]
        run = lambda: gemm.linear_packed(h, blk.mat("w_ff"), up, tail=tail, act="gelu",  # noqa: E731
                                         act_from=0)
        run()
        row(f"w_ff GEMM: shared up + GELU, router ({F} x {W})", time_us(run),
            (F * W + n * W + n * F) * 2, 2.0 * n * F * W)
        row(f"w_down GEMM + fp32 residual ({W} x {blk.f_ff})", time_us(
            lambda: gemm.linear_residual_f32(up, blk.mat("w_down"), w.x[:n])),
            (W * blk.f_ff + n * blk.f_ff) * 2 + n * W * 8, 2.0 * n * W * blk.f_ff)
        place, ew = w.choice(n, top)
        hg, ag, y = w.hg[: n * top, :W], w.ag(n * top, blk.ffp), w.y[: n * top, :W]
        tail.normal_()
        run = lambda: hy.moe_route(tail[:, blk.off_r:], E, top, h, hg, w.off, place, ew,  # noqa: E731
                                   w.sel, score=f.score, weight_input=True)
        row("expert routing + weighted regrouping", time_us(run), n * W * 2 * (1 + top))
        run()
        live = min(E, n * top)
        row(f"expert up + GELU ({E} x {blk.ffp} x {W})", time_us(
            lambda: gemm.grouped_linear(hg, blk.mat("e_up"), ag, w.off, E, n, act="gelu")),
            (live * blk.ffp * W + n * top * (W + blk.ffp)) * 2, 2.0 * n * top * blk.ffp * W)
        row(f"expert down ({E} x {W} x {blk.ffp})", time_us(
            lambda: gemm.grouped_linear(ag, blk.mat("e_down"), y, w.off, E, n)),
            (live * blk.ffp * W + n * top * (W + blk.ffp)) * 2, 2.0 * n * top * blk.ffp * W)
        row("residual norm + expert outputs", time_us(lambda: norm(experts=(y, place, None))),
            n * W * (10 + 2 * top))
        V = model.head_w.shape[0]
        nl = min(n, batch)
        logits = torch.empty(nl, V, device="cuda")
        row(f"LM head + scale, soft cap ({V} x {W}, {nl} rows)", time_us(
            lambda: gemm.linear_f32_out(h[:nl], model.head_w[:, :W], logits, scale=0.5,
                                        softcap=30.0)),
            (V * W + nl * W) * 2 + nl * V * 4, 2.0 * nl * V * W)
        del w
    from easy_to_hard_b200.ops import _lib
    assert _lib.read_status() == 0


def llama(size, batch, context, prompts, plen):
    from easy_to_hard_b200.models.engine import DecodeEngine
    from easy_to_hard_b200.ops import attention, functional as Fn, gemm
    m = llama_model(size, 1)
    eng = DecodeEngine(m, max(batch, prompts), max(context + 8, plen), use_graph=False)
    Ws, blk, W = eng.W[0], m.layers[0], m.config.dim
    H, G, D, ff = eng.n_head, eng.n_kv, eng.D, eng.ffn
    for phase, n, sq in (("decode", batch, 1), ("prompt", prompts * plen, plen)):
        head(f"LLaMA {size}, {phase}")
        bf = dict(dtype=torch.bfloat16, device="cuda")
        x, hh = torch.randn(n, W, **bf), torch.randn(n, W, **bf)
        q, att = torch.randn(n, H * D, **bf), torch.randn(n, H * D, **bf)
        act = torch.randn(n, ff, **bf)
        eng.pos.fill_(context if sq == 1 else 0)
        row("residual norm", time_us(lambda: Fn.fused_residual_rmsnorm(
            hh, blk.ffn_norm.weight, 1e-5, x_out=x)), n * W * 4)
        F = (H + 2 * G) * D
        row(f"wqkv GEMM + RoPE + KV write ({F} x {W})", time_us(
            lambda: gemm.linear_qkv_rope(x, Ws["wqkv"][0], q, freqs=eng.freqs, pos_base=eng.pos,
                                         sq=sq, n_head=H, n_kv=G, head_dim=D,
                                         kcache=eng.kcache[0], vcache=eng.vcache[0])),
            (F * W + n * W + n * F) * 2, 2.0 * n * F * W)
        kv = G * D * 2 * 2
        if sq == 1:
            row("attention decode", time_us(lambda: Fn.attn_decode(
                q, eng.kcache[0], eng.vcache[0], eng.pos, eng.left_pad, H, out=att)),
                n * (2 * H * D * 2 + (context + 1) * kv), 4.0 * n * (context + 1) * H * D)
        else:
            row("attention (causal flash)", time_us(lambda: attention.prefill_attention(
                q.view(prompts, plen, H, D), eng.kcache[0], eng.vcache[0],
                eng.left_pad[:prompts], att.view(prompts, plen, -1))),
                n * (2 * H * D * 2 + kv), 2.0 * prompts * plen * (plen + 1) * H * D)
        row(f"wo GEMM + residual ({W} x {H * D})", time_us(
            lambda: gemm.linear_residual(att, Ws["wo"][0], hh, out=hh)),
            (W * H * D + n * H * D + 2 * n * W) * 2, 2.0 * n * W * H * D)
        row(f"w1/w3 GEMM + SwiGLU (2 x {ff} x {W})", time_us(
            lambda: gemm.linear_swiglu(x, Ws["w1"][0], Ws["w3"][0], out=act)),
            (2 * ff * W + n * W + n * ff) * 2, 4.0 * n * ff * W)
        row(f"w2 GEMM + residual ({W} x {ff})", time_us(
            lambda: gemm.linear_residual(act, Ws["w2"][0], hh, out=hh)),
            (W * ff + n * ff + 2 * n * W) * 2, 2.0 * n * ff * W)
    from easy_to_hard_b200.ops import _lib
    assert _lib.read_status() == 0


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--model", default="bovinex", choices=["bovinex", "ruralorn"])
    ap.add_argument("--size", default="4k")
    ap.add_argument("--batch", type=int, default=64)
    ap.add_argument("--context", type=int, default=1024)
    ap.add_argument("--prompt", default="8x2048", help="prompts x tokens")
    a = ap.parse_args()
    p, t = (int(v) for v in a.prompt.split("x"))
    with torch.no_grad():
        if a.model == "ruralorn":
            ruralorn(a.size, a.batch, a.context, p, t)
            torch.cuda.empty_cache()
            bovinex(a.size, a.batch, a.context, p, t, attention_only=True)
        else:
            bovinex(a.size, a.batch, a.context, p, t)
            torch.cuda.empty_cache()
            llama(a.size, a.batch, a.context, p, t)
