"""Host side of the Ruralorn decoder: configuration, weight packing, rotation table, cache layout,
the bookkeeping of prompt segments."""
import pytest
import torch

import ruralorn_models as M
import ruralorn_oracle as O


def _model(cfg, W, **kw):
    from easy_to_hard_b200.models.hybrid import HybridLM, hybrid_config
    return HybridLM.from_tensors(hybrid_config(cfg), W, device="cpu", **kw)


def test_config_is_read_completely():
    from easy_to_hard_b200.models.hybrid import hybrid_config
    c = hybrid_config(M.ZOO["mixed"])
    assert (c.vocab_size, c.dim, c.norm_offset, c.n_layer, c.parallel) == (333, 120, 0.0, 3, False)
    assert (c.logit_scale, c.logit_softcap, c.embed_scale, c.norm_eps) == (0.5, 8.0, 3.0, 1e-5)
    m, f = c.layers[0].mixer, c.layers[0].mlp
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.window) == (6, 40, 24, 32, 72, 20)
    assert m.rot.dims == 24 and m.rot.base == 10000.0 and m.rot.interleaved
    assert m.scale == pytest.approx(1.1 / 8)
    assert (f.experts, f.top, f.ff, f.shared.ff, f.shared.act) == (5, 2, 44, 56, "gelu")
    assert (f.gated, f.act, f.score, f.weight_input, f.bias) == (False, "gelu", "sigmoid", True, False)
    assert c.layers[1].mixer.rot.base == 500.0 and c.layers[1].mlp.shared is None
    assert c.layers[2].mlp is None
    assert hybrid_config(M.ZOO["plain"]).layers[0].mixer.window == 0
    bare = dict(M.ZOO["plain"])
    del bare["logit_scale"], bare["logit_softcap"]
    assert (hybrid_config(bare).logit_scale, hybrid_config(bare).logit_softcap) == (1.0, 0.0)
    bad = M.config([dict(M.layer(), type="something")])
    with pytest.raises(ValueError, match="unknown mixer"):
        hybrid_config(bad)


def test_rotation_table_pairs_neighbours():
    from easy_to_hard_b200.models.hybrid import Rotary
    x = torch.randn(50, 2, 24, dtype=torch.float64)
    want = O.rotate_pairs(x, 700.0, 20)
    t = Rotary(20, 700.0, interleaved=True).table(50, pairs=12).double()
    assert t.shape == (50, 12, 2) and bool((t[:, 10:] == torch.tensor([1.0, 0.0])).all())
    c, s = t[:, None, :, 0], t[:, None, :, 1]
    u, v = x[..., 0::2], x[..., 1::2]
    assert torch.allclose(torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), want,
                          atol=1e-6)


@pytest.mark.parametrize("name", sorted(M.ZOO))
def test_packed_weights_compute_the_layers(name):
    """The packed matrices, applied with plain torch operations, give the layers of the oracle; the
    filling columns come out as zeros."""
    cfg = M.ZOO[name]
    W = M.weights(cfg, 3, dtype=torch.float32)
    model = _model(cfg, W, dtype=torch.float32)
    T, eps = 9, cfg["norm"]["eps"]
    h = torch.randn(T, cfg["width"])
    p8 = lambda n: (n + 7) // 8 * 8  # noqa: E731
    for i, (blk, L) in enumerate(zip(model.layers, cfg["layers"])):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        H, d, r, e, k = (m[n] for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        dp, rp, ep, kp = p8(d), p8(r), p8(e), p8(k)
        y = h @ blk.mat("w_in").T
        assert blk.b_in is None and blk.n_tail == 0 and y.shape[1] == blk.f_main
        q = y[:, blk.off_q: blk.off_c].view(T, H, dp + rp)
        want = O.queries(h, W, p + "mix.", dict(m, rot=dict(dims=0, base=2.0)))
        assert torch.allclose(torch.cat([q[..., :d], q[..., dp: dp + r]], -1), want, atol=1e-5)
        assert not q[..., d:dp].any() and not q[..., dp + r:].any()
        c = y[:, blk.off_c: blk.off_c + kp]
        c = c / torch.sqrt(c.square().sum(1, keepdim=True) / k + eps) * blk.c_norm
        kr = y[:, blk.off_c + kp: blk.off_c + kp + rp]
        c_want, kr_want = O.latents(h, W, p + "mix.", dict(m, rot=dict(dims=0, base=2.0)), eps)
        assert torch.allclose(c[:, :k], c_want, atol=1e-5) and not c[:, k:].any()
        assert torch.allclose(kr[:, :r], kr_want, atol=1e-5) and not kr[:, r:].any()
        keys, vals = O.expand(c_want, kr_want, W, p + "mix.", m)
        kv = c @ blk.w_kv.T
        assert torch.allclose(kv[:, : H * dp].view(T, H, dp)[..., :d], keys[..., :d], atol=1e-4)
        got = kv[:, H * dp:].view(T, H, ep)
        assert torch.allclose(got[..., :e], vals, atol=1e-4) and not got[..., e:].any()
        # scores through the absorbed queries
        ql = torch.einsum("thd,hkd->thk", q[..., :dp], blk.w_uk_t.view(H, kp, dp))
        s = torch.einsum("thk,sk->hts", ql, c)
        assert torch.allclose(s, torch.einsum("thd,shd->hts", want[..., :d], keys[..., :d]),
                              atol=1e-3)
        g = y[:, blk.off_g:].view(T, H, ep)
        assert torch.allclose(g[..., :e].flatten(1), h @ W[p + "mix.g"].T, atol=1e-5)
        o = torch.randn(T, H, e)
        op = torch.zeros(T, H, ep)
        op[..., :e] = o
        assert torch.allclose(op.flatten(1) @ blk.mat("w_out").T, o.flatten(1) @ W[p + "mix.o"].T,
                              atol=1e-4)
        if not f:
            assert blk.f_ff == 0 and not hasattr(blk, "norm2")
            continue
        u = h @ blk.mat("w_ff").T
        z = u[:, blk.f_ff + blk.off_r:][:, : f["router"]["experts"]]
        idx, w = O.route(z, f["router"]["top"])
        out = torch.zeros(T, cfg["width"])
        if f.get("shared"):
            out += O.gelu(u[:, : blk.f_ff]) @ blk.mat("w_down").T
        for t in range(T):
            for x, a in zip(idx[t].tolist(), w[t]):
                up = O.gelu((a * h[t]) @ blk.mat("e_up")[x * blk.ffp: (x + 1) * blk.ffp].T)
                out[t] += up @ blk.mat("e_down")[x * cfg["width"]: (x + 1) * cfg["width"]].T
        assert torch.allclose(out, O.moe(h, W, p + "mlp.", f), atol=1e-3)


def test_missing_and_misshapen_tensors_are_named():
    cfg = M.ZOO["mixed"]
    W = M.weights(cfg)
    bad = dict(W)
    del bad["l0.mlp.shared.down"]
    with pytest.raises(KeyError, match="l0.mlp.shared.down"):
        _model(cfg, bad)
    bad = dict(W)
    bad["l2.mix.uk"] = bad["l2.mix.uk"][:-1]
    with pytest.raises(ValueError, match="l2.mix.uk"):
        _model(cfg, bad)
    with pytest.raises(ValueError, match="1024"):
        _model(M.config([M.layer(rank=1032)]), {})
    with pytest.raises(ValueError, match="rotate"):
        _model(M.config([M.layer(rot=15)]), {})


def test_cache_keeps_latents_only():
    from easy_to_hard_b200.models.hybrid import hybrid_config
    from easy_to_hard_b200.models.slot_cache import SlotCache
    c = SlotCache(hybrid_config(M.ZOO["odd"]).layers, 2, 16, "cpu", torch.bfloat16)
    assert [tuple(t.shape for t in x) for x in c.layers] == [((2, 16, 40),), ((2, 16, 72),)]


def test_segment_bookkeeping():
    """Rows of the expanded context: what the cache holds inside the widest window, then the new
    tokens; short segments and segments with a long past are left to the absorbed kernel."""
    from easy_to_hard_b200.ops.hybrid import LatentAttention, LatentContext
    n = LatentAttention.TENSOR_CORE_TOKENS
    c = LatentContext([n + 6, n, n - 1, 1], [5, 40, 0, 9], [2, 0, 1, 3], 8, True, "cpu")
    assert (c.n_long, c.n_long_seg, c.seg_max) == (2 * n + 6, 2, n + 6)
    assert c.n_ctx == 5 + n + 6 + 7 + n
    src = [-1] * 5 + list(range(n + 6)) + [-1] * 7 + list(range(n + 6, 2 * n + 6))
    assert c.src.tolist() == src
    assert c.pos.tolist() == list(range(n + 11)) + list(range(33, 40 + n))
    assert c.slot.tolist() == [2] * (n + 11) + [0] * (7 + n)
    assert c.shift.tolist() == [0, n + 11 - 33]
    for kw in (dict(window=8, expand=False), dict(window=0, expand=True)):
        c = LatentContext([n], [LatentAttention.HISTORY * n + 1], [0], device="cpu", **kw)
        assert c.n_ctx == c.n_long == 0
    assert LatentContext([n], [LatentAttention.HISTORY * n], [0], 0, True, "cpu").n_long == n


def test_window_of_the_oracle():
    """The mask the other tests rely on, spelled out for one row."""
    v = O.visible(12, 4)
    assert v[9].tolist() == [False] * 6 + [True] * 4 + [False] * 2
    assert v[2].tolist() == [True] * 3 + [False] * 9 and O.visible(5, None).sum() == 15


def test_sources_of_a_design_are_those_its_layers_run_on():
    """What a fresh checkout compiles before it replays a trace: the named sources exist, define the
    entry points the layers call, and depend on no other source."""
    import re

    import bovinex_models as B
    from easy_to_hard_b200.models.hybrid import hybrid_config, kernel_sources
    from easy_to_hard_b200.ops import build
    names = kernel_sources(hybrid_config(M.ZOO["mixed"]))
    assert "latent_attn" in names and "moe" in names
    assert not {"attn_window", "gla", "gla_chunk", "loss", "flash_attn"} & set(names)
    bare = kernel_sources(hybrid_config(M.config([M.layer()])))
    assert "moe" not in bare
    assert {"attn_window", "gla", "moe"} <= set(kernel_sources(hybrid_config(B.ZOO["mixed"])))
    srcs = build.sources(names)
    assert all(s.is_file() for s in srcs)
    entry = set(re.findall(r'extern "C" int (e2h_\w+)', "".join(s.read_text() for s in srcs)))
    assert {"e2h_gemm_umma", "e2h_gemm_persistent", "e2h_gemm_f32", "e2h_stream_norm",
            "e2h_moe_route", "e2h_latent_prep", "e2h_latent_attn", "e2h_flash_window"} <= entry
    assert build.lib_path(names) != build.lib_path() != build.lib_path(bare)
