"""Host side of the hybrid decoders: configuration, weight packing, rotation table, slot cache,
safetensors files, the entry points' dispatch."""
import json

import pytest
import torch

import bovinex_models as M
import bovinex_oracle as O


def test_config_is_read_completely():
    from easy_to_hard_b200.models.hybrid import hybrid_config
    c = hybrid_config(M.ZOO["mixed"])
    a, g = c.layers[0], c.layers[1]
    assert (c.vocab_size, c.dim, c.norm_offset, c.n_layer) == (333, 120, 1.0, 4)
    assert (a.mixer.heads, a.mixer.kv_heads, a.mixer.dim, a.mixer.vdim) == (6, 3, 40, 24)
    assert (a.mixer.window, a.mixer.keep, a.mixer.rot.dims) == (20, 3, 24)
    assert a.mixer.rot.scaling.factor == 4.0 and a.mlp.ff == 76
    assert (g.mixer.tau, g.mlp.experts, g.mlp.top, g.mlp.ff) == (4.0, 5, 2, 44)
    p = hybrid_config(M.ZOO["plain"])
    assert p.layers[0].mlp is None and p.layers[1].mixer.window == 0
    assert p.layers[1].mixer.rot.scaling is None and p.layers[2].mixer.keep == 0
    with pytest.raises(ValueError, match="unknown architecture"):
        hybrid_config(dict(M.ZOO["mixed"], architecture="Nothing"))


@pytest.mark.parametrize("scaling", [None, M.YARN, dict(factor=2.0, original=512, fast=64.0,
                                                        slow=2.0)])
def test_rotation_table(scaling):
    from easy_to_hard_b200.models.hybrid import Rotary, Yarn
    rot = dict(dims=36, base=5000.0, scaling=scaling)
    r = Rotary(36, 5000.0, Yarn(**scaling) if scaling else None)
    x = torch.randn(50, 2, 40, dtype=torch.float64)
    want = O.rotate(x, rot)
    t = r.table(50).double()
    c, s = t[:, None, :, 0], t[:, None, :, 1]
    u, v = x[..., :18], x[..., 18:36]
    got = torch.cat([u * c - v * s, v * c + u * s, x[..., 36:]], -1)
    assert torch.allclose(got, want, atol=1e-6)
    # slow dimensions are interpolated, fast ones are not
    if scaling:
        freq, _ = r.frequencies()
        plain, _ = Rotary(36, 5000.0).frequencies()
        assert freq[0] == plain[0] and torch.isclose(freq[-1] * scaling["factor"], plain[-1])


@pytest.mark.parametrize("name", sorted(M.ZOO))
def test_packed_weights_compute_the_layers(name):
    """The packed matrices, applied with plain torch operations, give the layers of the oracle."""
    from easy_to_hard_b200.models.hybrid import HybridLM, hybrid_config
    cfg = M.ZOO[name]
    W = M.weights(cfg, 3, dtype=torch.float32)
    model = HybridLM.from_tensors(hybrid_config(cfg), W, device="cpu", dtype=torch.float32)
    h = torch.randn(5, cfg["width"])
    for i, (blk, L) in enumerate(zip(model.layers, cfg["layers"])):
        p, m = f"l{i}.mix.", blk.layer.mixer
        y = h @ blk.mat("w_in").T
        if blk.b_in is not None:
            y = y + blk.b_in
        assert blk.off_g % 8 == 0 and y.shape[1] % 8 == 0 and blk.f_main % 8 == 0
        kv = m.kv_heads if m.kind == "attention" else m.heads
        bias = (lambda n: W[p + n + ".b"]) if m.kind == "attention" else (lambda n: 0)
        for n, off, rows in (("q", blk.off_q, m.heads * m.dim), ("k", blk.off_k, kv * m.dim),
                             ("v", blk.off_v, kv * m.vdim)):
            assert torch.allclose(y[:, off: off + rows], h @ W[p + n].T + bias(n), atol=1e-5)
        att = torch.randn(5, m.heads * m.vdim)
        z = torch.zeros(5, blk.f_main - blk.off_g)
        z[:, : att.shape[1]] = att
        want = att @ W[p + "o"].T
        f = blk.layer.mlp
        if f is not None and f.kind == "dense":
            c = blk.off_u - blk.off_g
            z[:, c:] = torch.relu(y[:, blk.off_u: blk.f_main]).square()
            want = want + O.dense(h, W, f"l{i}.mlp.")
        assert torch.allclose(z @ blk.mat("w_out").T, want, atol=1e-4)
        if m.kind == "gla":
            a = y[:, blk.f_main: blk.f_main + m.rank]
            al = torch.sigmoid(a @ blk.a2.T + blk.a2_b).pow(1 / m.tau)
            assert torch.allclose(al.view(5, m.heads, m.dim), O.gla_decay(h, W, p, L["mixer"]),
                                  atol=1e-5)
        if f is not None and f.kind == "moe":
            r = y[:, blk.f_main + blk.off_r:][:, : f.experts]
            idx, w = O.route(r, f.top)
            out = torch.zeros(5, cfg["width"])
            for t in range(5):
                for e, a in zip(idx[t].tolist(), w[t]):
                    rows = slice(e * blk.ffp, (e + 1) * blk.ffp)
                    u = torch.nn.functional.silu(h[t] @ blk.mat("e_gate")[rows].T) * (
                        h[t] @ blk.mat("e_up")[rows].T)
                    out[t] += a * (u @ blk.mat("e_down")[e * cfg["width"]:
                                                         (e + 1) * cfg["width"]].T)
            assert torch.allclose(out, O.moe(h, W, f"l{i}.mlp.", L["mlp"]), atol=1e-4)


def test_missing_and_misshapen_tensors_are_named():
    from easy_to_hard_b200.models.hybrid import HybridLM, hybrid_config
    cfg = M.ZOO["mixed"]
    W = M.weights(cfg)
    bad = dict(W)
    del bad["l1.mlp.e3.up"]
    with pytest.raises(KeyError, match="l1.mlp.e3.up"):
        HybridLM.from_tensors(hybrid_config(cfg), bad, device="cpu")
    bad = dict(W)
    bad["l0.mix.k"] = bad["l0.mix.k"][:-1]
    with pytest.raises(ValueError, match="l0.mix.k"):
        HybridLM.from_tensors(hybrid_config(cfg), bad, device="cpu")
    with pytest.raises(ValueError, match="256"):
        hc = hybrid_config(M.config([M.attn(2, 1, 264, 16)]))
        HybridLM.from_tensors(hc, {}, device="cpu")


def test_slot_cache_books_positions_and_reuses_slots():
    from easy_to_hard_b200.models.hybrid import hybrid_config
    from easy_to_hard_b200.models.slot_cache import SlotCache
    c = SlotCache(hybrid_config(M.ZOO["mixed"]).layers, 2, 16, "cpu", torch.bfloat16)
    a, b = c.open("a"), c.open("b")
    assert {a, b} == {0, 1} and c.extend("a", 5) == 0 and c.extend("a", 2) == 5
    assert c.length("a") == 7 and c.length("b") == 0
    with pytest.raises(RuntimeError, match="slots"):
        c.open("c")
    with pytest.raises(RuntimeError, match="positions"):
        c.extend("a", 10)
    assert c.length("a") == 7
    c.close("a")
    assert "a" not in c and c.open("c") == a and c.length("c") == 0
    kc, vc = c.layers[0]
    assert kc.shape == (2, 3, 16, 40) and vc.shape == (2, 3, 16, 24)
    assert c.layers[3][0].shape == (2, 3, 20, 28) and c.layers[3][0].dtype == torch.float32


def test_safetensors_round_trip(tmp_path):
    from easy_to_hard_b200.utils.safetensors_io import load_safetensors, save_safetensors
    t = {"a": torch.randn(3, 5).bfloat16(), "b": torch.arange(7, dtype=torch.int32),
         "c": torch.randn(2), "d": torch.zeros(0, 4), "e": torch.tensor([True, False, True])}
    save_safetensors(tmp_path / "x.safetensors", t)
    r = load_safetensors(tmp_path / "x.safetensors")
    assert set(r) == set(t)
    for k in t:
        assert r[k].dtype == t[k].dtype and torch.equal(r[k], t[k])
    (tmp_path / "y.safetensors").write_bytes((tmp_path / "x.safetensors").read_bytes()[:-8])
    with pytest.raises(ValueError, match="fit"):
        load_safetensors(tmp_path / "y.safetensors")


def test_checkpoint_folder_selects_the_model_class(tmp_path):
    import inference_generate as ig
    from easy_to_hard_b200.models.hybrid import config_in
    (tmp_path / "model.safetensors").write_bytes(b"")
    assert config_in(tmp_path) is None
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["Other"]}))
    assert config_in(tmp_path) is None
    (tmp_path / "config.json").write_text(json.dumps(M.ZOO["mixed"]))
    assert config_in(tmp_path)["architecture"] == "Bovinex"
    with pytest.raises(RuntimeError, match="CUDA"):
        ig._load_model(tmp_path / "model.safetensors", "cpu", torch.float32, False)


def test_window_of_the_oracle():
    """The mask the other tests rely on, spelled out for one row."""
    v = O.visible(12, dict(size=4, keep_first=2))
    assert v[9].tolist() == [True, True] + [False] * 4 + [True] * 4 + [False] * 2
    assert v[3].tolist() == [True] * 4 + [False] * 8
    assert O.visible(5, None).sum() == 15
