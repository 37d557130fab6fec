"""Hybrid decoders: models whose layers mix attention with recurrent mixers and dense with
mixture-of-experts feed-forwards, described layer by layer in a ``config.json``.

A design is a reader that turns its ``config.json`` into the generic description below (mixers,
feed-forwards, rotation, masks, norms, each with its constants as parameters); everything
underneath -- weight packing, the slot cache, the engine and the kernels -- is shared. Adding a
design means adding a reader (and the mechanisms it has that no other design has).

The module holds the weights in the layout the engine's kernels read. With a parallel block (mixer
and feed-forward read one norm and are added together) a layer is two products:

* ``w_in``   q, k, v (or the latent projection), gate and the dense up projection stacked as one
  ``[F, width]`` matrix, with fp32 tail rows (low-rank decay input, router) that leave the GEMM
  unrounded;
* ``w_out``  ``[width, gated heads + ff]``: output projection and down projection side by side,
  reading the gated heads and the activated up projection where ``w_in`` left them.

In a sequential block (the feed-forward has a norm of its own) up projection and router are ``w_ff``
and the down projection is ``w_down``. Segments start at multiples of 8 columns; the filling rows /
columns are zero. Latent attention fills up every head, so that its kernels see multiples of 8 only.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field
from pathlib import Path
from typing import Callable, Dict, List, Mapping, Optional, Tuple, Union

import torch
import torch.nn as nn


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


# ------------------------------------------------------------------------------ description

@dataclass
class Yarn:
    """YaRN frequency interpolation: rotations faster than ``fast`` turns over the original
    context keep their frequency, slower than ``slow`` are divided by ``factor``."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass
class Rotary:
    dims: int                     # leading dimensions of a head that rotate
    base: float
    scaling: Optional[Yarn] = None
    interleaved: bool = False     # pairs (2i, 2i + 1); else (i, i + dims / 2)

    def frequencies(self) -> Tuple[torch.Tensor, float]:
        """(float64 angular frequency of every pair, amplitude of cos and sin)."""
        n = self.dims // 2
        i = torch.arange(n, dtype=torch.float64)
        freq = torch.pow(torch.tensor(float(self.base), dtype=torch.float64),
                         -2.0 * i / max(self.dims, 1))
        s = self.scaling
        if s is None:
            return freq, 1.0

        def turn_dim(turns: float) -> float:
            return (self.dims * math.log(s.original / (turns * 2 * math.pi))
                    / (2 * math.log(self.base)))

        lo = max(math.floor(turn_dim(s.fast)), 0)
        hi = min(math.ceil(turn_dim(s.slow)), self.dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
        return freq / s.factor * ramp + freq * (1 - ramp), 0.1 * math.log(s.factor) + 1.0

    def table(self, length: int, device=None, pairs: Optional[int] = None) -> torch.Tensor:
        """fp32 ``[length, pairs, 2]`` of (cos, sin), computed in double precision; pairs past
        ``dims / 2`` (the default) do not turn."""
        freq, amp = self.frequencies()
        ang = torch.outer(torch.arange(length, dtype=torch.float64), freq)
        t = torch.stack([amp * torch.cos(ang), amp * torch.sin(ang)], -1)
        if pairs is not None and pairs > len(freq):
            still = torch.tensor([1.0, 0.0], dtype=torch.float64)
            t = torch.cat([t, still.expand(length, pairs - len(freq), 2)], 1)
        return t.float().to(device)


@dataclass
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotary
    window: int = 0               # 0: unlimited
    keep: int = 0                 # first tokens that stay visible past the window
    kind: str = "attention"


@dataclass
class LatentMixer:
    """Keys and values of all heads are linear in one normed latent of ``kv_rank`` columns; a rotated
    key part of ``rot_dim`` columns is shared by the heads."""
    heads: int
    dim: int                      # unrotated part of a query / key
    rot_dim: int                  # rotated part behind it
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotary
    window: int = 0               # 0: unlimited
    kind: str = "latent"


@dataclass
class GlaMixer:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 0                 # of the decay projection; from the weights
    kind: str = "gla"


@dataclass
class DenseMlp:
    ff: int
    act: str = "relu2"            # w_down act(w_up h); "relu2" or "gelu"
    kind: str = "dense"


@dataclass
class MoeMlp:
    experts: int
    top: int
    ff: int                       # per expert
    gated: bool = True            # w_down (silu(w_gate h) * w_up h), else w_down act(w_up h)
    act: str = "silu"             # of experts without a gate: as in DenseMlp
    score: str = "softmax"        # weights: softmax over the chosen logits, or "sigmoid" of each
    weight_input: bool = False    # the weight multiplies the expert's input, not its output
    bias: bool = True             # of the router
    shared: Optional[DenseMlp] = None   # runs for every token and is added
    kind: str = "moe"


@dataclass
class HybridLayer:
    mixer: Union[AttentionMixer, LatentMixer, GlaMixer]
    mlp: Optional[Union[DenseMlp, MoeMlp]]


@dataclass
class HybridConfig:
    architecture: str
    vocab_size: int
    dim: int
    norm_eps: float
    embed_scale: float
    layers: List[HybridLayer]
    norm_offset: float = 0.0      # norms multiply by (offset + weight)
    parallel: bool = True         # mixer and feed-forward read one norm and are added together
    logit_scale: float = 1.0
    logit_softcap: float = 0.0    # logits <- cap * tanh(logits / cap); 0: none
    block_size: int = 1 << 20     # positions are unbounded; the cache is sized per run

    @property
    def n_layer(self) -> int:
        return len(self.layers)


# ------------------------------------------------------------------------------ designs

def read_bovinex(d: Mapping) -> HybridConfig:
    """Bovinex: parallel blocks; attention over a window plus the leading tokens, or gated linear
    attention; squared-ReLU or mixture-of-experts feed-forward."""
    layers = []
    for i, L in enumerate(d["layers"]):
        m = L["mixer"]
        if L["type"] == "attention":
            r = m["rot"]
            s = r.get("scaling")
            mask = m.get("mask") or {}
            mixer = AttentionMixer(
                heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                vdim=int(m["vdim"]), scale=float(m["scale"]),
                rot=Rotary(int(r["dims"]), float(r["base"]),
                           Yarn(float(s["factor"]), float(s["original"]), float(s["fast"]),
                                float(s["slow"])) if s else None),
                window=int(mask.get("size") or 0), keep=int(mask.get("keep_first") or 0))
        elif L["type"] == "gla":
            mixer = GlaMixer(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                             tau=float(m["tau"]))
        else:
            raise ValueError(f"layer {i}: unknown mixer {L['type']!r}")
        f = L.get("mlp")
        if f is None:
            mlp = None
        elif f["kind"] == "dense":
            mlp = DenseMlp(int(f["ff"]))
        elif f["kind"] == "moe":
            mlp = MoeMlp(int(f["router"]["experts"]), int(f["router"]["top"]),
                         int(f["expert"]["ff"]))
        else:
            raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
        layers.append(HybridLayer(mixer, mlp))
    return HybridConfig(architecture="Bovinex", vocab_size=int(d["vocab"]), dim=int(d["width"]),
                        norm_eps=float(d["norm"]["eps"]),
                        embed_scale=float(d["embedding"]["scale"]), layers=layers,
                        norm_offset=1.0)


def read_ruralorn(d: Mapping) -> HybridConfig:
    """Ruralorn: sequential blocks; windowed latent attention with an output gate; sigmoid-routed
    experts that are weighted at their input, beside a shared one; soft-capped logits."""
    layers = []
    for i, L in enumerate(d["layers"]):
        m = L["mixer"]
        if L["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer {L['type']!r}")
        r = m["rot"]
        mixer = LatentMixer(
            heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]),
            vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
            rot=Rotary(int(r["dims"]), float(r["base"]), interleaved=True),
            window=int((m.get("mask") or {}).get("size") or 0))
        f, mlp = L.get("mlp"), None
        if f is not None:
            if f["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
            shared = f.get("shared")
            mlp = MoeMlp(int(f["router"]["experts"]), int(f["router"]["top"]),
                         int(f["expert"]["ff"]), gated=False, act="gelu", score="sigmoid",
                         weight_input=True, bias=False,
                         shared=DenseMlp(int(shared["ff"]), "gelu") if shared else None)
        layers.append(HybridLayer(mixer, mlp))
    scale, cap = d.get("logit_scale"), d.get("logit_softcap")
    return HybridConfig(architecture="Ruralorn", vocab_size=int(d["vocab"]), dim=int(d["width"]),
                        norm_eps=float(d["norm"]["eps"]),
                        embed_scale=float(d["embedding"]["scale"]), layers=layers, parallel=False,
                        logit_scale=1.0 if scale is None else float(scale),
                        logit_softcap=0.0 if cap is None else float(cap))


# ------------------------------------------------------------------------------ weights

class _Stack:
    """Matrices below one another, every one from a multiple of 8 rows on."""

    def __init__(self):
        self.parts, self.n = [], 0

    def add(self, t: torch.Tensor, bias: Optional[torch.Tensor] = None) -> int:
        at = self.n
        self.parts.append((at, t, bias))
        self.n += pad8(t.shape[0])
        return at


def _pad_heads(t: torch.Tensor, heads: int, sizes) -> torch.Tensor:
    """[heads * sum(sizes), ...] -> every part of every head filled up to a multiple of 8 rows."""
    parts = t.view(heads, sum(sizes), *t.shape[1:]).split(list(sizes), 1)
    out = []
    for p, n in zip(parts, sizes):
        z = p.new_zeros(heads, pad8(n), *t.shape[1:])
        z[:, :n] = p
        out.append(z)
    return torch.cat(out, 1).flatten(0, 1)

class HybridBlock(nn.Module):
    """One layer's weights in kernel layout. Column offsets of the packed activation: ``off_q``,
    ``off_k`` (or ``off_c``: latent and shared key part), ``off_v``, ``off_g`` (gate, then gated
    heads) and, in a parallel block, ``off_u`` (dense up); it is ``f_main`` columns wide. ``n_tail``
    fp32 columns: decay input at 0, router (parallel block) at ``off_r``. A sequential block has
    ``f_ff`` columns of up projection and ``n_ff_tail`` fp32 columns (router at ``off_r``)."""

    def __init__(self, layer: HybridLayer, cfg: HybridConfig, get: Callable, device, dtype):
        super().__init__()
        self.layer = layer
        m, f = layer.mixer, layer.mlp
        W = cfg.dim
        kp = pad8(W)

        def fp32(name, n):
            return get(name, (n,)).to(device=device, dtype=torch.float32).contiguous()

        def lin(name, *shape):
            return get(name, shape).to(device=device, dtype=dtype)

        main, tail = _Stack(), _Stack()
        heads_out = getattr(self, "_" + m.kind)(m, main, tail, fp32, lin, get, W)
        ff, ff_tail = (main, tail) if cfg.parallel else (_Stack(), _Stack())
        # the feed-forward every token runs: a dense one, or the shared expert
        dense, name = (f, "mlp.") if f is None or f.kind == "dense" else (f.shared, "mlp.shared.")
        self.act = dense.act if dense is not None else None
        self.off_u = ff.n
        if dense is not None:
            ff.add(lin(name + "up", dense.ff, W))
        self.off_r = ff_tail.n
        if f is not None and f.kind == "moe":
            ff_tail.add(lin("mlp.router", f.experts, W),
                        fp32("mlp.router.b", f.experts) if f.bias else None)

        def stack(name, a, b):
            w = torch.zeros(a.n + b.n, kp, dtype=dtype, device=device)
            bias = torch.zeros(a.n + b.n, dtype=torch.float32, device=device)
            some = False
            for base, st in ((0, a), (a.n, b)):
                for at, t, v in st.parts:
                    w[base + at: base + at + t.shape[0], :W] = t
                    if v is not None:
                        bias[base + at: base + at + t.shape[0]] = v
                        some = True
            self._weight("w_" + name, w, W)
            self.register_buffer("b_" + name, bias if some else None)

        self.f_main, self.n_tail = main.n, tail.n
        stack("in", main, tail)
        self.f_ff = self.n_ff_tail = 0
        if not cfg.parallel and f is not None:
            self.f_ff, self.n_ff_tail = ff.n, ff_tail.n
            stack("ff", ff, ff_tail)
            if dense is not None:
                w = torch.zeros(W, self.f_ff, dtype=dtype, device=device)
                w[:, : dense.ff] = lin(name + "down", W, dense.ff)
                self._weight("w_down", w, self.f_ff)
        # output side: gated heads (+ filling), in a parallel block next to the activated up projection
        ko = self.f_main - self.off_g
        w_out = torch.zeros(W, ko, dtype=dtype, device=device)
        w_out[:, : heads_out.shape[1]] = heads_out
        if cfg.parallel and dense is not None:
            c = self.off_u - self.off_g
            w_out[:, c: c + dense.ff] = lin(name + "down", W, dense.ff)
        self._weight("w_out", w_out, ko)
        self.register_buffer("norm1", fp32("norm1", W))
        if not cfg.parallel and f is not None:
            self.register_buffer("norm2", fp32("norm2", W))
        if f is not None and f.kind == "moe":
            fp = pad8(f.ff)
            self.ffp = fp
            up = torch.zeros(f.experts * fp, kp, dtype=dtype, device=device)
            gate = torch.zeros_like(up) if f.gated else None
            down = torch.zeros(f.experts * W, fp, dtype=dtype, device=device)
            for e in range(f.experts):
                for dst, part in ((gate, "gate"), (up, "up")):
                    if dst is not None:
                        dst[e * fp: e * fp + f.ff, :W] = lin(f"mlp.e{e}.{part}", f.ff, W)
                down[e * W: (e + 1) * W, : f.ff] = lin(f"mlp.e{e}.down", W, f.ff)
            if f.gated:
                self._weight("e_gate", gate, W)
            self._weight("e_up", up, W)
            self._weight("e_down", down, fp)

    # A mixer's projections go to the stacks, its own tensors to the block; returns the output
    # projection's columns in the order of the gated heads.

    def _attention(self, m, main, tail, fp32, lin, get, W):
        sizes = (m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim)
        self.off_q, self.off_k, self.off_v = (
            main.add(lin(n, rows, W), fp32(n + ".b", rows))
            for n, rows in zip(("mix.q", "mix.k", "mix.v"), sizes))
        self.off_g = main.add(lin("mix.g", m.heads * m.vdim, W))
        self.register_buffer("q_norm", fp32("mix.q.norm", m.heads * m.dim))
        self.register_buffer("k_norm", fp32("mix.k.norm", m.kv_heads * m.dim))
        return lin("mix.o", W, m.heads * m.vdim)

    def _gla(self, m, main, tail, fp32, lin, get, W):
        self.off_q, self.off_k, self.off_v, self.off_g = (
            main.add(lin(n, m.heads * d, W)) for n, d in
            (("mix.q", m.dim), ("mix.k", m.dim), ("mix.v", m.vdim), ("mix.g", m.vdim)))
        m.rank = m.rank or int(get("mix.a1", None).shape[0])
        tail.add(lin("mix.a1", m.rank, W))
        self.register_buffer("a2", lin("mix.a2", m.heads * m.dim, m.rank).contiguous())
        self.register_buffer("a2_b", fp32("mix.a2.b", m.heads * m.dim))
        self.register_buffer("o_norm", fp32("mix.norm", m.vdim))
        return lin("mix.o", W, m.heads * m.vdim)

    def _latent(self, m, main, tail, fp32, lin, get, W):
        H, r, rp = m.heads, m.kv_rank, pad8(m.kv_rank)
        self.off_q = main.add(_pad_heads(lin("mix.q", H * (m.dim + m.rot_dim), W), H,
                                         (m.dim, m.rot_dim)))
        self.off_c = main.add(_pad_heads(lin("mix.dkv", r + m.rot_dim, W), 1, (r, m.rot_dim)))
        self.off_g = main.add(_pad_heads(lin("mix.g", H * m.vdim, W), H, (m.vdim,)))
        self.register_buffer("c_norm", _pad_heads(fp32("mix.dkv.norm", r), 1, (r,)))
        uk = _pad_heads(lin("mix.uk", H * m.dim, r), H, (m.dim,))
        uv = _pad_heads(lin("mix.uv", H * m.vdim, r), H, (m.vdim,))
        kv = uk.new_zeros(uk.shape[0] + uv.shape[0], rp)
        kv[:, :r] = torch.cat([uk, uv])
        self.register_buffer("w_kv", kv)                   # key and value expansion
        # the key expansion absorbed into the queries: [rank, dim] per head
        self.register_buffer("w_uk_t", kv[: uk.shape[0]].view(H, -1, rp).transpose(1, 2)
                             .reshape(H * rp, -1).contiguous())
        return _pad_heads(lin("mix.o", W, H * m.vdim).t(), H, (m.vdim,)).t()

    def _weight(self, name: str, t: torch.Tensor, cols: int) -> None:
        """Rows keep a stride that is a multiple of 8 elements; ``cols`` of them are weights."""
        self.register_buffer(name, t)
        setattr(self, name + "_k", cols)

    def mat(self, name: str) -> torch.Tensor:
        return getattr(self, name)[:, : getattr(self, name + "_k")]


class HybridLM(nn.Module):
    """Weights of a hybrid decoder. Generation runs on ``models.hybrid_engine.HybridEngine``."""

    tp_size = 1
    vocab_parallel = False

    def __init__(self, config: HybridConfig, get: Callable, device="cuda",
                 dtype=torch.bfloat16):
        """``get(name, shape)`` returns the tensor of that name (any device / dtype); shape None
        asks for whatever shape it has."""
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"hybrid decoders run in bfloat16 or float32, not {dtype}")
        _check(config)
        self.config, self.dtype = config, dtype
        W, kp = config.dim, pad8(config.dim)
        vp = pad8(config.vocab_size)
        self.register_buffer("embed", get("embed", (config.vocab_size, W)).to(
            device=device, dtype=dtype).contiguous())
        self.layers = nn.ModuleList(
            HybridBlock(L, config, lambda n, s, p=f"l{i}.": get(p + n, s), device, dtype)
            for i, L in enumerate(config.layers))
        self.register_buffer("norm", get("final.norm", (W,)).to(
            device=device, dtype=torch.float32).contiguous())
        head = torch.zeros(vp, kp, dtype=dtype, device=device)
        head[: config.vocab_size, :W] = get("head", (config.vocab_size, W)).to(
            device=device, dtype=dtype)
        self.register_buffer("head_w", head)

    @property
    def device(self) -> torch.device:
        return self.embed.device

    @classmethod
    def from_tensors(cls, config: HybridConfig, tensors: Mapping[str, torch.Tensor], **kw):
        def get(name, shape):
            if name not in tensors:
                raise KeyError(f"the checkpoint has no tensor {name!r}")
            t = tensors[name]
            if shape is not None and tuple(t.shape) != tuple(shape):
                raise ValueError(f"tensor {name!r} has shape {tuple(t.shape)}, "
                                 f"expected {tuple(shape)}")
            return t
        return cls(config, get, **kw)

    @classmethod
    def random(cls, config: HybridConfig, seed: int = 0, std: float = 0.02, device="cuda",
               dtype=torch.bfloat16):
        """Random weights (benchmarks); recurrent layers need ``rank`` set in their mixer."""
        g = torch.Generator(device=device).manual_seed(seed)
        rank = {f"l{i}.mix.a1": (L.mixer.rank, config.dim) for i, L in enumerate(config.layers)
                if L.mixer.kind == "gla"}

        def get(name, shape):
            t = torch.empty(shape or rank[name], dtype=dtype, device=device)
            return t.normal_(0.0, std, generator=g)
        return cls(config, get, device=device, dtype=dtype)

    def make_engine(self, batch_size: int, seq_length: int, **kw):
        from .hybrid_engine import HybridEngine
        return HybridEngine(self, batch_size, seq_length, **kw)

    def forward(self, *a, **kw):
        raise RuntimeError("hybrid decoders have no module forward: generation and scoring run on "
                           "their CUDA engine (models.engine.get_engine)")


def _check(cfg: HybridConfig) -> None:
    for i, L in enumerate(cfg.layers):
        m, f = L.mixer, L.mlp
        if m.kind == "latent":
            if m.kv_rank > 1024 or m.rot_dim > 256:
                raise ValueError(f"layer {i}: latents above 1024 or rotated parts above 256 columns "
                                 "are not supported")
            if m.rot_dim % 2 or m.rot.dims % 2 or m.rot.dims > m.rot_dim or not m.rot.interleaved:
                raise ValueError(f"layer {i}: cannot rotate {m.rot.dims} of {m.rot_dim} dimensions")
        elif m.dim > 256 or (m.kind == "attention" and m.vdim > 256):
            raise ValueError(f"layer {i}: head sizes above 256 are not supported")
        if m.kind == "attention":
            if m.heads % m.kv_heads:
                raise ValueError(f"layer {i}: {m.heads} query heads over {m.kv_heads} kv heads")
            if m.rot.dims % 2 or m.rot.dims > m.dim or m.rot.interleaved:
                raise ValueError(f"layer {i}: cannot rotate {m.rot.dims} of {m.dim} dimensions")
        if f is not None and f.kind == "moe" and not 1 <= f.top <= min(f.experts, 16):
            raise ValueError(f"layer {i}: top {f.top} of {f.experts} experts is not supported")


# ------------------------------------------------------------------------------ registry

HYBRID_DESIGNS: Dict[str, Callable[[Mapping], HybridConfig]] = {"Bovinex": read_bovinex,
                                                                  "Ruralorn": read_ruralorn}


def hybrid_config(d: Mapping) -> HybridConfig:
    name = d.get("architecture")
    if name not in HYBRID_DESIGNS:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(HYBRID_DESIGNS)}")
    return HYBRID_DESIGNS[name](d)


def kernel_sources(cfg: HybridConfig) -> List[str]:
    """Stems of the CUDA sources that a design's layers run on (all precisions)."""
    names = {"gemm_umma", "gemm_persistent", "gemm_f32", "stream_norm"}
    for L in cfg.layers:
        names |= {"attention": {"attn_window", "flash_window"}, "gla": {"gla", "gla_chunk"},
                  "latent": {"latent_attn", "flash_window"}}[L.mixer.kind]
        if L.mlp is not None and L.mlp.kind == "moe":
            names.add("moe")
    return sorted(names)


def config_in(folder: Union[str, Path]) -> Optional[dict]:
    """The parsed ``config.json`` of a checkpoint folder if it names one of the registered
    designs, else None (the folder then holds a gpt-fast checkpoint)."""
    path = Path(folder) / "config.json"
    if not path.is_file():
        return None
    with open(path) as fh:
        d = json.load(fh)
    return d if isinstance(d, dict) and d.get("architecture") in HYBRID_DESIGNS else None


def load_hybrid(folder: Union[str, Path], device="cuda", dtype=torch.bfloat16) -> HybridLM:
    from ..utils.safetensors_io import load_safetensors
    d = config_in(folder)
    if d is None:
        raise ValueError(f"{folder}: config.json names no registered design")
    return HybridLM.from_tensors(hybrid_config(d),
                                 load_safetensors(Path(folder) / "model.safetensors"),
                                 device=device, dtype=dtype).eval()
