"""Hybrid decoders: models whose layers mix attention with recurrent mixers and dense with
mixture-of-experts feed-forwards, described layer by layer in a ``config.json``.

A design is a reader that turns its ``config.json`` into the generic description below (mixers,
feed-forwards, rotation, masks, norms, each with its constants as parameters); everything
underneath -- weight packing, the slot cache, the engine and the kernels -- is shared. Adding a
design means adding a reader (and the mechanisms it has that no other design has).

The module holds the weights in the layout the engine's kernels read. With a parallel block (mixer
and feed-forward read one norm and are added together) a layer is two products:

* ``w_in``   q, k, v, gate and the dense up projection stacked as one ``[F, width]`` matrix, with
  fp32 tail rows (low-rank decay input, router) that leave the GEMM unrounded;
* ``w_out``  ``[width, gated heads + ff]``: output projection and down projection side by side,
  reading the gated heads and the activated up projection where ``w_in`` left them.

Segments start at multiples of 8 columns; the filling rows / columns are zero.
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
    dims: int                     # leading dimensions of a head that rotate (half layout)
    base: float
    scaling: Optional[Yarn] = None

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

    def table(self, length: int, device=None) -> torch.Tensor:
        """fp32 ``[length, dims / 2, 2]`` of (cos, sin), computed in double precision."""
        freq, amp = self.frequencies()
        ang = torch.outer(torch.arange(length, dtype=torch.float64), freq)
        return torch.stack([amp * torch.cos(ang), amp * torch.sin(ang)], -1).float().to(device)


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
    act: str = "relu2"            # w_down act(w_up h)
    kind: str = "dense"


@dataclass
class MoeMlp:
    experts: int
    top: int
    ff: int                       # w_down (silu(w_gate h) * w_up h) per expert
    kind: str = "moe"


@dataclass
class HybridLayer:
    mixer: Union[AttentionMixer, GlaMixer]
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


# ------------------------------------------------------------------------------ weights

class HybridBlock(nn.Module):
    """One layer's weights in kernel layout. Column offsets of the packed activation: ``off_q``,
    ``off_k``, ``off_v``, ``off_g`` (gate, then gated heads) and ``off_u`` (dense up); it is
    ``f_main`` columns wide. ``tail``: fp32 columns -- decay input at 0, router at ``off_r``."""

    def __init__(self, layer: HybridLayer, cfg: HybridConfig, get: Callable, device, dtype):
        super().__init__()
        self.layer = layer
        m, f = layer.mixer, layer.mlp
        W = cfg.dim
        kp = pad8(W)
        att = m.kind == "attention"
        kv = m.kv_heads if att else m.heads

        def fp32(name, n):
            return get(name, (n,)).to(device=device, dtype=torch.float32).contiguous()

        segs, at = [], 0
        for name, rows in (("mix.q", m.heads * m.dim), ("mix.k", kv * m.dim),
                           ("mix.v", kv * m.vdim), ("mix.g", m.heads * m.vdim)):
            segs.append((name, at, rows))
            at += pad8(rows)
        self.off_q, self.off_k, self.off_v, self.off_g = (s[1] for s in segs)
        self.off_u = at
        if f is not None and f.kind == "dense":
            segs.append(("mlp.up", at, f.ff))
            at += pad8(f.ff)
        self.f_main = at
        tail = 0
        if not att:
            m.rank = m.rank or int(get("mix.a1", None).shape[0])
            segs.append(("mix.a1", at, m.rank))
            tail = pad8(m.rank)
        self.off_r = tail
        if f is not None and f.kind == "moe":
            segs.append(("mlp.router", at + tail, f.experts))
            tail += pad8(f.experts)
        self.n_tail = tail
        w_in = torch.zeros(at + tail, kp, dtype=dtype, device=device)
        for name, row, rows in segs:
            w_in[row: row + rows, :W] = get(name, (rows, W)).to(device=device, dtype=dtype)
        self._weight("w_in", w_in, W)
        bias = None
        if att or tail > (pad8(m.rank) if not att else 0):
            bias = torch.zeros(at + tail, dtype=torch.float32, device=device)
            for name, row, rows in segs:
                if (att and name in ("mix.q", "mix.k", "mix.v")) or name == "mlp.router":
                    bias[row: row + rows] = fp32(name + ".b", rows)
        self.register_buffer("b_in", bias)
        # output side: gated heads (+ filling) next to the activated up projection
        ko = self.f_main - self.off_g
        w_out = torch.zeros(W, ko, dtype=dtype, device=device)
        w_out[:, : m.heads * m.vdim] = get("mix.o", (W, m.heads * m.vdim)).to(device=device,
                                                                              dtype=dtype)
        if f is not None and f.kind == "dense":
            c = self.off_u - self.off_g
            w_out[:, c: c + f.ff] = get("mlp.down", (W, f.ff)).to(device=device, dtype=dtype)
        self._weight("w_out", w_out, ko)
        self.register_buffer("norm1", fp32("norm1", W))
        if att:
            self.register_buffer("q_norm", fp32("mix.q.norm", m.heads * m.dim))
            self.register_buffer("k_norm", fp32("mix.k.norm", kv * m.dim))
        else:
            self.register_buffer("a2", get("mix.a2", (m.heads * m.dim, m.rank)).to(
                device=device, dtype=dtype).contiguous())
            self.register_buffer("a2_b", fp32("mix.a2.b", m.heads * m.dim))
            self.register_buffer("o_norm", fp32("mix.norm", m.vdim))
        if f is not None and f.kind == "moe":
            fp = pad8(f.ff)
            self.ffp = fp
            gate = torch.zeros(f.experts * fp, kp, dtype=dtype, device=device)
            up = torch.zeros_like(gate)
            down = torch.zeros(f.experts * W, fp, dtype=dtype, device=device)
            for e in range(f.experts):
                for dst, name in ((gate, "gate"), (up, "up")):
                    dst[e * fp: e * fp + f.ff, :W] = get(f"mlp.e{e}.{name}", (f.ff, W)).to(
                        device=device, dtype=dtype)
                down[e * W: (e + 1) * W, : f.ff] = get(f"mlp.e{e}.down", (W, f.ff)).to(
                    device=device, dtype=dtype)
            self._weight("e_gate", gate, W)
            self._weight("e_up", up, W)
            self._weight("e_down", down, fp)

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
        if m.dim > 256 or (m.kind == "attention" and m.vdim > 256):
            raise ValueError(f"layer {i}: head sizes above 256 are not supported")
        if m.kind == "attention":
            if m.heads % m.kv_heads:
                raise ValueError(f"layer {i}: {m.heads} query heads over {m.kv_heads} kv heads")
            if m.rot.dims % 2 or m.rot.dims > m.dim:
                raise ValueError(f"layer {i}: cannot rotate {m.rot.dims} of {m.dim} dimensions")
        if f is not None and f.kind == "moe" and not 1 <= f.top <= min(f.experts, 16):
            raise ValueError(f"layer {i}: top {f.top} of {f.experts} experts is not supported")


# ------------------------------------------------------------------------------ registry

HYBRID_DESIGNS: Dict[str, Callable[[Mapping], HybridConfig]] = {"Bovinex": read_bovinex}


def hybrid_config(d: Mapping) -> HybridConfig:
    name = d.get("architecture")
    if name not in HYBRID_DESIGNS:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(HYBRID_DESIGNS)}")
    return HYBRID_DESIGNS[name](d)


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
