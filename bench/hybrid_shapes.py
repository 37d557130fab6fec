"""Layer shapes of the hybrid-decoder benchmarks: Bovinex and Ruralorn configurations whose layers
resemble a real model's, LLaMA configurations of the size of the Bovinex ones (same width, query
heads, kv heads, layers and active feed-forward parameters), and Bovinex configurations of the size of
the Ruralorn ones (attention and expert layers only; same width, query heads, window, experts and
active feed-forward parameters)."""
from __future__ import annotations

import os
import sys

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

SIZES = {
    # width, heads, kv heads, window, gla heads, dense ff, experts, top, expert ff, llama ff, vocab
    "2k": (2048, 16, 4, 1024, 8, 8192, 8, 2, 2752, 5504, 32000),
    "4k": (4096, 32, 8, 2048, 16, 16384, 8, 2, 5504, 11008, 32000),
}


def bovinex_config(size: str, layers: int = 8, attention_only: bool = False):
    """attention + dense, gla + experts, gla + dense, attention + experts, repeated; or attention +
    experts only."""
    from easy_to_hard_b200.models.hybrid import (AttentionMixer, DenseMlp, GlaMixer, HybridConfig,
                                                 HybridLayer, MoeMlp, Rotary, Yarn)
    W, H, G, win, gh, ff, E, top, eff, _, vocab = SIZES[size]

    def att():
        return AttentionMixer(H, G, 128, 128, 128 ** -0.5,
                              Rotary(128, 1e6, Yarn(4.0, 4096, 32.0, 1.0)), win, 4)

    def gla():
        return GlaMixer(gh, 128, 256, 16.0, 16)
    kinds = [(att, DenseMlp(ff)), (gla, MoeMlp(E, top, eff)), (gla, DenseMlp(ff)),
             (att, MoeMlp(E, top, eff))]
    if attention_only:
        kinds = kinds[3:] * 4
    return HybridConfig("Bovinex", vocab, W, 1e-5, W ** 0.5,
                        [HybridLayer(kinds[i % 4][0](), kinds[i % 4][1]) for i in range(layers)],
                        norm_offset=1.0)


def bovinex_model(size: str, layers: int = 8):
    from easy_to_hard_b200.models.hybrid import HybridLM
    return HybridLM.random(bovinex_config(size, layers))


def bovinex_attention_model(size: str, layers: int = 8):
    from easy_to_hard_b200.models.hybrid import HybridLM
    return HybridLM.random(bovinex_config(size, layers, attention_only=True))


# latent rank, dim, rotated dim, value dim of a head; expert ff and shared ff (two matrices each) with
# as many active parameters as the gated experts of the Bovinex shapes
LATENT = (512, 128, 64, 128)
RURALORN_FF = {"2k": (3440, 1376), "4k": (6880, 2752)}


def ruralorn_config(size: str, layers: int = 8):
    from easy_to_hard_b200.models.hybrid import (DenseMlp, HybridConfig, HybridLayer, LatentMixer,
                                                 MoeMlp, Rotary)
    W, H, _, win, _, _, E, top, _, _, vocab = SIZES[size]
    rank, dim, rot, vdim = LATENT
    ff, shared = RURALORN_FF[size]

    def layer():
        return HybridLayer(LatentMixer(H, dim, rot, vdim, rank, (dim + rot) ** -0.5,
                                       Rotary(rot, 1e6, interleaved=True), win),
                           MoeMlp(E, top, ff, gated=False, act="gelu", score="sigmoid",
                                  weight_input=True, bias=False, shared=DenseMlp(shared, "gelu")))
    return HybridConfig("Ruralorn", vocab, W, 1e-5, W ** 0.5, [layer() for _ in range(layers)],
                        parallel=False, logit_scale=0.5, logit_softcap=30.0)


def ruralorn_model(size: str, layers: int = 8):
    from easy_to_hard_b200.models.hybrid import HybridLM
    return HybridLM.random(ruralorn_config(size, layers))


def llama_model(size: str, layers: int = 8):
    import torch
    from easy_to_hard_b200.models.model import ModelArgs, Transformer
    W, H, G, _, _, _, _, _, _, ff, vocab = SIZES[size]
    cfg = ModelArgs(block_size=8192, vocab_size=vocab, n_layer=layers, n_head=H, dim=W,
                    intermediate_size=ff, n_local_heads=G, rope_base=1000000)
    with torch.device("cuda"):
        m = Transformer(cfg, freeze_tok_embeddings=True, freeze_output=True,
                        freeze_norm=True).to(torch.bfloat16)
    g = torch.Generator(device="cuda").manual_seed(0)
    for t in list(m.parameters()) + list(m.buffers()):
        if t.dim() == 2:
            t.data.normal_(0.0, 0.02, generator=g)
    return m.eval()
