"""Shared by the Bizenex tests: small configurations of their own (sizes chosen so that nothing that could be equal is equal:
key and value head sizes, heads and key/value heads, latent and head sizes; temperatures that step at every position, inside
a page and beyond it; readers of one owner side by side; groups of one expert, of two and of several, all groups kept; `top`
of one, of several and of all), model folders with random weights in which some tensors are set by hand so that what they do
shows, and the comparison with the plain implementation."""
from __future__ import annotations

import functools
import os
from typing import Dict, Sequence

import torch

import helpers
import mini_llama_cpp_release_b200 as ml
import plain_bizenex as pb
from kebesun_helpers import check  # noqa: F401  (the same bounds on rows of logits)
from mini_llama_cpp_release_b200.config import ModelConfig


def attention(heads, kv_heads, dim, vdim, scale, coef=None, every=1):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if coef is not None:
        m["q_temp"] = {"coef": coef, "every": every}
    return m


def latent(heads, dim, vdim, kv_rank, scale, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def moe(ff, experts, top, groups=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = dict(zip(("count", "keep"), groups))
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def layer(mixer, mlp=None):
    return {"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, eps, cap, layers):
    return {"architecture": "Bizenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


# both mixers, with and without experts; layers 2 and 4 read layer 1's latents, one with more heads and other head sizes
MIXED = model(300, 112, 1e-5, 12.0, [
    layer(attention(6, 3, 24, 40, 0.3, 0.4, 20), moe(48, 6, 2, (3, 2))),
    layer(latent(5, 16, 24, 40, 0.25), moe(32, 9, 4, (3, 2))),
    layer(latent(7, 8, 36, 40, 0.4, kv_from=1), None),
    layer(attention(4, 1, 48, 16, 0.2, 0.8, 1), moe(40, 5, 5)),
    layer(latent(5, 32, 12, 40, 0.15, kv_from=1), moe(24, 8, 1, (2, 1))),
])

# heads of 64 and 128 entries (the tensor-core attention kernels of prompts), latent rows of 64 and 128, a reader of each
WIDE = model(257, 128, 2e-6, 20.0, [
    layer(latent(4, 32, 64, 128, 0.17), moe(64, 8, 3, (4, 3))),
    layer(attention(4, 2, 64, 64, 0.2, 0.3, 64), moe(80, 12, 2, (4, 2))),
    layer(latent(3, 48, 32, 64, 0.14), None),
    layer(attention(2, 2, 128, 96, 0.11, 1.5, 100), moe(64, 4, 4, (2, 2))),
    layer(latent(18, 16, 16, 64, 0.3, kv_from=2), moe(48, 16, 3, (8, 3))),
    layer(latent(2, 64, 80, 128, 0.1, kv_from=0), moe(64, 8, 2)),
])

# sizes the fast paths do not take: a width and feed-forwards that are no multiples of 8, a latent of three entries and one of
# more than 256, groups of one expert each, 33 experts, no temperature, no cap on the logits
ODD = model(77, 100, 1e-5, None, [
    layer(attention(5, 5, 12, 10, 0.5), moe(20, 3, 3)),
    layer(latent(3, 6, 10, 3, 0.6), moe(12, 4, 2, (4, 3))),
    layer(latent(2, 20, 14, 270, 0.2), None),
    layer(latent(4, 10, 6, 270, 0.3, kv_from=2), moe(28, 7, 1)),
    layer(attention(3, 1, 20, 28, 0.3, 0.2, 7), moe(20, 33, 3, (11, 4))),
])

TINY_MIXER = attention(1, 1, 8, 8, 0.5)
ONLY_ATTENTION = model(200, 64, 1e-5, 10.0, [layer(attention(6, 2, 20, 28, 0.3, 0.5, 33))])
ONLY_LATENT = model(200, 64, 1e-5, 10.0, [layer(latent(6, 20, 28, 48, 0.3))])
ONLY_MOE = model(200, 64, 1e-5, 10.0, [layer(TINY_MIXER, moe(40, 12, 3, (4, 2)))])
SHARED = model(150, 64, 1e-5, 8.0, [layer(latent(4, 16, 24, 32, 0.3)), layer(latent(3, 24, 16, 32, 0.25, kv_from=0)),
                                    layer(latent(6, 8, 8, 32, 0.4, kv_from=0))])

CONFIGS = {"mixed": MIXED, "wide": WIDE, "odd": ODD, "attention": ONLY_ATTENTION, "latent": ONLY_LATENT, "moe": ONLY_MOE,
           "shared": SHARED}


def shape_weights(weights: Dict[str, torch.Tensor], seed: int, peaked: float = 1.0) -> None:
    """Random weights hide some faults.  The norms' biases are spread out, the sinks weigh as much as a key or more (a sink
    that is left out, scaled or counted twice shows), the output gates lie away from one half, routers are made decisive (so
    that the chosen experts do not hang on the last bit), and with `peaked` the latent layers' query matrices are scaled so
    that single keys decide rows (the attention layers' queries are normed: their scale is the configuration's)."""
    g = torch.Generator().manual_seed(seed)
    for name, t in weights.items():
        if name.endswith((".norm1.b", ".norm2.b", "final.norm.b")):
            t.copy_(torch.randn(t.shape, generator=g) * 0.3)
        elif name.endswith(".mix.sink"):
            t.copy_(torch.randn(t.shape, generator=g) * 1.5 + 2.0)
        elif name.endswith(".mix.g"):
            t.mul_(3.0)
        elif name.endswith(".router"):
            t.mul_(6.0)
        elif name.endswith(".mix.q") and peaked != 1.0:
            t.mul_(peaked)
        elif name.endswith(".mix.o"):
            t.mul_(2.0)


@functools.lru_cache(maxsize=None)
def folder_of(name: str, seed: int = 1, std: float = 0.08, peaked: float = 1.0) -> str:
    from safetensors.torch import load_file, save_file
    folder = os.path.join(helpers.tmp_root(), f"bizenex_{name}_{seed}_{std}_{peaked}")
    raw = CONFIGS[name]
    if peaked != 1.0:              # normed queries: their scores are sharpened by the scale
        raw = dict(raw, layers=[dict(l, mixer=dict(l["mixer"], scale=l["mixer"]["scale"] * peaked)) if l["type"] == "attention" else l
                                for l in raw["layers"]])
    ml.write_random_model(ModelConfig.from_dict(raw), folder, seed, torch.bfloat16, std=std)
    path = os.path.join(folder, "model.safetensors")
    weights = {k: v.float() for k, v in load_file(path).items()}
    shape_weights(weights, seed, peaked)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in weights.items()}, path)
    return folder


@functools.lru_cache(maxsize=None)
def oracle(folder: str):
    return pb.read_config(folder), pb.read_weights(folder, torch.float64)


def oracle_logits(folder: str, tokens: Sequence[int]) -> torch.Tensor:
    cfg, w = oracle(folder)
    return pb.forward(cfg, w, tokens).float()
