"""Shared by the Betepel tests: small configurations of their own (sizes chosen so that nothing that could be equal is equal:
key and value head sizes, heads and key/value heads, experts' and shared experts' sizes; windows below, at and above a page,
kept first tokens inside a page and beyond one; readers of one owner under its mask and under others; rotations that keep,
slow down and mix frequencies; one, several and all experts a token), model folders with random weights in which some tensors
are set by hand so that what they do shows, and the comparison with the plain implementation."""
from __future__ import annotations

import functools
import os
from typing import Dict, Sequence

import torch

import helpers
import mini_llama_cpp_release_b200 as ml
import plain_betepel as pb
from mini_llama_cpp_release_b200.config import ModelConfig


def rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def attention(heads, kv_heads, dim, vdim, scale, diff, rotation, size=None, keep_first=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "rot": rotation}
    if size is not None:
        m["mask"] = {"size": size, "keep_first": keep_first or 0}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def parallel(left, right, left_scale, right_scale):
    heads, kv_heads, dim, vdim, scale, rotation, size = left
    return {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rotation,
                     "mask": {"size": size}},
            "right": dict(zip(("decay", "dim", "vdim"), right), heads=len(right[0])),
            "left_scale": left_scale, "right_scale": right_scale}


def mlstm(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def moe(ff, experts, top, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp=None):
    return {"type": "parallel" if "left" in mixer else "mlstm" if "gate_cap" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, eps, logit_scale, layers):
    return {"architecture": "Betepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


SLOW = (4.0, 1.5, 5.0, 100)              # over 100 positions: some pairs keep their frequency, some are slowed down, some between

# every mixer, with and without experts; layer 3 reads layer 0's keys under the same mask, layer 5 under another one
MIXED = model(300, 112, 1e-5, 1.5, [
    layer(attention(6, 3, 24, 40, 0.3, 0.4, rot(12, 1000.0, SLOW), 30, 7), moe(48, 6, 2, 56)),
    layer(parallel((4, 2, 20, 28, 0.3, rot(16, 500.0), 21), ((0.9, 0.3, 0.995), 24, 12), 0.7, 1.3), moe(40, 5, 1, 24)),
    layer(mlstm(3, 20, 28, 12.0), None),
    layer(attention(6, 3, 24, 40, 0.25, 0.7, rot(12, 1000.0, SLOW), 30, 7, kv_from=0), moe(32, 7, 3)),
    layer(mlstm(2, 36, 20, 6.0), moe(24, 4, 4, 72)),
    layer(attention(3, 3, 24, 40, 0.35, 0.2, rot(12, 1000.0, SLOW), 50, 3, kv_from=0), moe(56, 9, 2, 40)),
])

# heads of 64 and 128 entries (the tensor-core attention kernels of prompts), memories of up to 128 x 128
WIDE = model(257, 128, 2e-6, 0.8, [
    layer(attention(6, 3, 32, 64, 0.2, 0.5, rot(32, 10000.0, (6.0, 1.0, 3.0, 256)), 64, 18), moe(64, 8, 2, 96)),
    layer(parallel((4, 1, 64, 48, 0.15, rot(64, 10000.0), 65), ((0.99, 0.6), 64, 96), 1.2, 0.6), moe(80, 12, 1, 64)),
    layer(mlstm(2, 128, 64, 13.0), moe(64, 3, 3, 128)),
    layer(attention(2, 2, 64, 128, 0.12, 0.8, rot(24, 1000000.0, (2.0, 2.0, 3.0, 64)), 100, 70), None),
    layer(attention(10, 2, 64, 128, 0.14, 0.3, rot(24, 1000000.0, (2.0, 2.0, 3.0, 64)), kv_from=3), moe(48, 16, 5, 48)),
    layer(mlstm(4, 32, 128, 4.0), moe(64, 8, 2, 64)),
])

# sizes the fast paths do not take: a width and feed-forwards that are no multiples of 8, value heads wider than two key
# heads, key rows of more than 256 entries, heads of one, no rotation, no mask, no scaling, a window of one, one expert
ODD = model(77, 100, 1e-5, 3.0, [
    layer(attention(5, 5, 6, 18, 0.6, 0.35, rot(4, 300.0), 9, 2), moe(20, 3, 3, 12)),
    layer(parallel((3, 3, 10, 6, 0.5, rot(0, 1.0), 1), ((0.8,), 5, 7), -0.9, 2.1), moe(12, 1, 1, 20)),
    layer(mlstm(3, 5, 7, 2.0), moe(28, 5, 2)),
    layer(attention(2, 1, 136, 30, 0.1, 0.6, rot(136, 5000.0, (3.0, 1.0, 2.0, 50)), 40), None),
    layer(mlstm(1, 200, 33, 9.0), moe(20, 33, 3, 36)),
    layer(attention(4, 1, 136, 30, 0.09, -0.2, rot(136, 5000.0, (3.0, 1.0, 2.0, 50)), 25, 70, kv_from=3), moe(20, 4, 2, 8)),
])

TINY_MIXER = mlstm(1, 8, 8, 5.0)
ONLY_ATTENTION = model(200, 64, 1e-5, 2.0, [layer(attention(6, 2, 20, 28, 0.3, 0.5, rot(12, 2000.0, SLOW), 45, 5))])
ONLY_PARALLEL = model(200, 64, 1e-5, 2.0, [layer(parallel((6, 2, 20, 28, 0.3, rot(20, 2000.0), 33), ((0.95, 0.5, 0.999, 0.7), 20, 12), 1.25, 0.85))])
ONLY_MLSTM = model(200, 64, 1e-5, 2.0, [layer(mlstm(4, 20, 28, 14.0))])
ONLY_MOE = model(200, 64, 1e-5, 2.0, [layer(TINY_MIXER, moe(40, 12, 3, 32))])
SHARED = model(150, 64, 1e-5, 1.0, [layer(attention(4, 2, 16, 24, 0.3, 0.5, rot(16, 1000.0, SLOW), 20, 6)),
                                    layer(attention(2, 2, 16, 24, 0.35, 0.3, rot(16, 1000.0, SLOW), 20, 6, kv_from=0)),
                                    layer(attention(6, 2, 16, 24, 0.25, 0.6, rot(16, 1000.0, SLOW), 90, 0, kv_from=0))])

CONFIGS = {"mixed": MIXED, "wide": WIDE, "odd": ODD, "attention": ONLY_ATTENTION, "parallel": ONLY_PARALLEL, "mlstm": ONLY_MLSTM,
           "moe": ONLY_MOE, "shared": SHARED}


def shape_weights(weights: Dict[str, torch.Tensor], seed: int, peaked: float = 1.0) -> None:
    """Random weights hide some faults.  Gains stored around zero are spread out, biases weigh as much as what they are added
    to, lambda lies away from `diff`, gates away from one half, forget gates differ from head to head between a memory of a
    few tokens and one of hundreds, and with `peaked` the query matrices are scaled so that single keys decide rows."""
    g = torch.Generator().manual_seed(seed)
    for name, t in weights.items():
        if not t.is_floating_point():
            continue
        if name.endswith((".norm1", ".norm2", "final.norm", "embed.norm")):
            t.copy_(torch.randn(t.shape, generator=g) * 0.3)
        elif name.endswith(".right.norm") or name.endswith(".mix.norm"):
            t.copy_(torch.randn(t.shape, generator=g) * 0.4 + 1.0)
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t.copy_(torch.randn(t.shape, generator=g) * 0.45 / t.numel() ** 0.25)
            if name.endswith("1"):
                t.abs_()
        elif name.endswith(".f.b"):
            t.copy_(torch.linspace(-0.5, 6.0, t.numel()) if t.numel() > 1 else torch.full_like(t, 4.0))
        elif name.endswith(".i.b"):
            t.copy_(torch.randn(t.shape, generator=g) * 1.5)
        elif name.endswith((".i", ".f", ".g")) and ".mix." in name:
            t.mul_(2.0)
        elif name.endswith((".q.b", ".k.b", ".v.b")):
            t.copy_(torch.randn(t.shape, generator=g) * 0.5)
        elif name.endswith(".o"):
            t.mul_(2.0)
        if name.endswith((".mix.q", ".mix.q.b", ".left.q", ".left.q.b")) and peaked != 1.0:
            t.mul_(peaked)


@functools.lru_cache(maxsize=None)
def folder_of(name: str, seed: int = 1, std: float = 0.08, peaked: float = 1.0) -> str:
    from safetensors.torch import load_file, save_file
    folder = os.path.join(helpers.tmp_root(), f"betepel_{name}_{seed}_{std}_{peaked}")
    ml.write_random_model(ModelConfig.from_dict(CONFIGS[name]), folder, seed, torch.bfloat16, std=std)
    path = os.path.join(folder, "model.safetensors")
    weights = {k: (v.float() if v.is_floating_point() else v) for k, v in load_file(path).items()}
    shape_weights(weights, seed, peaked)
    save_file({k: (v.to(torch.bfloat16) if v.is_floating_point() else v).contiguous() for k, v in weights.items()}, path)
    return folder


@functools.lru_cache(maxsize=None)
def oracle(folder: str):
    return pb.read_config(folder), pb.read_weights(folder, torch.float64)


_LOGITS: Dict[tuple, torch.Tensor] = {}


def oracle_logits(folder: str, tokens: Sequence[int]) -> torch.Tensor:
    """Logits of every position (kept: several tests ask for the same sequence)."""
    key = (folder, tuple(tokens))
    if key not in _LOGITS:
        cfg, w = oracle(folder)
        _LOGITS[key] = pb.forward(cfg, w, tokens).float()
    return _LOGITS[key]


# Bounds on a row's max|engine - plain| / max|plain|: the worst row, nine rows in ten, the mean.  The experts are chosen by the
# token's id, so no rounding can change a choice.  But the heads of the memories and of the differential attention are divided
# by their own root mean square: a token whose head happens to be nearly nothing before that (two maps that nearly cancel, a
# query nearly orthogonal to the memory) has the 16-bit rounding of its inputs magnified, in every cut and batch alike.
TOL = {"float32": (1e-4, 1e-4, 1e-4), "bfloat16": (3e-1, 6e-2, 3e-2)}


def check(got: torch.Tensor, want: torch.Tensor, dtype: str, what: str) -> None:
    assert got.shape == want.shape, (what, got.shape, want.shape)
    assert bool(torch.isfinite(got).all()), what
    errs = [helpers.rel_err(got[i], want[i]) for i in range(got.shape[0])]
    worst, mean, most = max(errs), sum(errs) / len(errs), sorted(errs)[int(0.9 * (len(errs) - 1))]
    assert worst <= TOL[dtype][0] and most <= TOL[dtype][1] and mean <= TOL[dtype][2], \
        f"{what}: worst {worst:.3e} (row {errs.index(worst)}), nine in ten {most:.3e}, mean {mean:.3e}"
