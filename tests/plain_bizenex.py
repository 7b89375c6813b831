"""Plain, slow implementation of the Bizenex decoder, used only as the tests' oracle.

Whole sequences on the CPU, no cache: attention sees the prefix through an explicit mask, keys and values of the latent
attention are expanded for every position, every token visits its experts one by one.  One function per mechanism; nothing is
shared with the product package (config.json is parsed here, weights are read with the `safetensors` package).  The default
element type is float64, which bounds how much of a difference between the engine and this file is rounding.

The model, in this file's notation (N: layer norm with gain and bias):

    x = E[token]
    per layer:   x <- x + mixer(N1(x)),   then   x <- x + ff(N2(x))   (ff may be absent)
    logits = c tanh(W_head N_f(x) / c)

Two mixers: "attention" (grouped heads, unit-RMS queries and keys without gains, queries scaled up with their position, a
softmax with one more in its denominator) and "latent_attention" (keys and values expanded from a normed latent, which may be
an earlier layer's; a learned sink per head; a sigmoid gate on the heads' outputs).  One feed-forward: a mixture of SwiGLU
experts chosen inside the best groups by sigmoid scores, weighted by the chosen scores divided by their sum.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, Optional

import torch


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def read_weights(folder: str, dtype=torch.float64) -> Dict[str, torch.Tensor]:
    from safetensors.torch import load_file
    return {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}


# --------------------------------------------------------------------------- norms and activations

def layer_norm(v: torch.Tensor, w: Dict[str, torch.Tensor], name: str, eps: float) -> torch.Tensor:
    centred = v - v.mean(dim=-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(dim=-1, keepdim=True) + eps) * w[name] + w[name + ".b"]


def unit_rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(dim=-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# --------------------------------------------------------------------------- attention

def query_temperature(positions: torch.Tensor, temp: Optional[dict], dtype) -> torch.Tensor:
    """[T]: 1 + coef ln(1 + floor((p + 1) / every)); ones without a temperature."""
    if not temp:
        return torch.ones(len(positions), dtype=dtype)
    steps = torch.div(positions + 1, int(temp["every"]), rounding_mode="floor").to(dtype)
    return 1.0 + float(temp["coef"]) * torch.log(steps + 1.0)


def sink_softmax(scores: torch.Tensor, sink) -> torch.Tensor:
    """Row-wise exp(s_j) / (exp(sink) + sum_j exp(s_j)), by explicit exponentials around the larger of the two."""
    sink = torch.as_tensor(sink, dtype=scores.dtype)
    top = torch.maximum(scores.max(dim=-1, keepdim=True).values, sink)
    e = torch.exp(scores - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def attend(q, k, v, scale: float, sinks, probs_out: Optional[list] = None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv], causal; query head h reads key/value head h // (H/G); sinks [H]."""
    T, H, _ = q.shape
    G = k.shape[1]
    past = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = q.new_zeros(T, H, v.shape[2])
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~past, -math.inf)
        p = sink_softmax(s, sinks[h])
        if probs_out is not None:
            probs_out.append(p)
        out[:, h] = p @ v[:, g]
    return out


def attention(h, w, p, m, eps, positions, probs_out=None):
    """Mixer "attention"."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w[p + "q"].T).reshape(T, H, d), eps)
    k = unit_rms((h @ w[p + "k"].T).reshape(T, G, d), eps)
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    q = q * query_temperature(positions, m.get("q_temp"), h.dtype)[:, None, None]
    o = attend(q, k, v, m["scale"], torch.zeros(H, dtype=h.dtype), probs_out)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def latent_of(h, w, p, eps):
    """The cached latent: W_dkv h over its root mean square, times a gain."""
    return unit_rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]


def latent_attention(h, w, p, m, eps, kept: dict, index: int, probs_out=None):
    """Mixer "latent_attention".  `kept[j]` holds layer j's latents for a later layer that names it in kv_from."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    if m.get("kv_from") is not None:
        c = kept[int(m["kv_from"])]
    else:
        c = kept[index] = latent_of(h, w, p, eps)
    q = (h @ w[p + "q"].T).reshape(T, H, d)
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    o = attend(q, k, v, m["scale"], w[p + "sink"], probs_out).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# --------------------------------------------------------------------------- mixture of experts

def route_one(s: torch.Tensor, router: dict):
    """(ids, weights) of one token from its sigmoid scores s [E]: the largest scores inside the best groups."""
    scores = [float(v) for v in s]
    allowed = list(range(len(scores)))
    groups = router.get("groups")
    if groups:
        size = len(scores) // int(groups["count"])
        rank = []
        for g in range(int(groups["count"])):
            best = sorted(scores[g * size:(g + 1) * size], reverse=True)[:2]
            rank.append((-sum(best), g))
        kept = {g for _, g in sorted(rank)[:int(groups["keep"])]}
        allowed = [e for e in allowed if e // size in kept]
    ids = sorted(allowed, key=lambda e: (-scores[e], e))[:int(router["top"])]
    total = sum(scores[e] for e in ids) + 1e-20
    return ids, [scores[e] / total for e in ids]


def expert(v, w, p):
    return (silu(v @ w[p + "gate"].T) * (v @ w[p + "up"].T)) @ w[p + "down"].T


def moe_ff(h, w, p, mlp):
    s = torch.sigmoid(h @ w[p + "router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in zip(*route_one(s[t], mlp["router"])):
            out[t] = out[t] + weight * expert(h[t], w, f"{p}e{e}.")
    return out


# --------------------------------------------------------------------------- the model

def layer(x, w, i, spec, cfg, positions, kept):
    n, eps = f"l{i}.", float(cfg["norm"]["eps"])
    h = layer_norm(x, w, n + "norm1", eps)
    if spec["type"] == "attention":
        x = x + attention(h, w, n + "mix.", spec["mixer"], eps, positions)
    elif spec["type"] == "latent_attention":
        x = x + latent_attention(h, w, n + "mix.", spec["mixer"], eps, kept, i)
    else:
        raise ValueError(spec["type"])
    if spec.get("mlp") is not None:
        x = x + moe_ff(layer_norm(x, w, n + "norm2", eps), w, n + "mlp.", spec["mlp"])
    return x


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, stream_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from its first token; `stream_out` collects the stream behind every layer."""
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    positions = torch.arange(len(ids))
    x = w["embed"][ids]
    kept: dict = {}
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, i, spec, cfg, positions, kept)
        if stream_out is not None:
            stream_out.append(x.clone())
    logits = layer_norm(x, w, "final.norm", float(cfg["norm"]["eps"])) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return logits if cap is None else float(cap) * torch.tanh(logits / float(cap))
