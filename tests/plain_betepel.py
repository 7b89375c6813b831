"""Plain, slow implementation of the Betepel decoder, used only as the tests' oracle.

Whole sequences on the CPU, no cache: attention sees the prefix through an explicit mask, recurrences walk token by token,
every token visits its experts one by one.  One function per mechanism; nothing is shared with the product package
(config.json is parsed here, weights are read with the `safetensors` package).  The default element type is float64, which
bounds how much of a difference between the engine and this file is rounding.

The model, in this file's notation (R: division by the root mean square, times 1 + w):

    x = R_e(E[token])
    per layer:   x <- x + ( mixer(R_1(x)) + ff(R_2(x)) )          (both read the same x; ff may be absent)
    logits = E R_f(x) * c

Three mixers: "attention" (differential: two softmax maps per head over the same values, subtracted; a window that keeps the
sequence's first tokens; one sigmoid gate per head; optionally another layer's keys and values), "parallel" (windowed
attention beside linear attention with a constant decay per head, added with two factors) and "mlstm" (a matrix memory with
exponential input and sigmoid forget gates, stabilised by a running maximum).  The feed-forward: experts chosen by the
token's id from a table, all of one weight, and one more expert that every token passes.
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

def unit_rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(dim=-1, keepdim=True) + eps)


def rms_norm(v: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """A gain stored around zero."""
    return unit_rms(v, eps) * (1.0 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# --------------------------------------------------------------------------- rotation

def frequencies(rot: dict, dtype=torch.float64) -> torch.Tensor:
    """base^(-2i/dims), slowed down where the wavelength is long: kept below original/high, divided by `factor` above
    original/low, and in between a mixture that is linear in original/wavelength."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc:
        factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
        out = []
        for fi in f:
            length = 2.0 * math.pi / fi
            if length < original / high:
                out.append(fi)
            elif length > original / low:
                out.append(fi / factor)
            else:
                s = (original / length - low) / (high - low)
                out.append((1.0 - s) * fi / factor + s * fi)
        f = out
    return torch.tensor(f, dtype=dtype)


def rotate(x: torch.Tensor, rot: Optional[dict], positions: torch.Tensor) -> torch.Tensor:
    """x [T, heads, d]: the first dims entries of each head in pairs (i, i + dims/2)."""
    if not rot or not int(rot["dims"]):
        return x
    dims = int(rot["dims"])
    a = positions.to(x.dtype)[:, None] * frequencies(rot, x.dtype)[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v, rest = x[..., :dims // 2], x[..., dims // 2:dims], x[..., dims:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], dim=-1)


# --------------------------------------------------------------------------- attention

def visible(T: int, mask: Optional[dict]) -> torch.Tensor:
    """[T, T] of bool: row i sees column j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    if mask and mask.get("size") is not None:
        ok = ok & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first") or 0)))
    return ok


def softmax_map(q, k, v, scale: float, ok: torch.Tensor, probs_out: Optional[list] = None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads key/value head h // (H/G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = q.new_zeros(T, H, v.shape[2])
    for h in range(H):
        g = h // (H // G)
        p = torch.softmax(((q[:, h] @ k[:, g].T) * scale).masked_fill(~ok, -math.inf), dim=-1)
        if probs_out is not None:
            probs_out.append(p)
        out[:, h] = p @ v[:, g]
    return out


def diff_lambda(w, p, diff: float) -> torch.Tensor:
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def diff_combine(a1, a2, lam, diff: float, eps: float) -> torch.Tensor:
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def diff_attention(h, w, p, m, eps, positions, kept: dict, index: int, probs_out=None):
    """Mixer "attention".  `kept[j]` holds layer j's keys (rotated) and values for a later layer that names it in kv_from."""
    T = h.shape[0]
    H, G, d, dv, diff = m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["diff"])
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, 2, d)
    q1, q2 = rotate(q[:, :, 0], m.get("rot"), positions), rotate(q[:, :, 1], m.get("rot"), positions)
    if m.get("kv_from") is not None:
        k1, k2, v = kept[int(m["kv_from"])]
    else:
        k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, 2, d)
        k1, k2 = rotate(k[:, :, 0], m.get("rot"), positions), rotate(k[:, :, 1], m.get("rot"), positions)
        v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
        kept[index] = (k1, k2, v)
    ok = visible(T, m.get("mask"))
    a1 = softmax_map(q1, k1, v, m["scale"], ok, probs_out)
    a2 = softmax_map(q2, k2, v, m["scale"], ok, probs_out)
    o = diff_combine(a1, a2, diff_lambda(w, p, diff), diff, eps)
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def window_attention(h, w, p, m, positions, probs_out=None):
    """The left half of mixer "parallel"."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate((h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, d), m.get("rot"), positions)
    k = rotate((h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, d), m.get("rot"), positions)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
    o = softmax_map(q, k, v, m["scale"], visible(T, m.get("mask")), probs_out)
    return o.reshape(T, H * dv) @ w[p + "o"].T


# --------------------------------------------------------------------------- linear attention with a constant decay

def decay_walk(q, k, v, decay) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, dv], decay [H]: S <- decay S + k v^T, o = S^T q."""
    T, H, d = q.shape
    S = q.new_zeros(H, d, v.shape[2])
    lam = torch.tensor([float(x) for x in decay], dtype=q.dtype)[:, None, None]
    out = []
    for t in range(T):
        S = lam * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def lightning(h, w, p, m, eps):
    """The right half of mixer "parallel"."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k = silu(h @ w[p + "q"].T).reshape(T, H, d), silu(h @ w[p + "k"].T).reshape(T, H, d)
    v = silu(h @ w[p + "v"].T).reshape(T, H, dv)
    o = decay_walk(q, k, v, m["decay"]).reshape(T, H * dv)
    return (unit_rms(o, eps) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, w, p, m, eps, positions):
    left = window_attention(h, w, p + "left.", m["left"], positions)
    right = lightning(h, w, p + "right.", m["right"], eps)
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


# --------------------------------------------------------------------------- matrix memory with exponential gates

def log_gates(h, w, p, cap: float):
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    return i, f


def memory_walk(q, k, v, i, f) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, dv], log gates i, f [T, H]; the running maximum starts at zero."""
    T, H, d = q.shape
    S, n, m = q.new_zeros(H, d, v.shape[2]), q.new_zeros(H, d), q.new_zeros(H)
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        size = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append((S * q[t][:, :, None]).sum(1) / size[:, None])
    return torch.stack(out)


def mlstm(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    o = unit_rms(memory_walk(q, k, v, *log_gates(h, w, p, float(m["gate_cap"]))), eps).reshape(T, H * dv)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# --------------------------------------------------------------------------- experts by the token's id

def expert(v, w, p):
    return (silu(v @ w[p + "gate"].T) * (v @ w[p + "up"].T)) @ w[p + "down"].T


def table_moe(h, w, p, mlp, ids):
    top = int(mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in w[p + "table"][ids[t]].tolist():
            out[t] = out[t] + expert(h[t], w, f"{p}e{e}.") / top
    return out + expert(h, w, p + "shared.") if mlp.get("shared") else out


# --------------------------------------------------------------------------- the model

def mixer(h, w, p, spec, eps, positions, kept, index):
    if spec["type"] == "attention":
        return diff_attention(h, w, p, spec["mixer"], eps, positions, kept, index)
    if spec["type"] == "parallel":
        return parallel(h, w, p, spec["mixer"], eps, positions)
    if spec["type"] == "mlstm":
        return mlstm(h, w, p, spec["mixer"], eps)
    raise ValueError(spec["type"])


def layer(x, w, i, spec, cfg, positions, kept, ids):
    n, eps = f"l{i}.", float(cfg["norm"]["eps"])
    y = mixer(rms_norm(x, w[n + "norm1"], eps), w, n + "mix.", spec, eps, positions, kept, i)
    if spec.get("mlp") is not None:
        y = y + table_moe(rms_norm(x, w[n + "norm2"], eps), w, n + "mlp.", spec["mlp"], ids)
    return x + y


def embed(cfg: dict, w: Dict[str, torch.Tensor], ids: torch.Tensor) -> torch.Tensor:
    return rms_norm(w["embed"][ids], w["embed.norm"], float(cfg["norm"]["eps"]))


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, stream_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from its first token; `stream_out` collects the stream behind every layer."""
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    positions = torch.arange(len(ids))
    x = embed(cfg, w, ids)
    kept: dict = {}
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, i, spec, cfg, positions, kept, ids)
        if stream_out is not None:
            stream_out.append(x.clone())
    return rms_norm(x, w["final.norm"], float(cfg["norm"]["eps"])) @ w["embed"].T * float(cfg["logit_scale"])
