"""Betepel: a decoder of parallel blocks with two norms each, whose config.json lists its layers.

    x = N_e(E[token])                                              N: RMS norm with gain 1 + w
    per layer:  x <- x + ( mixer(N1(x)) + ff(N2(x)) )              (both of the same x; ff may be absent)
    logits = c · E N_f(x)                                          (the embedding's table; c = logit_scale)

Mixers: "attention" (differential attention with a window that keeps the sequence's first tokens, a sigmoid gate per head,
rotation stretched by wavelength; optionally the keys and values of an earlier layer: `parts/attention.py:
DifferentialAttention`), "parallel" (windowed attention, `SinkAttention` without norm and sink, beside linear attention with a
constant decay per head, `parts/recurrent.py: DecayAttention`, added with two factors: `ParallelMixer`) and "mlstm" (a matrix
memory with exponential gates: `parts/recurrent.py: MatrixMemory`).
Feed-forward: SwiGLU experts chosen by the token's id from a stored table, each of weight 1/top, and a shared expert for every
token (`parts/feed_forward.py: MixtureOfExperts`), or none.

config.json (every size and constant comes from it):
    architecture, vocab, width, logit_scale, norm {eps},
    layers[i]: type, mixer {...}, mlp {kind: "moe", expert {ff}, router {experts, top}, shared {ff}} | null
      attention:  heads, kv_heads, dim, vdim, scale, diff, rot {base, dims, scaling {factor, low, high, original}},
                  mask {size, keep_first}, kv_from
      parallel:   left {heads, kv_heads, dim, vdim, scale, rot {base, dims}, mask {size}},
                  right {heads, dim, vdim, decay [heads]}, left_scale, right_scale
      mlstm:      heads, dim, vdim, gate_cap
Tensors: embed, embed.norm, final.norm, l<i>.norm1, l<i>.norm2, l<i>.mix.<...>, l<i>.mlp.<...>.  The model names no largest
position; sequences are bounded by the cache alone.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from ..config.model_config import ConfigError, ModelConfig, as_int
from ..config.registry import register_architecture
from ..config.specs import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .mepolix import NO_POSITION_LIMIT, _count, _need, _number

MIXERS = ("attention", "parallel", "mlstm")


@dataclass(frozen=True, kw_only=True)
class BetepelConfig(ModelConfig):
    hidden_size: int
    norm_eps: float
    logit_scale: float
    layers: Tuple[Dict[str, Any], ...]

    KEYS = ("vocab", "width", "norm", "layers", "logit_scale")

    @classmethod
    def parse(cls, raw: Dict[str, Any]) -> "BetepelConfig":
        for key in ("vocab", "width", "layers", "norm"):
            if key not in raw:
                raise ConfigError(f"missing config key: {key}")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("config key layers must be a list with at least one layer")
        shared = dict(cls.shared_fields({**raw, "vocab_size": raw["vocab"],
                                         "max_position_embeddings": raw.get("max_position_embeddings", NO_POSITION_LIMIT)}))
        cfg = cls(**shared, hidden_size=as_int(raw, "width"), norm_eps=_number(raw["norm"], "eps", "norm"),
                  logit_scale=_number(raw, "logit_scale", "config") if raw.get("logit_scale") is not None else 1.0,
                  layers=tuple(raw["layers"]),
                  extra={k: v for k, v in raw.items() if k not in cls.SHARED_KEYS and k not in cls.KEYS})
        cfg.validate()
        return cfg

    def validate(self) -> None:
        super().validate()
        if self.hidden_size <= 0:
            raise ConfigError(f"width must be positive, got {self.hidden_size}")
        if not self.norm_eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.norm_eps}")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in MIXERS:
                raise ConfigError(f"{where}.type must be one of {', '.join(MIXERS)}; got {kind!r}")
            m = _need(layer, "mixer", where)
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind", "moe") != "moe":
                raise ConfigError(f"{where}.mlp.kind must be \"moe\", got {mlp.get('kind')!r}")
            src = m.get("kv_from")
            if src is None:
                continue
            if kind != "attention":
                raise ConfigError(f"{where}.mixer.kv_from belongs to attention layers")
            if isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < i:
                raise ConfigError(f"{where}.mixer.kv_from must name an earlier layer, got {src!r}")
            owner = self.layers[src]
            if owner.get("type") != "attention" or (owner.get("mixer") or {}).get("kv_from") is not None:
                raise ConfigError(f"{where}.mixer.kv_from names layer {src}, which is no attention layer with keys of its own")
            for key in ("kv_heads", "dim", "vdim"):
                if owner["mixer"].get(key) != m.get(key):
                    raise ConfigError(f"{where}.mixer.{key} differs from layer {src}'s, whose keys and values it reads")

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "logit_scale": self.logit_scale, "norm": {"eps": self.norm_eps}, "layers": [dict(l) for l in self.layers]}
        if self.max_position_embeddings != NO_POSITION_LIMIT:
            d["max_position_embeddings"] = self.max_position_embeddings
        d["torch_dtype"] = self.torch_dtype
        for key in ("bos_token_id", "eos_token_id"):
            v = getattr(self, key)
            if v is not None:
                d[key] = list(v) if isinstance(v, tuple) and len(v) > 1 else (v[0] if isinstance(v, tuple) else v)
        d.update(self.extra)
        return d


def _rotation(m: Dict[str, Any], where: str) -> PartSpec:
    rot = m.get("rot") or {}
    dims = int(rot.get("dims") or 0)
    if not dims:
        return PartSpec("position", "rope_partial", dict(dims=0, base=1.0, scaling=None))
    if dims % 2 or dims > int(m["dim"]):
        raise ConfigError(f"{where}.rot.dims must be even and at most dim, got {dims}")
    return PartSpec("position", "rope_partial", dict(dims=dims, base=_number(rot, "base", where + ".rot"),
                                                     scaling=dict(rot["scaling"]) if rot.get("scaling") else None))


def _mask(m: Dict[str, Any], where: str) -> Tuple[Optional[int], int]:
    """(window, first tokens that stay visible); no size: every earlier token."""
    mask = m.get("mask") or {}
    if mask.get("size") is None:
        return None, 0
    return _count(mask, "size", where + ".mask"), int(mask.get("keep_first") or 0)


def _heads(c: BetepelConfig, m: Dict[str, Any], where: str) -> Dict[str, Any]:
    return dict(hidden_size=c.hidden_size, num_heads=_count(m, "heads", where), num_kv_heads=_count(m, "kv_heads", where),
                head_dim=_count(m, "dim", where), v_head_dim=_count(m, "vdim", where), scale=_number(m, "scale", where),
                norm_eps=c.norm_eps, position=_rotation(m, where))


def _attention(c: BetepelConfig, m: Dict[str, Any], where: str, keep_all_keys: bool = False) -> PartSpec:
    window, keep = _mask(m, where)
    return PartSpec("mixer", "differential_attention", dict(
        _heads(c, m, where), diff=_number(m, "diff", where), window=window, keep_first=keep, bias=True, head_gate=True,
        own_kv=m.get("kv_from") is None, keep_all_keys=keep_all_keys))


def _parallel(c: BetepelConfig, m: Dict[str, Any], where: str) -> PartSpec:
    left, right = _need(m, "left", where), _need(m, "right", where)
    window, keep = _mask(left, where + ".left")
    attn = PartSpec("mixer", "sink_attention", dict(
        _heads(c, left, where + ".left"), qk_norm=False, sink=False, bias=True, window=window, keep_first=keep,
        value_scale=_number(m, "left_scale", where)))
    lin = PartSpec("mixer", "decay_attention", dict(
        hidden_size=c.hidden_size, num_heads=_count(right, "heads", where + ".right"), head_dim=_count(right, "dim", where + ".right"),
        v_head_dim=_count(right, "vdim", where + ".right"), decay=tuple(float(d) for d in _need(right, "decay", where + ".right")),
        norm_eps=c.norm_eps, out_scale=_number(m, "right_scale", where)))
    return PartSpec("mixer", "parallel", dict(left=attn, right=lin))


def _mlstm(c: BetepelConfig, m: Dict[str, Any], where: str) -> PartSpec:
    return PartSpec("mixer", "matrix_memory", dict(
        hidden_size=c.hidden_size, num_heads=_count(m, "heads", where), head_dim=_count(m, "dim", where),
        v_head_dim=_count(m, "vdim", where), gate_cap=_number(m, "gate_cap", where), norm_eps=c.norm_eps))


def _feed_forward(c: BetepelConfig, mlp: Dict[str, Any], where: str) -> PartSpec:
    router, expert = _need(mlp, "router", where), _need(mlp, "expert", where)
    shared = None
    if mlp.get("shared"):
        shared = PartSpec("feed_forward", "swiglu", dict(hidden_size=c.hidden_size, names={"gate": "gate", "up": "up", "down": "down"},
                                                         intermediate_size=_count(mlp["shared"], "ff", where + ".shared")))
    return PartSpec("feed_forward", "mixture", dict(
        hidden_size=c.hidden_size, intermediate_size=_count(expert, "ff", where + ".expert"),
        num_experts=_count(router, "experts", where + ".router"), top=_count(router, "top", where + ".router"),
        gated=True, activation="silu", routing="table", router_bias=False, vocab_size=c.vocab_size, shared=shared))


@register_architecture("Betepel", config_class=BetepelConfig)
def betepel(config: BetepelConfig) -> ModelSpec:
    c = config

    def norm(tensor: str, scale: float = 1.0) -> PartSpec:
        return PartSpec("norm", "rmsnorm", dict(size=c.hidden_size, eps=c.norm_eps, tensor=tensor, offset=1.0, scale=scale))
    # a layer whose keys another layer reads under another mask keeps all of them
    other_mask = {int(l["mixer"]["kv_from"]) for l in c.layers if l["mixer"].get("kv_from") is not None
                  and _mask(l["mixer"], "") != _mask(c.layers[int(l["mixer"]["kv_from"])]["mixer"], "")}
    layers: List[LayerSpec] = []
    for i, layer in enumerate(c.layers):
        where, m = f"layers[{i}].mixer", layer["mixer"]
        mixer = (_attention(c, m, where, keep_all_keys=i in other_mask) if layer["type"] == "attention"
                 else _parallel(c, m, where) if layer["type"] == "parallel" else _mlstm(c, m, where))
        params: Dict[str, Any] = dict(mixer=mixer, mixer_norm=norm("norm1"),
                                      names={"mixer": "mix.", "mixer_norm": "", "feed_forward": "mlp.", "feed_forward_norm": ""})
        if layer.get("mlp") is not None:
            params["feed_forward"] = _feed_forward(c, layer["mlp"], f"layers[{i}].mlp")
            params["feed_forward_norm"] = norm("norm2")
        layers.append(LayerSpec(f"l{i}.", PartSpec("block", "parallel_prenorm", params)))
    return ModelSpec(
        config=c,
        embedding=PartSpec("embedding", "token_embedding", dict(vocab_size=c.vocab_size, hidden_size=c.hidden_size, tensor="embed",
                                                                norm=norm("embed.norm"))),
        layers=tuple(layers),
        # one run per layer, in order: a layer that names kv_from reads that layer's cache entry instead of keeping one
        schedule=tuple(ScheduleEntry(layer=i, reads_cache_of=layer["mixer"].get("kv_from")) for i, layer in enumerate(c.layers)),
        # the head is linear and has no bias: the factor on the logits is one on the final norm's gain
        final_norm=norm("norm", scale=c.logit_scale),
        head=PartSpec("head", "linear_head", dict(vocab_size=c.vocab_size, hidden_size=c.hidden_size, tied_to="embed", tensor="head")),
        names={"embedding": "", "final_norm": "final.", "head": ""},
    )
