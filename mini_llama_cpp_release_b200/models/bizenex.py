"""Bizenex: a pre-norm decoder without any rotation, whose config.json lists its layers.

    x = E[token]
    per layer:  x <- x + mixer(N1(x));   x <- x + ff(N2(x))        (the second only with a feed-forward)
                N: layer norm with a gain and a bias
    logits = c · tanh(W_head N_f(x) / c)                           (c = logit_softcap)

Mixers: "attention" (grouped query heads; queries and keys divided by their root mean square per head, without gains;
queries scaled up with their position; a softmax with one more in its denominator: `parts/attention.py: SinkAttention` with
those options) and "latent_attention" (keys and values expanded from a cached normed latent, no rotated part; a learned sink
per head; a sigmoid gate on the heads' outputs; optionally the latents of an earlier layer: `parts/attention.py:
LatentAttention` with those options).
Feed-forward: a mixture of SwiGLU experts routed by sigmoid scores inside the best groups of experts (a group's score is the
sum of its two largest), weighted by the chosen scores over their sum (`parts/feed_forward.py: MixtureOfExperts`), or none.

config.json (every size and constant comes from it):
    architecture, vocab, width, logit_softcap, norm {eps},
    layers[i]: type, mixer {...}, mlp {kind: "moe", expert {ff}, router {experts, top, groups {count, keep}}} | null
      attention:         heads, kv_heads, dim, vdim, scale, q_temp {coef, every}
      latent_attention:  heads, dim, vdim, kv_rank, scale, kv_from
Tensors: embed, head, final.norm{,.b}, l<i>.norm1{,.b}, l<i>.norm2{,.b}, l<i>.mix.<...>, l<i>.mlp.<...>.  The model names no
largest position; sequences are bounded by the cache alone.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from ..config.model_config import ConfigError, ModelConfig, as_int
from ..config.registry import register_architecture
from ..config.specs import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .mepolix import NO_POSITION_LIMIT, _count, _need, _number

MIXERS = ("attention", "latent_attention")


@dataclass(frozen=True, kw_only=True)
class BizenexConfig(ModelConfig):
    hidden_size: int
    norm_eps: float
    logit_softcap: Optional[float]
    layers: Tuple[Dict[str, Any], ...]

    KEYS = ("vocab", "width", "norm", "layers", "logit_softcap")

    @classmethod
    def parse(cls, raw: Dict[str, Any]) -> "BizenexConfig":
        for key in ("vocab", "width", "layers", "norm"):
            if key not in raw:
                raise ConfigError(f"missing config key: {key}")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("config key layers must be a list with at least one layer")
        shared = dict(cls.shared_fields({**raw, "vocab_size": raw["vocab"],
                                         "max_position_embeddings": raw.get("max_position_embeddings", NO_POSITION_LIMIT)}))
        cfg = cls(**shared, hidden_size=as_int(raw, "width"), norm_eps=_number(raw["norm"], "eps", "norm"),
                  logit_softcap=_number(raw, "logit_softcap", "config") if raw.get("logit_softcap") is not None else None,
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
        if self.logit_softcap is not None and not self.logit_softcap > 0:
            raise ConfigError(f"logit_softcap must be positive, got {self.logit_softcap}")
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
            if kind != "latent_attention":
                raise ConfigError(f"{where}.mixer.kv_from belongs to latent_attention layers")
            if isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < i:
                raise ConfigError(f"{where}.mixer.kv_from must name an earlier layer, got {src!r}")
            owner = self.layers[src]
            if owner.get("type") != "latent_attention" or (owner.get("mixer") or {}).get("kv_from") is not None:
                raise ConfigError(f"{where}.mixer.kv_from names layer {src}, which is no latent_attention layer with a latent of its own")
            if owner["mixer"].get("kv_rank") != m.get("kv_rank"):
                raise ConfigError(f"{where}.mixer.kv_rank differs from layer {src}'s, whose latents it reads")

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.norm_eps}, "layers": [dict(l) for l in self.layers]}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.max_position_embeddings != NO_POSITION_LIMIT:
            d["max_position_embeddings"] = self.max_position_embeddings
        d["torch_dtype"] = self.torch_dtype
        for key in ("bos_token_id", "eos_token_id"):
            v = getattr(self, key)
            if v is not None:
                d[key] = list(v) if isinstance(v, tuple) and len(v) > 1 else (v[0] if isinstance(v, tuple) else v)
        d.update(self.extra)
        return d


_UNROTATED = PartSpec("position", "rope_partial", dict(dims=0, base=1.0, scaling=None))


def _attention(c: BizenexConfig, m: Dict[str, Any], where: str) -> PartSpec:
    temp = m.get("q_temp")
    return PartSpec("mixer", "sink_attention", dict(
        hidden_size=c.hidden_size, num_heads=_count(m, "heads", where), num_kv_heads=_count(m, "kv_heads", where),
        head_dim=_count(m, "dim", where), v_head_dim=_count(m, "vdim", where), scale=_number(m, "scale", where),
        norm_eps=c.norm_eps, position=_UNROTATED, qk_norm=True, qk_gain=False, sink=False, const_sink=0.0,
        q_temp=(_number(temp, "coef", where + ".q_temp"), _count(temp, "every", where + ".q_temp")) if temp else None))


def _latent(c: BizenexConfig, m: Dict[str, Any], where: str) -> PartSpec:
    return PartSpec("mixer", "latent_attention", dict(
        hidden_size=c.hidden_size, num_heads=_count(m, "heads", where), head_dim=_count(m, "dim", where), rot_dim=0,
        v_head_dim=_count(m, "vdim", where), kv_rank=_count(m, "kv_rank", where), scale=_number(m, "scale", where),
        norm_eps=c.norm_eps, position=_UNROTATED, sink=True, out_gate=True, own_kv=m.get("kv_from") is None))


def _feed_forward(c: BizenexConfig, mlp: Dict[str, Any], where: str) -> PartSpec:
    router, expert = _need(mlp, "router", where), _need(mlp, "expert", where)
    groups = router.get("groups") or {}
    return PartSpec("feed_forward", "mixture", dict(
        hidden_size=c.hidden_size, intermediate_size=_count(expert, "ff", where + ".expert"),
        num_experts=_count(router, "experts", where + ".router"), top=_count(router, "top", where + ".router"),
        gated=True, activation="silu", routing="scores", score="sigmoid", router_bias=False,
        group_count=_count(groups, "count", where + ".router.groups") if groups else 1,
        group_keep=_count(groups, "keep", where + ".router.groups") if groups else 1, group_score="top2"))


@register_architecture("Bizenex", config_class=BizenexConfig)
def bizenex(config: BizenexConfig) -> ModelSpec:
    c = config
    norm = lambda tensor: PartSpec("norm", "layernorm", dict(size=c.hidden_size, eps=c.norm_eps, tensor=tensor, bias=".b"))
    builders = {"attention": _attention, "latent_attention": _latent}
    layers: List[LayerSpec] = []
    for i, layer in enumerate(c.layers):
        params: Dict[str, Any] = dict(
            mixer=builders[layer["type"]](c, layer["mixer"], f"layers[{i}].mixer"), mixer_norm=norm("norm1"),
            names={"mixer": "mix.", "mixer_norm": "", "feed_forward": "mlp.", "feed_forward_norm": ""})
        if layer.get("mlp") is not None:
            params["feed_forward"] = _feed_forward(c, layer["mlp"], f"layers[{i}].mlp")
            params["feed_forward_norm"] = norm("norm2")
        layers.append(LayerSpec(f"l{i}.", PartSpec("block", "prenorm", params)))
    return ModelSpec(
        config=c,
        embedding=PartSpec("embedding", "token_embedding", dict(vocab_size=c.vocab_size, hidden_size=c.hidden_size, tensor="embed")),
        layers=tuple(layers),
        # one run per layer, in order: a layer that names kv_from reads that layer's cache entry instead of keeping one
        schedule=tuple(ScheduleEntry(layer=i, reads_cache_of=layer["mixer"].get("kv_from")) for i, layer in enumerate(c.layers)),
        final_norm=norm("norm"),
        head=PartSpec("head", "linear_head", dict(vocab_size=c.vocab_size, hidden_size=c.hidden_size, tensor="head",
                                                  softcap=c.logit_softcap)),
        names={"embedding": "", "final_norm": "final.", "head": ""},
    )
