"""Bizenex without a GPU: its configuration, what its layers ask of the cache, the names of its tensors, and the plain
implementation's mechanisms against each other."""
import copy
import math

import pytest
import torch

import bizenex_helpers as bh
import plain_bizenex as pb
from mini_llama_cpp_release_b200.cache.paged import plan_groups
from mini_llama_cpp_release_b200.config import ModelConfig
from mini_llama_cpp_release_b200.config.model_config import ConfigError
from mini_llama_cpp_release_b200.config.registry import build_model_spec
from mini_llama_cpp_release_b200.engine.model import build_parts
from mini_llama_cpp_release_b200.parts.base import CacheNeed

rnd_gen = torch.Generator().manual_seed(0)


def rnd(*shape):
    return torch.randn(*shape, generator=rnd_gen, dtype=torch.float64)


def changed(config, path, value):
    bad = copy.deepcopy(config)
    d = bad
    for key in path[:-1]:
        d = d[key]
    d[path[-1]] = value
    return bad


def test_config_round_trip_and_checks():
    cfg = ModelConfig.from_dict(bh.MIXED)
    assert cfg.architecture == "Bizenex" and cfg.vocab_size == 300 and cfg.hidden_size == 112
    assert (cfg.logit_softcap, cfg.norm_eps) == (12.0, 1e-5)
    assert ModelConfig.from_dict(cfg.to_dict()) == cfg
    odd = ModelConfig.from_dict(bh.ODD)
    assert odd.logit_softcap is None and ModelConfig.from_dict(odd.to_dict()) == odd
    for path, value in [(("layers", 0, "type"), "gla"), (("layers", 0, "mlp", "kind"), "dense"), (("norm", "eps"), 0.0),
                        (("logit_softcap",), -1.0), (("layers", 2, "mixer", "kv_from"), 2), (("layers", 2, "mixer", "kv_from"), 0),
                        (("layers", 4, "mixer", "kv_from"), 2), (("layers", 2, "mixer", "kv_rank"), 48),
                        (("layers", 3, "mixer", "kv_from"), 1), (("layers", 2, "mixer", "kv_from"), True)]:
        with pytest.raises(ConfigError):
            ModelConfig.from_dict(changed(bh.MIXED, path, value))
    # what the parts refuse when the model is built
    for path, value in [(("layers", 0, "mixer", "kv_heads"), 4), (("layers", 0, "mixer", "q_temp", "every"), 0),
                        (("layers", 0, "mlp", "router", "top"), 7), (("layers", 0, "mlp", "router", "groups", "count"), 4),
                        (("layers", 1, "mlp", "router", "groups", "keep"), 1), (("layers", 1, "mixer", "scale"), 0.0),
                        (("layers", 1, "mixer", "kv_rank"), 0)]:
        with pytest.raises((ConfigError, ValueError)):
            build_parts(build_model_spec(ModelConfig.from_dict(changed(bh.MIXED, path, value))))


def test_what_the_layers_ask_of_the_cache_and_which_tensors_they_read():
    spec = build_model_spec(ModelConfig.from_dict(bh.MIXED))
    assert [(e.layer, e.reads_cache_of) for e in spec.schedule] == [(0, None), (1, None), (2, 1), (3, None), (4, 1)]
    assert all(l.block.kind == "prenorm" for l in spec.layers)
    parts = build_parts(spec)
    mixers = [parts.blocks[e.layer].mixer for e in spec.schedule]
    needs = [m.cache_need() for m in mixers]
    row = CacheNeed("all", 1, 48, None, 0, True)                        # ceil16(40): one row per token, values read out of it
    assert needs == [CacheNeed("all", 3, 48), row, row, CacheNeed("all", 1, 48), row]      # ceil16(max(24, 40)), ceil16(max(48, 16))
    groups, where = plan_groups(needs, [e.reads_cache_of for e in spec.schedule])
    assert len(groups) == 3 and where[2] == where[4] == where[1]
    assert sum(len(g.entries) for g in groups) == 3                     # the readers own no pages
    assert all(m.state_spec() is None for m in mixers)
    assert [(m.q_temp, m.const_sink, m.qk_gain) for m in (mixers[0], mixers[3])] == [((0.4, 20), 0.0, False), ((0.8, 1), 0.0, False)]
    names = {t.name: tuple(t.shape) for p in parts.all_parts() for t in p.all_tensors()}
    assert names["embed"] == (300, 112) and names["head"] == (300, 112)
    assert names["final.norm"] == (112,) and names["final.norm.b"] == (112,)
    assert names["l0.norm1.b"] == (112,) and names["l0.norm2"] == (112,) and names["l4.norm2.b"] == (112,)
    assert "l2.norm1" in names and "l2.norm2" not in names and not any(k.startswith("l2.mlp") for k in names)
    assert names["l0.mix.q"] == (144, 112) and names["l0.mix.k"] == (72, 112) and names["l0.mix.v"] == (120, 112) and names["l0.mix.o"] == (112, 240)
    assert not any(k.startswith("l0.mix.") and k.endswith(("norm", "sink", ".b", ".g")) for k in names)
    assert names["l1.mix.q"] == (80, 112) and names["l1.mix.dkv"] == (40, 112) and names["l1.mix.dkv.norm"] == (40,)
    assert names["l1.mix.uk"] == (80, 40) and names["l1.mix.uv"] == (120, 40) and names["l1.mix.sink"] == (5,)
    assert names["l1.mix.g"] == (120, 112) and names["l1.mix.o"] == (112, 120)
    assert names["l2.mix.uk"] == (56, 40) and names["l2.mix.uv"] == (252, 40) and names["l2.mix.sink"] == (7,)
    assert not any(k.startswith(("l2.mix.dkv", "l4.mix.dkv")) for k in names)                # the readers have no latents of their own
    assert names["l0.mlp.router"] == (6, 112) and names["l0.mlp.e5.gate"] == (48, 112) and names["l0.mlp.e5.down"] == (112, 48)
    assert "l0.mlp.e6.up" not in names and "l0.mlp.router.b" not in names


def test_plain_mechanisms_against_each_other():
    # layer norm: no mean, unit variance before the gain; a shift of all entries changes nothing
    v, w = rnd(5, 12), {"n": rnd(12), "n.b": rnd(12)}
    y = (pb.layer_norm(v, w, "n", 1e-12) - w["n.b"]) / w["n"]
    assert torch.allclose(y.mean(-1), torch.zeros(5, dtype=y.dtype), atol=1e-9) and torch.allclose((y * y).mean(-1), torch.ones(5, dtype=y.dtype), atol=1e-9)
    assert torch.allclose(pb.layer_norm(v + 3.0, w, "n", 1e-6), pb.layer_norm(v, w, "n", 1e-6))
    assert torch.allclose(pb.layer_norm(v, w, "n", 1e-6), torch.nn.functional.layer_norm(v, (12,), w["n"], w["n.b"], 1e-6))
    # the temperature steps where (p + 1) reaches a multiple of `every`
    t = pb.query_temperature(torch.arange(12), {"coef": 0.5, "every": 5}, torch.float64)
    assert torch.equal(t[:4], torch.ones(4, dtype=t.dtype)) and math.isclose(float(t[4]), 1 + 0.5 * math.log(2)) and t[4] == t[8]
    assert math.isclose(float(t[9]), 1 + 0.5 * math.log(3)) and t[9] == t[11]
    assert math.isclose(float(pb.query_temperature(torch.arange(3), {"coef": 2.0, "every": 1}, torch.float64)[2]), 1 + 2 * math.log(4))
    # a sink is a further score without a value; minus infinity is no sink at all
    s = rnd(4, 6) * 30
    p = pb.sink_softmax(s, 1.3)
    assert torch.allclose(p, torch.softmax(torch.cat([s, torch.full((4, 1), 1.3, dtype=s.dtype)], dim=1), dim=1)[:, :6])
    assert torch.allclose(pb.sink_softmax(s, -math.inf), torch.softmax(s, dim=-1))
    assert torch.allclose(pb.sink_softmax(s[:, :2] / 30, 0.0), torch.exp(s[:, :2] / 30) / (1 + torch.exp(s[:, :2] / 30).sum(-1, keepdim=True)))
    # the two expansions of the latent may move to the other side of the softmax
    m = bh.latent(3, 4, 6, 5, 0.4)
    w = {"q": rnd(12, 8), "dkv": rnd(5, 8), "dkv.norm": rnd(5), "uk": rnd(12, 5), "uv": rnd(18, 5), "sink": rnd(3), "g": rnd(18, 8), "o": rnd(8, 18)}
    h = rnd(9, 8)
    y = pb.latent_attention(h, w, "", m, 1e-5, {}, 0)
    c = pb.latent_of(h, w, "", 1e-5)
    q = torch.einsum("thd,hdr->thr", (h @ w["q"].T).view(9, 3, 4), w["uk"].view(3, 4, 5))
    o = pb.attend(q, c[:, None], c[:, None], 0.4, w["sink"])
    o = torch.einsum("thr,hvr->thv", o, w["uv"].view(3, 6, 5)).reshape(9, 18) * torch.sigmoid(h @ w["g"].T)
    assert torch.allclose(y, o @ w["o"].T)
    # a reader's latents are the owner's, not its own input's
    kept = {}
    pb.latent_attention(h, w, "", m, 1e-5, kept, 3)
    other = rnd(9, 8)
    assert not torch.allclose(pb.latent_attention(other, w, "", dict(m, kv_from=3), 1e-5, kept, 4), pb.latent_attention(other, w, "", m, 1e-5, {}, 4))
    # groups: by the sum of a group's two largest, not by its largest; the group without the best expert can win
    scores = torch.tensor([0.9, 0.1, 0.6, 0.55, 0.2, 0.3], dtype=torch.float64)
    ids, wts = pb.route_one(scores, {"top": 2, "groups": {"count": 3, "keep": 1}})
    assert ids == [2, 3] and math.isclose(wts[0], 0.6 / 1.15) and math.isclose(sum(wts), 1.0)
    assert pb.route_one(scores, {"top": 2, "groups": {"count": 3, "keep": 2}})[0] == [0, 2]
    assert pb.route_one(scores, {"top": 3, "groups": {"count": 6, "keep": 4}})[0] == [0, 2, 3]       # groups of one expert each
    assert pb.route_one(scores, {"top": 6})[0] == [0, 2, 3, 5, 4, 1]
