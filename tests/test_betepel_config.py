"""Betepel without a GPU: its configuration, what its layers ask of the cache, the names of its tensors, the frequencies, the
random-weights mode's table, and the plain implementation's mechanisms against each other."""
import copy
import math

import pytest
import torch

import betepel_helpers as bh
import plain_betepel as pb
from mini_llama_cpp_release_b200.cache.paged import plan_groups
from mini_llama_cpp_release_b200.config import ModelConfig
from mini_llama_cpp_release_b200.config.model_config import ConfigError
from mini_llama_cpp_release_b200.config.registry import build_model_spec
from mini_llama_cpp_release_b200.engine.model import build_parts
from mini_llama_cpp_release_b200.parts.base import CacheNeed
from mini_llama_cpp_release_b200.parts.rotary import stretched_frequencies

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
    assert cfg.architecture == "Betepel" and cfg.vocab_size == 300 and cfg.hidden_size == 112
    assert (cfg.logit_scale, cfg.norm_eps) == (1.5, 1e-5)
    assert ModelConfig.from_dict(cfg.to_dict()) == cfg
    for path, value in [(("layers", 0, "type"), "gla"), (("layers", 0, "mlp", "kind"), "dense"), (("norm", "eps"), 0.0),
                        (("logit_scale",), "2"), (("layers", 3, "mixer", "kv_from"), 3), (("layers", 3, "mixer", "kv_from"), 1),
                        (("layers", 5, "mixer", "kv_from"), 3), (("layers", 3, "mixer", "vdim"), 24), (("layers", 3, "mixer", "kv_heads"), 1),
                        (("layers", 3, "mixer", "dim"), 20), (("layers", 2, "mixer", "kv_from"), 0), (("layers", 3, "mixer", "kv_from"), True)]:
        with pytest.raises(ConfigError):
            ModelConfig.from_dict(changed(bh.MIXED, path, value))
    # what the parts refuse when the model is built
    for path, value in [(("layers", 0, "mixer", "kv_heads"), 4), (("layers", 0, "mixer", "scale"), 0.0), (("layers", 0, "mixer", "rot", "dims"), 26),
                        (("layers", 0, "mixer", "rot", "dims"), 7), (("layers", 0, "mixer", "mask", "size"), 0),
                        (("layers", 0, "mlp", "router", "top"), 7), (("layers", 1, "mixer", "right", "decay"), [0.5]),
                        (("layers", 2, "mixer", "gate_cap"), 0.0), (("layers", 2, "mixer", "dim"), 300), (("layers", 0, "mlp", "shared", "ff"), 0)]:
        with pytest.raises((ConfigError, ValueError)):
            build_parts(build_model_spec(ModelConfig.from_dict(changed(bh.MIXED, path, value))))


def test_what_the_layers_ask_of_the_cache_and_which_tensors_they_read():
    spec = build_model_spec(ModelConfig.from_dict(bh.MIXED))
    assert [(e.layer, e.reads_cache_of) for e in spec.schedule] == [(0, None), (1, None), (2, None), (3, 0), (4, None), (5, 0)]
    assert all(l.block.kind == "parallel_prenorm" for l in spec.layers)
    parts = build_parts(spec)
    mixers = [parts.blocks[e.layer].mixer for e in spec.schedule]
    needs = [m.cache_need() for m in mixers]
    # layer 0 is read under another mask by layer 5, so it keeps every key; a key row holds both maps (2 · 24, rounded to 16)
    assert needs[0] == CacheNeed("all", 3, 48) and needs[3] == CacheNeed("window", 3, 48, 30, 7)
    assert needs[1] == CacheNeed("window", 2, 32, 21) and needs[2] is None and needs[4] is None
    groups, where = plan_groups(needs, [e.reads_cache_of for e in spec.schedule])
    assert len(groups) == 2 and where[3] == where[5] == where[0] and sum(len(g.entries) for g in groups) == 2
    states = [m.state_spec() if hasattr(m, "state_spec") else None for m in mixers]
    assert [s.shape[0] if s is not None else 0 for s in states] == [0, 3 * 24 * 12, 3 * 29 * 20 + 3, 0, 2 * 21 * 36 + 2, 0]
    names = {t.name: tuple(t.shape) for p in parts.all_parts() for t in p.all_tensors()}
    assert names["embed"] == (300, 112) and "head" not in names and names["embed.norm"] == names["final.norm"] == (112,)
    assert names["l0.norm2"] == (112,) and "l2.norm2" not in names and not any(k.startswith("l2.mlp") for k in names)
    assert names["l0.mix.q"] == (288, 112) and names["l0.mix.q.b"] == (288,) and names["l0.mix.k"] == (144, 112) and names["l0.mix.k.b"] == (144,)
    assert names["l0.mix.v"] == (120, 112) and names["l0.mix.g"] == (6, 112) and names["l0.mix.o"] == (112, 240) and names["l0.mix.lk2"] == (24,)
    assert not any(k.startswith(("l3.mix.k", "l3.mix.v", "l5.mix.k", "l5.mix.v")) for k in names) and names["l5.mix.q"] == (144, 112)
    assert names["l1.mix.left.v.b"] == (56,) and names["l1.mix.right.g"] == (36, 112) and names["l1.mix.right.norm"] == (36,)
    assert names["l2.mix.i"] == (3, 112) and names["l2.mix.f.b"] == (3,) and names["l2.mix.norm"] == (84,) and names["l2.mix.o"] == (112, 84)
    assert names["l0.mlp.table"] == (300, 2) and names["l0.mlp.e5.gate"] == (48, 112) and names["l0.mlp.shared.down"] == (112, 56)
    assert "l0.mlp.e6.up" not in names and "l0.mlp.router" not in names and not any(k.startswith("l3.mlp.shared") for k in names)
    # an owner that only readers of its own mask read keeps its window, and so does one that nobody reads
    same = copy.deepcopy(bh.MIXED)
    same["layers"][5]["mixer"]["mask"] = dict(same["layers"][0]["mixer"]["mask"])
    first = build_parts(build_model_spec(ModelConfig.from_dict(same))).blocks[0].mixer
    assert first.cache_need() == CacheNeed("window", 3, 48, 30, 7)


def test_a_reader_that_keeps_more_first_keys_than_the_owner_is_refused():
    owner, reader = CacheNeed("window", 2, 32, 40, 4), CacheNeed("window", 2, 32, 40, 5)
    plan_groups([owner, CacheNeed("window", 2, 32, 30, 4)], [None, 0])
    with pytest.raises(ValueError, match="first 5"):
        plan_groups([owner, reader], [None, 0])


@pytest.mark.parametrize("dims, base, scaling", [(12, 1000.0, bh.SLOW), (64, 500000.0, (8.0, 1.0, 4.0, 8192)), (24, 1e6, (2.0, 2.0, 3.0, 64)),
                                                 (16, 100.0, (4.0, 1.0, 1.0, 50)), (8, 10.0, (3.0, 1.0, 4.0, 100000)), (8, 1e4, (3.0, 1.0, 4.0, 2))])
def test_frequencies_stretched_by_wavelength(dims, base, scaling):
    f, mult = stretched_frequencies(dims, base, dict(zip(("factor", "low", "high", "original"), scaling)))
    want = pb.frequencies(bh.rot(dims, base, scaling))
    assert mult == 1.0 and torch.allclose(torch.from_numpy(f).double(), want, rtol=1e-6)
    plain = pb.frequencies(bh.rot(dims, base))
    assert torch.all(want <= plain) and torch.all(want >= plain / scaling[0] * (1 - 1e-12))
    with pytest.raises(ValueError):
        stretched_frequencies(dims, base, dict(factor=0.0, low=1.0, high=4.0, original=64))
    with pytest.raises(ValueError):
        stretched_frequencies(dims, base, dict(factor=2.0, low=4.0, high=1.0, original=64))


def test_the_slow_rotation_of_the_tests_has_all_three_kinds_of_pairs():
    kept, plain = pb.frequencies(bh.rot(12, 1000.0, bh.SLOW)), pb.frequencies(bh.rot(12, 1000.0))
    ratio = plain / kept
    assert float(ratio[0]) == 1.0 and math.isclose(float(ratio[-1]), 4.0) and any(1.0 < float(r) < 3.999 for r in ratio)


def test_random_tables_hold_different_experts_in_a_row():
    from safetensors.torch import load_file
    import os
    w = load_file(os.path.join(bh.folder_of("mixed"), "model.safetensors"))
    table = w["l3.mlp.table"]
    assert table.dtype == torch.int32 and table.shape == (300, 3) and int(table.min()) == 0 and int(table.max()) == 6
    assert all(len(set(row)) == 3 for row in table.tolist()) and sorted(set(w["l4.mlp.table"][0].tolist())) == [0, 1, 2, 3]
    assert not torch.equal(w["l0.mlp.table"][:, 0], w["l5.mlp.table"][:, 0])


def test_plain_mechanisms_against_each_other():
    # the two maps: with lambda = 0 what is left is ordinary attention of the first map, normed
    m = bh.attention(4, 2, 6, 10, 0.4, 0.0, bh.rot(4, 100.0), 5, 2)
    w = {"q": rnd(48, 8), "q.b": rnd(48), "k": rnd(24, 8), "k.b": rnd(24), "v": rnd(20, 8), "v.b": rnd(20), "g": torch.zeros(4, 8, dtype=torch.float64),
         "o": rnd(8, 40), **{n: torch.zeros(6, dtype=torch.float64) for n in ("lq1", "lk1", "lq2", "lk2")}}
    h, pos = rnd(14, 8), torch.arange(14)
    kept = {}
    y = pb.diff_attention(h, w, "", m, 1e-6, pos, kept, 7)
    first = pb.softmax_map(pb.rotate((h @ w["q"].T + w["q.b"]).view(14, 4, 2, 6)[:, :, 0], m["rot"], pos), kept[7][0], kept[7][2], 0.4, pb.visible(14, m["mask"]))
    assert torch.allclose(y, (pb.unit_rms(first, 1e-6) * 0.5).reshape(14, 40) @ w["o"].T)
    # one map's score is the score of a padded query against both maps' keys in one row
    k1, k2, _ = kept[7]
    q = rnd(14, 6)
    assert torch.allclose(torch.cat([torch.zeros_like(q), q], 1) @ torch.cat([k1[:, 0], k2[:, 0]], 1).T, q @ k2[:, 0].T)
    assert torch.allclose(pb.diff_lambda(dict(w, lq1=rnd(6) * 0, lk1=rnd(6)), "", 0.3), torch.tensor(0.3, dtype=torch.float64))
    # a reader's keys and values are the owner's
    other = rnd(14, 8)
    again = pb.diff_attention(other, w, "", dict(m, kv_from=7), 1e-6, pos, kept, 8)
    assert not torch.allclose(again, pb.diff_attention(other, w, "", m, 1e-6, pos, {}, 8))
    # windows: exactly `size` keys, and the first ones
    ok = pb.visible(12, {"size": 3, "keep_first": 2})
    assert ok[11].tolist() == [True, True] + [False] * 7 + [True] * 3 and ok[2].tolist() == [True] * 3 + [False] * 9
    assert pb.visible(9, {"size": 1})[5].tolist() == [False] * 5 + [True] + [False] * 3 and torch.equal(pb.visible(5, None), torch.ones(5, 5).tril().bool())
    # rotation: a shift of both positions changes no score; entries behind `dims` pass
    x, r = rnd(2, 1, 8), bh.rot(4, 50.0, (2.0, 1.0, 2.0, 40))
    a, b = pb.rotate(x, r, torch.tensor([3, 9])), pb.rotate(x, r, torch.tensor([10, 16]))
    assert torch.allclose((a[0] * a[1]).sum(), (b[0] * b[1]).sum()) and torch.equal(a[..., 4:], x[..., 4:])
    # constant decay: the walk is a sum over all earlier tokens
    q, k, v = rnd(9, 2, 4), rnd(9, 2, 4), rnd(9, 2, 3)
    o = pb.decay_walk(q, k, v, (0.9, 0.5))
    want = sum((0.5 ** (8 - j)) * (k[j, 1] @ q[8, 1]) * v[j, 1] for j in range(9))
    assert torch.allclose(o[8, 1], want)
    # the running maximum only stabilises: the same numbers without it (m = 0 throughout gives exp(-m) = 1, so weigh by hand)
    i, f = rnd(9, 2) * 2, torch.nn.functional.logsigmoid(rnd(9, 2))
    o = pb.memory_walk(q, k, v, i, f)
    S, n, top = torch.zeros(2, 4, 3, dtype=torch.float64), torch.zeros(2, 4, dtype=torch.float64), torch.zeros(2, dtype=torch.float64)
    for t in range(9):
        S = torch.exp(f[t])[:, None, None] * S + torch.exp(i[t])[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = torch.exp(f[t])[:, None] * n + torch.exp(i[t])[:, None] * k[t]
        top = torch.maximum(f[t] + top, i[t])
    size = torch.maximum((n * q[8]).sum(-1).abs(), torch.ones(2, dtype=torch.float64)) + 1e-6 * torch.exp(top)
    assert torch.allclose(o[8], (S * q[8][:, :, None]).sum(1) / size[:, None])
    # experts by the token's id: the same id, the same experts; the weights are equal
    mlp = bh.moe(4, 3, 2, 5)
    w = {f"e{e}.{r}": rnd(*s) for e in range(3) for r, s in (("gate", (4, 6)), ("up", (4, 6)), ("down", (6, 4)))}
    w.update({"shared.gate": rnd(5, 6), "shared.up": rnd(5, 6), "shared.down": rnd(6, 5), "table": torch.tensor([[0, 2], [1, 0]])})
    hh = rnd(3, 6)
    y = pb.table_moe(hh, w, "", mlp, torch.tensor([1, 0, 1]))
    assert torch.allclose(y[1], 0.5 * pb.expert(hh[1], w, "e0.") + 0.5 * pb.expert(hh[1], w, "e2.") + pb.expert(hh[1], w, "shared."))
