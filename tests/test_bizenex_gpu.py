"""Bizenex through the engine against the plain implementation: each mechanism alone, whole models, whole prompts against
token-by-token decoding, portions down to two tokens, unequal batches against each request alone, slots and pages that are
used again, keys far back and at page borders, sinks and temperatures made to show, long decoding, greedy generation through
`LLM.generate`; and the kernels' new options on their own against plain torch."""
import math

import pytest
import torch

import bizenex_helpers as bh
import helpers
import plain_bizenex as pb
from bizenex_helpers import check, folder_of, oracle_logits
from helpers import random_tokens
from mini_llama_cpp_release_b200 import kernels
from mini_llama_cpp_release_b200.engine import MiniBatch
from mini_llama_cpp_release_b200.engine.batch import SequenceChunk
from test_mepolix_gpu import run_in_portions

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def vocab_of(name):
    return bh.CONFIGS[name]["vocab"]


# ------------------------------------------------------------------ whole prompts, layer by layer

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, n", [("attention", 150), ("latent", 150), ("moe", 70), ("shared", 160), ("mixed", 150), ("wide", 200),
                                     ("odd", 90)])
def test_whole_prompt_against_plain(name, n, dtype):
    folder = folder_of(name)
    ctx = helpers.engine(folder, dtype).context
    tokens = random_tokens(n, vocab_of(name), 11)
    check(run_in_portions(ctx, tokens, [n]), oracle_logits(folder, tokens), dtype, f"{name} whole prompt", many=n > 100)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_stream_after_every_layer(dtype):
    """The blocks one by one: the float32 stream behind each layer (with the addition the block left for the next one carried
    out) against the plain implementation's."""
    from mini_llama_cpp_release_b200.parts.base import MixerMemory
    from mini_llama_cpp_release_b200.parts.block import DEFERRED, finish_deferred
    for name in ("mixed", "odd"):
        folder = folder_of(name)
        ctx = helpers.engine(folder, dtype).context
        model, cache = ctx.model, ctx.cache
        tokens = random_tokens(75, vocab_of(name), 12)
        cfg, w = bh.oracle(folder)
        want = []
        pb.forward(cfg, w, tokens, want)
        slot = ctx.acquire()
        step = ctx.describe(MiniBatch([SequenceChunk(slot, tokens, [len(tokens) - 1])]))
        x = model.parts.embedding.forward(step.tokens)
        pending = None
        for k, entry in enumerate(model.spec.schedule):
            memory = MixerMemory(kv=cache.view(k, step.page_tables), state=cache.state[k], writes_cache=entry.reads_cache_of is None)
            x, pending = model.parts.blocks[entry.layer].forward(x, pending, step, memory)
            now = x.clone()
            left = step.handover.get(DEFERRED)
            assert (left is not None) == (cfg["layers"][k]["mlp"] is not None) and (left is None or pending is None)
            if left is not None:
                type(left)(now, expert_rows=left.expert_rows).finish()         # on a copy: the next block does it itself
            elif pending is not None:
                now += pending.sum(dim=0) if pending.dim() == 3 else pending
            if dtype == "float32":
                err = helpers.rel_err(now, want[k].float())
                assert err <= 2e-5, (name, k, err)
            else:
                # a router that sees 16-bit inputs may choose another expert for a token whose scores nearly tie, and that
                # token's row is then another row: a few rows are spared
                rows = sorted(helpers.rel_err(now[t], want[k][t].float()) for t in range(now.shape[0]))
                assert rows[int(0.9 * len(rows))] <= 4e-2, (name, k, rows[-8:])
        finish_deferred(step)
        ctx.release(slot)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_tokens_of_a_sequence(dtype):
    """One to five tokens: the first token's softmax holds its own key beside the sink."""
    for name in ("mixed", "wide", "odd"):
        folder = folder_of(name)
        ctx = helpers.engine(folder, dtype).context
        for n in (1, 2, 3, 5):
            tokens = random_tokens(n, vocab_of(name), 20 + n)
            check(run_in_portions(ctx, tokens, [n]), oracle_logits(folder, tokens), dtype, f"{name} first {n}")
            check(run_in_portions(ctx, tokens, list(range(1, n + 1))), oracle_logits(folder, tokens), dtype, f"{name} first {n}, one by one")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide", "odd"])
def test_token_by_token_decoding_equals_the_whole_prompt(name, dtype):
    folder = folder_of(name)
    ctx = helpers.engine(folder, dtype).context
    n = 100
    tokens = random_tokens(n, vocab_of(name), 31)
    want = oracle_logits(folder, tokens)
    check(run_in_portions(ctx, tokens, [20] + list(range(21, n + 1))), want, dtype, f"{name} decoded", many=True)
    if dtype == "float32":
        whole = run_in_portions(ctx, tokens, [n])
        stepped = run_in_portions(ctx, tokens, list(range(1, n + 1)))
        check(stepped, whole, dtype, f"{name} stepped against whole")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_portions_of_several_sizes_down_to_two_tokens(name, dtype):
    folder = folder_of(name)
    ctx = helpers.engine(folder, dtype).context
    n = 140
    tokens = random_tokens(n, vocab_of(name), 41)
    want = oracle_logits(folder, tokens)
    for cuts in ([2, 4, 7, 49, 50, 51, 64, 65, 66, 128, 130, n], [63, 64, 129, n], [1, 3, 100, n]):
        check(run_in_portions(ctx, tokens, cuts), want, dtype, f"{name} portions {cuts}", many=True)
    ctx.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_far_back_and_at_page_borders_in_prompts_and_in_decoding(dtype):
    """A prompt over eleven pages, then short portions (few rows against many keys), then single tokens, every token against
    the plain implementation."""
    for name in ("mixed", "wide"):
        folder = folder_of(name)
        ctx = helpers.engine(folder, dtype).context
        n = 730
        tokens = random_tokens(n, vocab_of(name), 51)
        want = oracle_logits(folder, tokens)
        cuts = [640, 641, 660, 704, 705] + list(range(706, n + 1))
        check(run_in_portions(ctx, tokens, cuts), want, dtype, f"{name} long", many=True)
        ctx.cache.check()


@pytest.mark.parametrize("name", ["attention", "latent", "shared"])
def test_single_keys_decide_the_logits(name):
    """The scores are many times larger, so the softmax of many rows is a choice of one or two keys, wherever among the
    visible ones they lie: hundreds of places back, at page borders, the newest.  A kernel that lost one of them, or read
    another layer's latents, would miss whole rows."""
    folder = folder_of(name, seed=5, peaked=12.0)
    n = 400
    tokens = random_tokens(n, vocab_of(name), 61)
    cfg, w = bh.oracle(folder)
    want = pb.forward(cfg, w, tokens).float()
    m, eps, probs = cfg["layers"][0]["mixer"], cfg["norm"]["eps"], []
    h = pb.layer_norm(w["embed"][torch.as_tensor(tokens)], w, "l0.norm1", eps)
    if name == "attention":
        pb.attention(h, w, "l0.mix.", m, eps, torch.arange(n), probs)
    else:
        pb.latent_attention(h, w, "l0.mix.", m, eps, {}, 0, probs)
    # the plain attention is as peaked as claimed, and some row's favourite key lies far back
    big = torch.stack([p.max(dim=-1).values for p in probs])[:, 100:]
    far = (torch.arange(n) - torch.stack([p.argmax(dim=-1) for p in probs]))[:, 100:]
    assert float((big > 0.5).double().mean()) > 0.05, float((big > 0.5).double().mean())
    assert int(far[big > 0.5].max()) > 250
    for dtype in DTYPES:
        ctx = helpers.engine(folder, dtype).context
        check(run_in_portions(ctx, tokens, [n]), want, dtype, f"{name} peaked, whole", many=True)
        check(run_in_portions(ctx, tokens, [300] + list(range(301, n + 1))), want, dtype, f"{name} peaked, decoded", many=True)
        check(run_in_portions(ctx, tokens, [190, 200, 333, n]), want, dtype, f"{name} peaked, portions", many=True)


def changed_oracle(name, folder, tokens, change):
    """The plain logits with a mistake planted in the plain implementation's weights or configuration."""
    cfg, w = bh.oracle(folder)
    import copy
    cfg, w = copy.deepcopy(cfg), dict(w)
    change(cfg, w)
    return pb.forward(cfg, w, tokens).float()


@pytest.mark.parametrize("what", ["sink", "one more", "temperature", "period", "gate", "norm bias", "owner"])
def test_what_the_mechanisms_do_shows_in_the_logits(what):
    """A mistake planted in the plain implementation moves the logits by many times the bounds that the tests above hold the
    engine to: a sink left out, the one more in the denominator left out, no temperature, a temperature whose period is one
    off, a gate that is always open, a norm without its bias, a reader on other latents."""
    name = {"one more": "attention", "temperature": "attention", "period": "attention", "owner": "shared"}.get(what, "latent")
    folder = folder_of(name)
    tokens = random_tokens(120, vocab_of(name), 65)
    right = oracle_logits(folder, tokens)
    if what == "one more":
        original, pb.sink_softmax = pb.sink_softmax, (lambda s, sink: torch.softmax(s, dim=-1))
        try:
            wrong = changed_oracle(name, folder, tokens, lambda cfg, w: None)
        finally:
            pb.sink_softmax = original
    else:
        def change(cfg, w):
            mix = cfg["layers"][0]["mixer"]
            if what == "sink":
                w["l0.mix.sink"] = torch.full_like(w["l0.mix.sink"], -1e30)
            elif what == "temperature":
                mix.pop("q_temp")
            elif what == "period":
                mix["q_temp"]["every"] += 1
            elif what == "gate":
                w["l0.mix.o"], w["l0.mix.g"] = w["l0.mix.o"] * 0.5, torch.zeros_like(w["l0.mix.g"])
            elif what == "norm bias":
                w["l0.norm1.b"] = torch.zeros_like(w["l0.norm1.b"])
            elif what == "owner":
                cfg["layers"][1]["mixer"].pop("kv_from")
                w["l1.mix.dkv"], w["l1.mix.dkv.norm"] = w["l0.mix.dkv"], w["l0.mix.dkv.norm"]
        wrong = changed_oracle(name, folder, tokens, change)
    moved = max(helpers.rel_err(wrong[t], right[t]) for t in range(len(tokens)))
    assert moved > 1e-2 if what != "period" else moved > 1e-3, (what, moved)
    got = run_in_portions(helpers.engine(folder, "float32").context, tokens, [40, 41, 90, 120])
    check(got, right, "float32", f"{what} in place")


# ------------------------------------------------------------------ batches, slots, pages

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide", "odd"])
def test_a_batch_of_unequal_requests_equals_each_alone(name, dtype):
    folder = folder_of(name)
    ctx = helpers.engine(folder, dtype).context
    lens = [1, 66, 130, 17, 2]
    prompts = [random_tokens(n + 6, vocab_of(name), 70 + i) for i, n in enumerate(lens)]
    slots = [ctx.acquire() for _ in prompts]
    got = [[] for _ in prompts]
    logits = ctx.forward_batch(MiniBatch([SequenceChunk(s, p[:n], list(range(n))) for s, p, n in zip(slots, prompts, lens)]))
    row = 0
    for i, n in enumerate(lens):
        got[i].append(logits[row:row + n].float().cpu())
        row += n
    live = list(range(len(prompts)))
    for step in range(6):                               # the shorter-lived requests leave one by one
        live = [i for i in live if step < 6 - i or i == 0]
        logits = ctx.forward_batch(MiniBatch.decode([slots[i] for i in live], [prompts[i][lens[i] + step] for i in live]))
        for r, i in enumerate(live):
            got[i].append(logits[r:r + 1].float().cpu())
    for s in slots:
        ctx.release(s)
    mine = [torch.cat(rows) for rows in got]
    want = [oracle_logits(folder, p)[:m.shape[0]] for p, m in zip(prompts, mine)]
    if dtype == "float32":
        for i, p in enumerate(prompts):
            check(mine[i], want[i], dtype, f"{name} request {i} in a batch", many=mine[i].shape[0] > 32)
            alone = run_in_portions(ctx, p[:mine[i].shape[0]], [lens[i]] + list(range(lens[i] + 1, mine[i].shape[0] + 1)))
            check(mine[i], alone, dtype, f"{name} request {i}: batch against alone")
    else:
        # a router that sees 16-bit inputs may choose otherwise where two scores nearly tie; the rows of all requests are held
        # to the bound together, so that the few such rows are spared whichever request they fall into
        check(torch.cat(mine), torch.cat(want), dtype, f"{name} requests in a batch", many=True)
    ctx.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_beside_single_tokens_in_one_step(dtype):
    """Some requests of a step go on by one token while others bring a portion of a prompt or start."""
    folder = folder_of("mixed")
    ctx = helpers.engine(folder, dtype).context
    prompts = [random_tokens(n, vocab_of("mixed"), 75 + n) for n in (150, 90, 64)]
    plan = [[(0, 70)], [(0, 1), (1, 65)], [(0, 1), (1, 2), (2, 63)], [(0, 40), (1, 1), (2, 1)], [(0, 38), (1, 22)]]
    slots, at = [ctx.acquire() for _ in prompts], [0, 0, 0]
    got = [[] for _ in prompts]
    for entries in plan:
        chunks = [SequenceChunk(slots[i], prompts[i][at[i]:at[i] + n], list(range(n))) for i, n in entries]
        logits = ctx.forward_batch(MiniBatch(chunks)).float().cpu()
        row = 0
        for i, n in entries:
            got[i].append(logits[row:row + n])
            row, at[i] = row + n, at[i] + n
    assert at == [150, 90, 64]
    for s in slots:
        ctx.release(s)
    mine = torch.cat([torch.cat(rows) for rows in got])
    check(mine, torch.cat([oracle_logits(folder, p) for p in prompts]), dtype, "a mixed step", many=True)


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_that_are_used_again_start_from_nothing(dtype):
    folder = folder_of("mixed")
    ctx = helpers.engine(folder, dtype).context
    a = random_tokens(200, vocab_of("mixed"), 81)
    b = random_tokens(90, vocab_of("mixed"), 82)
    s = ctx.acquire()
    ctx.forward_batch(MiniBatch.from_tokens(s, a))
    ctx.release(s)
    s2 = ctx.acquire()
    assert s2 == s                                       # the slot and its pages are the ones a used
    got = ctx.forward_batch(MiniBatch([SequenceChunk(s2, b[:60], list(range(60)))])).float().cpu()
    rest = torch.cat([ctx.forward_batch(MiniBatch.single(s2, t)).float().cpu() for t in b[60:]])
    ctx.release(s2)
    check(torch.cat([got, rest]), oracle_logits(folder, b), dtype, "a slot used again")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_batch_larger_than_a_step_is_cut_and_changes_nothing(dtype):
    import mini_llama_cpp_release_b200 as ml
    folder = folder_of("mixed")
    llm = ml.load(folder, dtype=dtype, max_tokens=1024, max_batch_tokens=50)
    prompts = [random_tokens(n, vocab_of("mixed"), 90 + n) for n in (70, 45, 120)]
    slots = [llm.context.acquire() for _ in prompts]
    logits = llm.context.forward_batch(MiniBatch([SequenceChunk(s, p, [0, len(p) // 2, len(p) - 1]) for s, p in zip(slots, prompts)]))
    want = torch.cat([oracle_logits(folder, p)[[0, len(p) // 2, len(p) - 1]] for p in prompts])
    check(logits.float().cpu(), want, dtype, "cut batch")


# ------------------------------------------------------------------ generation

def confident_greedy(folder, prompt, n, margin=2e-4):
    cfg, w = bh.oracle(folder)
    ids, sure = list(prompt), 0
    undecided = False
    for _ in range(n):
        row = pb.forward(cfg, w, ids)[-1]
        top = torch.topk(row, 2).values
        if not undecided and float(top[0] - top[1]) > margin:
            sure += 1
        else:
            undecided = True
        ids.append(int(torch.argmax(row)))
    return ids[len(prompt):], sure


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_greedy_generation_through_generate_matches_plain(name):
    folder = folder_of(name)
    llm = helpers.engine(folder, "float32")
    prompts = [random_tokens(n, vocab_of(name), 100 + n) for n in (5, 1, 33, 70)]
    out = llm.generate(prompts, n_predict=24, stop_token_ids=[])
    total = 0
    for p, got in zip(prompts, out):
        want, sure = confident_greedy(folder, p, 24)
        assert len(got) == 24 and got[:sure] == want[:sure], (got, want, sure)
        total += sure
    assert total >= 48, total
    llm.context.cache.check()
    assert llm.context.cache.slots.n_held == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_through_the_captured_step(dtype):
    """150 generated tokens through the decode runner's graph; page borders and many steps of the temperatures lie among them;
    each step's logits against the plain implementation run on the ids the engine chose."""
    folder = folder_of("mixed")
    llm = helpers.engine(folder, dtype)
    prompts = [random_tokens(50, vocab_of("mixed"), 121), random_tokens(3, vocab_of("mixed"), 122)]
    seen = []
    out = llm.generate(prompts, n_predict=150, stop_token_ids=[],
                       on_step=lambda live, chosen, logits: seen.append((list(live), logits.float().cpu().clone())))
    assert llm.context.use_graphs
    refs = [oracle_logits(folder, p + o) for p, o in zip(prompts, out)]
    for i in range(len(prompts)):
        got = torch.stack([logits[live.index(i)] for live, logits in seen if i in live])
        assert got.shape[0] == 150
        check(got, refs[i][len(prompts[i]) - 1:len(prompts[i]) - 1 + 150], dtype, f"generated tokens of request {i}", many=True)


# ------------------------------------------------------------------ the kernels on their own

@pytest.mark.parametrize("n, d", [(37, 96), (1, 100), (200, 128), (130, 1536), (9, 2048), (140, 2052), (300, 41), (3, 12)])
def test_layer_norm_with_a_bias_after_slices_or_expert_rows(n, d):
    g = torch.Generator().manual_seed(n + d)
    rnd = lambda *s: torch.randn(*s, generator=g).cuda()
    x, gain, bias, y, rows = rnd(n, d) + 0.7, rnd(d), rnd(d), rnd(3, n, d), rnd(50, d)
    top = 3
    row_of = torch.randint(0, 50, (n, top), generator=g).int().cuda()
    weights = torch.rand(n, top, generator=g).cuda()
    summed = (weights.double()[:, :, None] * rows[row_of.long()].double()).sum(1)
    ln = lambda v, b: torch.nn.functional.layer_norm(v, (d,), gain.double(), b.double() if b is not None else None, 1e-5)
    for out_dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 5e-3)):
        out = torch.empty(n, d, dtype=out_dtype, device="cuda")
        for b in (bias, None):
            stream = x.clone()
            kernels.layernorm(stream, None, gain, 1e-5, out, of_branch=False, bias=b)
            assert torch.equal(stream, x) and helpers.rel_err(out, ln(x.double(), b)) <= tol
            kernels.layernorm(stream, y, gain, 1e-5, out, of_branch=False, bias=b)
            want = x.double() + y.double().sum(0)
            assert helpers.rel_err(stream, want) <= 1e-6 and helpers.rel_err(out, ln(want, b)) <= tol
            stream = x.clone()
            kernels.layernorm(stream, None, gain, 1e-5, out, of_branch=False, bias=b, expert_rows=(rows, row_of, weights))
            want = x.double() + summed
            assert helpers.rel_err(stream, want) <= 1e-6 and helpers.rel_err(out, ln(want, b)) <= tol
            stream = x.clone()
            kernels.layernorm(stream, y, gain, 1e-5, out, of_branch=True, bias=b)
            want = x.double() + ln(y.double().sum(0), b)
            assert helpers.rel_err(stream, want) <= 3e-6 and helpers.rel_err(out, want) <= tol
    # the experts' sum alone, for whoever reads the stream without a norm of this kind
    stream = x.clone()
    kernels.scaled_add_experts(stream, None, None, rows, row_of, weights, None)
    assert helpers.rel_err(stream, x.double() + summed) <= 1e-6


@pytest.mark.parametrize("n, E, top, count, keep", [(50, 6, 2, 3, 2), (1, 4, 4, 2, 2), (300, 33, 3, 11, 4), (17, 200, 7, 8, 3),
                                                    (80, 8, 1, 8, 3), (40, 9, 2, 1, 1), (60, 64, 6, 2, 1)])
def test_routing_by_sigmoid_scores_inside_the_best_groups(n, E, top, count, keep):
    g = torch.Generator().manual_seed(n + E)
    K = 72
    router = torch.randn(E, K, generator=g).cuda() * 0.3
    cfg = {"top": top, "groups": {"count": count, "keep": keep}}
    for dtype in (torch.float32, torch.bfloat16):
        hx = torch.randn(n, K, generator=g).to(dtype).cuda()
        ids = torch.empty(n, top, dtype=torch.int32, device="cuda")
        wts = torch.empty(n, top, dtype=torch.float32, device="cuda")
        kernels.moe_route_scored(hx, router, None, top, count, keep, 1.0, ids, wts, score="sigmoid", group_score="top2")
        s = torch.sigmoid(hx.double() @ router.double().t()).cpu()
        right = seen = 0
        for t in range(n):
            want_ids, want_w = pb.route_one(s[t], cfg)
            near = sorted(s[t].tolist())
            if min((b - a for a, b in zip(near, near[1:])), default=1.0) < 1e-6:
                continue                          # scores too close for float32 to tell apart
            seen += 1
            if ids[t].tolist() == want_ids:
                right += 1
                assert torch.allclose(wts[t].cpu().double(), torch.tensor(want_w, dtype=torch.float64), atol=1e-6, rtol=1e-5)
        assert seen >= n * 0.5 and right >= seen * 0.98 - 1, (right, seen, n)
        assert torch.allclose(wts.sum(-1), torch.ones(n, device="cuda"), atol=1e-5)


def test_the_routers_two_group_scores_and_two_kinds_of_scores_are_different_rules():
    """One token whose best expert's group loses by the sum of two and wins by the largest; the softmax form keeps its own."""
    router = torch.diag(torch.tensor([3.0, 0.2, 1.5, 1.4, 0.1, 0.3])).cuda()
    hx = torch.ones(1, 6).cuda()
    ids = torch.empty(1, 2, dtype=torch.int32, device="cuda")
    wts = torch.empty(1, 2, dtype=torch.float32, device="cuda")
    z = torch.tensor([3.0, 0.2, 1.5, 1.4, 0.1, 0.3], dtype=torch.float64)
    for score, group, chosen in (("sigmoid", "top2", [2, 3]), ("sigmoid", "max", [0, 1]), ("softmax", "max", [0, 1]), ("softmax", "top2", [0, 1])):
        kernels.moe_route_scored(hx, router, None, 2, 3, 1, 1.0, ids, wts, score=score, group_score=group)
        s = torch.sigmoid(z) if score == "sigmoid" else torch.softmax(z, dim=0)
        assert ids[0].tolist() == chosen, (score, group)
        assert torch.allclose(wts[0].cpu().double(), s[chosen] / s[chosen].sum(), atol=1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_query_norm_without_a_gain_and_the_temperature(dtype):
    from test_kernels_gpu import make_paged
    g = torch.Generator().manual_seed(4)
    H, KV, dim, vdim, D, n, start = 4, 2, 20, 28, 32, 70, 30
    proj = torch.randn(n, 3 + H * dim + KV * (dim + vdim), generator=g)
    kv = make_paged([torch.zeros(start + n, KV, D)], [torch.zeros(start + n, KV, D)], dtype)
    positions = torch.arange(start, start + n, dtype=torch.int32, device="cuda")
    tok_seq = torch.zeros(n, dtype=torch.int32, device="cuda")
    for temp in (None, (0.7, 1), (0.7, 16), (2.0, 1000)):
        q = torch.full((n, H * D), 9.0, dtype=dtype, device="cuda")
        kernels.qk_norm_rope_cache(proj.cuda(), 3, 3 + H * dim, 3 + (H + KV) * dim, None, None, 1e-5, positions, tok_seq, None, 0, H, KV,
                                   dim, vdim, 1.0, q, kv, q_temp=temp)
        factor = pb.query_temperature(positions.cpu().long(), dict(zip(("coef", "every"), temp)) if temp else None, torch.float64)
        want = torch.zeros(n, H, D, dtype=torch.float64)
        want[:, :, :dim] = pb.unit_rms(proj[:, 3:3 + H * dim].double().view(n, H, dim), 1e-5) * factor[:, None, None]
        assert helpers.rel_err(q.view(n, H, D), want) <= (2e-6 if dtype == torch.float32 else 5e-3), temp
        keys = pb.unit_rms(proj[:, 3 + H * dim:3 + (H + KV) * dim].double().view(n, KV, dim), 1e-5)      # the keys stay as they are
        for t in (0, 33, 34, n - 1):
            p = start + t
            page = int(kv.page_table[0, p // kv.page_size])
            pool = kv.k_pool.view(-1)[kv.entry_offset:].view(-1, KV, kv.page_size, D)
            assert helpers.rel_err(pool[page, :, p % kv.page_size, :dim], keys[t]) <= (2e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("n, H, n_in, n_out, pad", [(5, 3, 20, 28, 4), (130, 2, 128, 66, 8), (1, 7, 48, 80, 0), (16, 2, 136, 64, 8),
                                                    (17, 5, 264, 40, 8), (200, 1, 8, 200, 0), (64, 4, 512, 128, 16), (33, 2, 30, 15, 1)])
@pytest.mark.parametrize("rows_of_d", [True, False])
def test_per_head_product_in_both_layouts_with_and_without_a_gate(n, H, n_in, n_out, pad, rows_of_d):
    """The float32-arithmetic form and, for 16-bit weights of sizes it takes, the tensor-core form.  The inputs are a constant
    plus a small part and the weights' rows add up to zero, so an input that was only kept in 16 bits would show."""
    g = torch.Generator().manual_seed(6)
    src = torch.randn(n, H, n_in + pad, generator=g)
    w = torch.randn(H, n_out, n_in, generator=g)
    gate = torch.randn(n, 5 + H * n_out, generator=g) * 2
    for in_dtype, w_dtype, out_dtype in ((torch.float32, torch.float32, torch.float32), (torch.float32, torch.bfloat16, torch.bfloat16),
                                         (torch.bfloat16, torch.bfloat16, torch.bfloat16)):
        x = src
        ww = w.to(w_dtype)
        if in_dtype == torch.float32:
            x = src + 64.0
            half = n_in // 2
            ww = ww.clone()
            ww[..., half:2 * half] = -ww[..., :half]
            ww[..., 2 * half:] = 0
        s = x.to(in_dtype).cuda()
        stored = (ww if rows_of_d else ww.transpose(1, 2)).contiguous().cuda()               # [H][j][d] or [H][d][j]
        strides = (n_out * n_in, 1, n_in) if rows_of_d else (n_out * n_in, n_out, 1)
        out = torch.full((n, H * n_out + 2), 7.0, dtype=out_dtype, device="cuda")
        args = (s, (H * (n_in + pad), n_in + pad), stored, strides, out, (H * n_out + 2, n_out), n, H, n_in, n_out)
        want = torch.einsum("thd,hjd->thj", s[:, :, :n_in].double().cpu(), ww.double()).reshape(n, H * n_out)
        tol = 1e-4 if out_dtype == torch.float32 else 5e-3           # the constant part cancels: float32 keeps six digits of it
        kernels.head_project(*args)
        assert helpers.rel_err(out[:, :H * n_out], want) <= tol, (in_dtype, w_dtype)
        kernels.head_project(*args, gate=gate.cuda(), gate_col=5)
        assert helpers.rel_err(out[:, :H * n_out], want * torch.sigmoid(gate[:, 5:].double())) <= tol, (in_dtype, w_dtype)
        assert bool((out[:, H * n_out:] == 7.0).all())                                        # nothing beyond the heads' columns
