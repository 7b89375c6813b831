"""Betepel through the engine against the plain implementation: each mechanism alone, whole models, whole prompts against
token-by-token decoding, portions down to two tokens, unequal batches against each request alone, slots and pages that are
used again, keys far back, at page borders and at the edges of every window, long decoding, greedy generation through
`LLM.generate`; and the kernels on their own against plain torch."""
import copy

import pytest
import torch

import betepel_helpers as bh
import helpers
import plain_betepel as pb
from betepel_helpers import check, folder_of, oracle_logits
from helpers import random_tokens
from mini_llama_cpp_release_b200 import kernels
from mini_llama_cpp_release_b200.engine import MiniBatch
from mini_llama_cpp_release_b200.engine.batch import SequenceChunk
from test_mepolix_gpu import run_in_portions, step_of

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def vocab_of(name):
    return bh.CONFIGS[name]["vocab"]


# ------------------------------------------------------------------ whole prompts, layer by layer

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, n", [("attention", 150), ("parallel", 150), ("mlstm", 150), ("moe", 70), ("shared", 160), ("mixed", 150),
                                     ("wide", 200), ("odd", 90)])
def test_whole_prompt_against_plain(name, n, dtype):
    folder = folder_of(name)
    ctx = helpers.engine(folder, dtype).context
    tokens = random_tokens(n, vocab_of(name), 11)
    check(run_in_portions(ctx, tokens, [n]), oracle_logits(folder, tokens), dtype, f"{name} whole prompt")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_stream_after_every_layer(dtype):
    """The blocks one by one: the float32 stream behind each layer (with the addition the block left for the next one carried
    out) against the plain implementation's."""
    from mini_llama_cpp_release_b200.parts.base import MixerMemory
    from mini_llama_cpp_release_b200.parts.block import DEFERRED, finish_deferred
    for name in ("mixed", "odd", "wide"):
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
        assert helpers.rel_err(x, pb.embed(cfg, w, torch.as_tensor(tokens)).float()) <= 1e-6
        pending = None
        for k, entry in enumerate(model.spec.schedule):
            memory = MixerMemory(kv=cache.view(k, step.page_tables), state=cache.state[k], writes_cache=entry.reads_cache_of is None)
            x, pending = model.parts.blocks[entry.layer].forward(x, pending, step, memory)
            now = x.clone()
            left = step.handover.get(DEFERRED)
            assert (left is not None) == (cfg["layers"][k]["mlp"] is not None)
            if left is not None:
                type(left)(now, expert_rows=left.expert_rows).finish()         # on a copy: the next block does it itself
            if pending is not None:
                now += pending.sum(dim=0) if pending.dim() == 3 else pending
            err = helpers.rel_err(now, want[k].float())
            assert err <= (2e-5 if dtype == "float32" else 1e-1), (name, k, err)
            rows = sorted(helpers.rel_err(now[t], want[k][t].float()) for t in range(now.shape[0]))
            assert rows[int(0.9 * len(rows))] <= (2e-5 if dtype == "float32" else 5e-2), (name, k, rows[-8:])
        finish_deferred(step)
        ctx.release(slot)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_tokens_of_a_sequence(dtype):
    """One to five tokens: the first token's softmax holds its own key alone, memories start from nothing, the running maximum
    from zero."""
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
    n = 140
    tokens = random_tokens(n, vocab_of(name), 31)
    want = oracle_logits(folder, tokens)
    check(run_in_portions(ctx, tokens, [20] + list(range(21, n + 1))), want, dtype, f"{name} decoded")
    if dtype == "float32":
        whole = run_in_portions(ctx, tokens, [n])
        stepped = run_in_portions(ctx, tokens, list(range(1, n + 1)))
        check(stepped, whole, dtype, f"{name} stepped against whole")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide", "odd"])
def test_portions_of_several_sizes_down_to_two_tokens(name, dtype):
    folder = folder_of(name)
    ctx = helpers.engine(folder, dtype).context
    n = 140
    tokens = random_tokens(n, vocab_of(name), 31)
    want = oracle_logits(folder, tokens)
    for cuts in ([2, 4, 7, 49, 50, 51, 64, 65, 66, 128, 130, n], [63, 64, 129, n], [1, 3, 100, n], list(range(2, n + 1, 2))):
        check(run_in_portions(ctx, tokens, cuts), want, dtype, f"{name} portions {cuts[:6]}")
    ctx.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_windows_that_have_passed_pages_in_prompts_and_in_decoding(dtype):
    """A prompt over eight pages, then short portions (few rows against many keys), then single tokens, every token against the
    plain implementation; the pages that a window has left are given back on the way, those of kept first tokens are not."""
    for name in ("mixed", "wide"):
        folder = folder_of(name)
        ctx = helpers.engine(folder, dtype).context
        n = 560
        tokens = random_tokens(n, vocab_of(name), 51)
        want = oracle_logits(folder, tokens)
        cuts = [470, 471, 490, 512, 513] + list(range(514, n + 1))
        check(run_in_portions(ctx, tokens, cuts), want, dtype, f"{name} long")
        ctx.cache.check()


def favourites(name, n, tokens):
    """Of the first layer's softmax maps in the plain implementation: how sure rows are of a key, and how far back it lies."""
    folder = folder_of(name, seed=5, peaked=14.0)
    cfg, w = bh.oracle(folder)
    m, eps, probs = cfg["layers"][0]["mixer"], cfg["norm"]["eps"], []
    h = pb.rms_norm(pb.embed(cfg, w, torch.as_tensor(tokens)), w["l0.norm1"], eps)
    if name == "parallel":
        pb.window_attention(h, w, "l0.mix.left.", m["left"], torch.arange(n), probs)
    else:
        pb.diff_attention(h, w, "l0.mix.", m, eps, torch.arange(n), {}, 0, probs)
    big = torch.stack([p.max(dim=-1).values for p in probs])
    far = torch.arange(n) - torch.stack([p.argmax(dim=-1) for p in probs])
    return folder, m.get("left", m)["mask"], big, far


@pytest.mark.parametrize("name", ["attention", "parallel", "shared"])
def test_single_keys_decide_the_logits(name):
    """The scores are many times larger, so the softmax of many rows is a choice of one or two keys: the oldest of the window,
    kept first tokens hundreds of places back, keys at page borders.  A kernel whose window was one off, or that lost a kept
    token, would miss whole rows."""
    n = 330
    tokens = random_tokens(n, vocab_of(name), 61)
    folder, mask, big, far = favourites(name, n, tokens)
    sure = big > 0.5
    size, keep = mask["size"], mask.get("keep_first", 0)
    assert float(sure.double().mean()) > 0.2
    # some rows are sure of the oldest key of their window; where first tokens are kept, some of the last one kept, far back
    rows = torch.arange(n).expand_as(far)
    assert bool((sure & (far == size - 1) & (rows >= size + keep)).any())
    if keep:
        assert bool((sure & (rows - far == keep - 1) & (far > 200)).any())
    want = oracle_logits(folder, tokens)
    for dtype in DTYPES:
        # in 16 bits a row that hesitates between two keys is decided by rounding: the bound on single rows is wider
        bound = (lambda got, what: check(got, want, dtype, what)) if dtype == "float32" else \
            (lambda got, what: _mostly(got, want, what))
        ctx = helpers.engine(folder, dtype).context
        bound(run_in_portions(ctx, tokens, [n]), f"{name} peaked, whole")
        bound(run_in_portions(ctx, tokens, [250] + list(range(251, n + 1))), f"{name} peaked, decoded")
        bound(run_in_portions(ctx, tokens, [1, 2, 20, 62, 130, 190, 200, 292, n]), f"{name} peaked, portions")


def _mostly(got, want, what):
    errs = sorted(helpers.rel_err(got[i], want[i]) for i in range(got.shape[0]))
    assert errs[int(0.9 * len(errs))] <= 0.15 and sum(errs) / len(errs) <= 5e-2, f"{what}: {errs[-30::5]}, mean {sum(errs) / len(errs):.3e}"


def test_the_edges_of_windows_show_in_the_logits():
    """The plain implementation with a window one longer or shorter, or one kept token more or fewer, gives other logits by many
    times the bounds the engine is held to above, in rows beyond the window."""
    n = 330
    for name, change in [("attention", ("size", 1)), ("attention", ("size", -1)), ("attention", ("keep_first", 1)), ("attention", ("keep_first", -1)),
                         ("parallel", ("size", 1)), ("parallel", ("size", -1)), ("shared", ("size", -1)), ("shared", ("keep_first", -1))]:
        tokens = random_tokens(n, vocab_of(name), 61)
        folder = folder_of(name, seed=5, peaked=14.0)
        right = oracle_logits(folder, tokens)
        cfg, w = bh.oracle(folder)
        cfg = copy.deepcopy(cfg)
        m = cfg["layers"][0]["mixer"]
        m.get("left", m)["mask"][change[0]] += change[1]
        wrong = pb.forward(cfg, w, tokens).float()
        moved = sorted(helpers.rel_err(wrong[t], right[t]) for t in range(n))
        assert moved[-1] > 0.1 and moved[int(0.95 * n)] > 1e-2, (name, change, moved[-3:], moved[int(0.95 * n)])


@pytest.mark.parametrize("what", ["lambda", "diff", "second map", "head gate", "stretch", "owner", "own mask", "left scale", "right scale", "decay",
                                  "one norm", "input gate", "forget gate", "cap", "denominator", "table", "shared", "embedding norm", "logit scale",
                                  "norm's one", "key bias"])
def test_what_the_mechanisms_do_shows_in_the_logits(what):
    """A mistake planted in the plain implementation moves the logits by many times the bounds that the engine is held to."""
    name = {"owner": "shared", "own mask": "shared", "left scale": "parallel", "right scale": "parallel", "decay": "parallel", "one norm": "parallel",
            "input gate": "mlstm", "forget gate": "mlstm", "cap": "mlstm", "denominator": "mlstm", "table": "moe",
            "shared": "moe"}.get(what, "attention")
    folder = folder_of(name)
    tokens = random_tokens(120, vocab_of(name), 65)
    right = oracle_logits(folder, tokens)
    cfg, w = bh.oracle(folder)
    cfg, w, patched = copy.deepcopy(cfg), dict(w), {}
    m = cfg["layers"][0]["mixer"]
    zero = lambda n: w.update({n: torch.zeros_like(w[n])})
    if what == "lambda":
        zero("l0.mix.lq1")
    elif what == "diff":
        m["diff"] += 0.1
    elif what == "second map":
        w["l0.mix.k"] = w["l0.mix.k"].view(2, 2, 20, 64)[:, [1, 0]].reshape(80, 64)
    elif what == "head gate":
        w["l0.mix.o"] = w["l0.mix.o"] * 0.5
        zero("l0.mix.g")
    elif what == "stretch":
        m["rot"].pop("scaling")
    elif what == "owner":
        cfg["layers"][1]["mixer"].pop("kv_from")
        w.update({f"l1.mix.{n}": w[f"l0.mix.{n}"] for n in ("k", "k.b", "v", "v.b")})
    elif what == "own mask":
        cfg["layers"][2]["mixer"]["mask"] = m["mask"]
    elif what in ("left scale", "right scale"):
        m[what.replace(" ", "_")] = 1.0
    elif what == "decay":
        m["right"]["decay"][2] = 0.99
    elif what == "one norm":          # a root mean square per head instead of one for all
        original = pb.unit_rms
        patched["unit_rms"] = lambda v, eps: original(v.reshape(len(v), 4, 12), eps).reshape(len(v), 48) if v.shape[-1] == 48 else original(v, eps)
    elif what == "input gate":
        zero("l0.mix.i.b")
    elif what == "forget gate":
        zero("l0.mix.f.b")
    elif what == "cap":
        m["gate_cap"] = 5.0
    elif what == "denominator":         # no floor under |n·q|
        def walk(q, k, v, i, f):
            T, H, d = q.shape
            S, n = q.new_zeros(H, d, v.shape[2]), q.new_zeros(H, d)
            top, out = q.new_zeros(H), []
            for t in range(T):
                new = torch.maximum(f[t] + top, i[t])
                keep, take, top = torch.exp(f[t] + top - new), torch.exp(i[t] - new), new
                S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
                n = keep[:, None] * n + take[:, None] * k[t]
                size = (n * q[t]).sum(-1).abs() + 1e-6
                out.append((S * q[t][:, :, None]).sum(1) / size[:, None])
            return torch.stack(out)
        patched["memory_walk"] = walk
    elif what == "table":
        w["l0.mlp.table"] = w["l0.mlp.table"].roll(1, 0)
    elif what == "shared":
        zero("l0.mlp.shared.down")
    elif what == "embedding norm":
        zero("embed.norm")
    elif what == "logit scale":
        cfg["logit_scale"] = 1.9
    elif what == "norm's one":
        w["l0.norm1"] = w["l0.norm1"] - 1.0
    elif what == "key bias":
        zero("l0.mix.k.b")
    before = {k: getattr(pb, k) for k in patched}
    try:
        for k, v in patched.items():
            setattr(pb, k, v)
        wrong = pb.forward(cfg, w, tokens).float()
    finally:
        for k, v in before.items():
            setattr(pb, k, v)
    moved = max(helpers.rel_err(wrong[t], right[t]) for t in range(len(tokens)))
    # behind the denominator the heads are normed to a root mean square of one: its size shows through eps alone
    assert moved > (2e-4 if what == "denominator" else 1e-2), (what, moved)
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
    for i, p in enumerate(prompts):
        mine = torch.cat(got[i])
        check(mine, oracle_logits(folder, p)[:mine.shape[0]], dtype, f"{name} request {i} in a batch")
        if dtype == "float32":
            alone = run_in_portions(ctx, p[:mine.shape[0]], [lens[i]] + list(range(lens[i] + 1, mine.shape[0] + 1)))
            check(mine, alone, dtype, f"{name} request {i}: batch against alone")
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
    for i, p in enumerate(prompts):
        check(torch.cat(got[i]), oracle_logits(folder, p), dtype, f"request {i} of mixed steps")


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


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_step_of_a_shape_that_comes_again_is_replayed_with_its_own_state(dtype):
    """The same shape of step several times in a row (captured at its second coming): every sequence has its own memories and
    its own experts, also when the graph is replayed."""
    folder = folder_of("mixed")
    ctx = helpers.engine(folder, dtype).context
    for i in range(4):
        tokens = random_tokens(144, vocab_of("mixed"), 95 + i)
        check(run_in_portions(ctx, tokens, [72, 144]), oracle_logits(folder, tokens), dtype, f"replayed step {i}")


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
    out = llm.generate(prompts, n_predict=16, stop_token_ids=[])
    total = 0
    for p, got in zip(prompts, out):
        want, sure = confident_greedy(folder, p, 16)
        assert len(got) == 16 and got[:sure] == want[:sure], (got, want, sure)
        total += sure
    assert total >= 32, total
    llm.context.cache.check()
    assert llm.context.cache.slots.n_held == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_through_the_captured_step(dtype):
    """150 generated tokens through the decode runner's graph; page borders and the windows' edges pass over them; each step's
    logits against the plain implementation run on the ids the engine chose."""
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
        check(got, refs[i][len(prompts[i]) - 1:len(prompts[i]) - 1 + 150], dtype, f"generated tokens of request {i}")


# ------------------------------------------------------------------ the kernels on their own

@pytest.mark.parametrize("n, d", [(37, 96), (1, 100), (300, 128), (256, 1536), (9, 2048), (300, 2052), (300, 41), (3, 12), (70, 896), (5, 13000)])
def test_two_norms_of_a_stream_that_takes_slices_and_expert_rows(n, d):
    g = torch.Generator().manual_seed(n + d)
    rnd = lambda *s: torch.randn(*s, generator=g).cuda()
    x, g1, g2, y, rows = rnd(n, d), rnd(d), rnd(d), rnd(3, n, d), rnd(50, d)
    row_of = torch.randint(0, 50, (n, 3), generator=g).int().cuda()
    weights = torch.rand(n, 3, generator=g).cuda()
    summed = (weights.double()[:, :, None] * rows[row_of.long()].double()).sum(1)
    for out_dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 5e-3)):
        for branch, experts in ((None, False), (y, False), (y[0].contiguous(), True), (None, True), (y, True)):
            for second in (True, False):
                stream = x.clone()
                o1 = torch.empty(n, d, dtype=out_dtype, device="cuda")
                o2 = torch.empty_like(o1) if second else None
                kernels.rms_pair(stream, g1, g2 if second else None, 1e-5, o1, o2, y=branch, expert_rows=(rows, row_of, weights) if experts else None)
                want = x.double()
                if branch is not None:
                    want = want + (branch.double().sum(0) if branch.dim() == 3 else branch.double())
                if experts:
                    want = want + summed
                assert helpers.rel_err(stream, want) <= 1e-6 and (branch is not None or experts or torch.equal(stream, x))
                unit = pb.unit_rms(want, 1e-5)
                assert helpers.rel_err(o1, unit * g1.double()) <= tol
                assert o2 is None or helpers.rel_err(o2, unit * g2.double()) <= tol


@pytest.mark.parametrize("table_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d", [20, 320, 2052])
def test_embedding_and_its_norm(d, table_dtype):
    g = torch.Generator().manual_seed(d)
    table = (torch.randn(90, d, generator=g) * 0.02).to(table_dtype).cuda()
    gain = torch.randn(d, generator=g).cuda()
    for n in (33, 300):
        ids = torch.randint(0, 90, (n,), generator=g).int().cuda()
        out = torch.empty(n, d, device="cuda")
        kernels.embed_rms(table, ids, gain, 1e-4, out, scale=3.0)
        assert helpers.rel_err(out, pb.unit_rms(table[ids.long()].double() * 3.0, 1e-4) * gain.double()) <= 2e-6


@pytest.mark.parametrize("n, H, vdim, D", [(9, 3, 40, 48), (130, 5, 64, 64), (33, 2, 128, 128), (7, 4, 200, 256), (5, 1, 30, 272), (3, 2, 500, 512), (4, 3, 7, 16)])
def test_the_difference_of_two_maps(n, H, vdim, D):
    g = torch.Generator().manual_seed(n + D)
    gate = torch.randn(n, 3 + H, generator=g).cuda()
    for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 5e-3)):
        o = torch.randn(n, H, 2, D, generator=g).to(dtype).cuda()
        out = torch.empty(n, H * vdim, dtype=dtype, device="cuda")
        a, b = o[:, :, 0, :vdim].double(), o[:, :, 1, :vdim].double()
        want = pb.diff_combine(a, b, 0.7, 0.4, 1e-5)
        kernels.diff_combine(o.view(n, -1), gate, 3, 0.7, 1e-5, 0.6, H, vdim, out)
        assert helpers.rel_err(out, (want * torch.sigmoid(gate[:, 3:].double())[:, :, None]).reshape(n, -1)) <= tol
        kernels.diff_combine(o.view(n, -1), None, 0, 0.7, 1e-5, 0.6, H, vdim, out)
        assert helpers.rel_err(out, want.reshape(n, -1)) <= tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, vdim, dims", [(20, 28, 12), (16, 40, 16), (32, 64, 0), (6, 30, 2)])
def test_two_keys_in_a_row_and_queries_at_their_places(dim, vdim, dims, dtype):
    from test_kernels_gpu import make_paged
    g = torch.Generator().manual_seed(dim)
    H, KV, n, start = 4, 2, 70, 30
    D = (max(2 * dim, vdim) + 15) // 16 * 16
    nq, nk = H * 2 * dim, KV * 2 * dim
    proj = torch.randn(n, 3 + nq + nk + KV * vdim, generator=g)
    qb, kb, vb = torch.randn(nq, generator=g), torch.randn(nk, generator=g), torch.randn(KV * vdim, generator=g)
    kv = make_paged([torch.zeros(start + n, KV, D)], [torch.zeros(start + n, KV, D)], dtype)
    positions = torch.arange(start, start + n, dtype=torch.int32, device="cuda")
    rot = bh.rot(dims, 1000.0, bh.SLOW)
    table = kernels.rope_table(pb.frequencies(rot).float().cuda(), start + n) if dims else None
    q = torch.full((n, 2 * H * D), 9.0, dtype=dtype, device="cuda")
    kernels.qk_norm_rope_cache(proj.cuda(), 3, 3 + nq, 3 + nq + nk, None, None, -1.0, positions, torch.zeros(n, dtype=torch.int32, device="cuda"),
                               table, dims, 2 * H, KV, dim, vdim, 1.5, q, kv, q_bias=qb.cuda(), k_bias=kb.cuda(), v_bias=vb.cuda(), maps=2)
    tol = 5e-6 if dtype == torch.float32 else 5e-3
    p = proj.double()
    turn = lambda x: pb.rotate(x, rot, positions.cpu())
    wq = turn((p[:, 3:3 + nq] + qb).view(n, 2 * H, dim)).view(n, H, 2, dim)
    want = torch.zeros(n, H, 2, D, dtype=torch.float64)
    want[:, :, 0, :dim], want[:, :, 1, dim:2 * dim] = wq[:, :, 0], wq[:, :, 1]
    assert helpers.rel_err(q.view(n, H, 2, D), want) <= tol and bool(((q.view(n, H, 2, D).cpu() == 0) == (want == 0)).all())
    keys = torch.zeros(n, KV, D, dtype=torch.float64)
    keys[:, :, :2 * dim] = turn((p[:, 3 + nq:3 + nq + nk] + kb).view(n, 2 * KV, dim)).view(n, KV, 2 * dim)
    vals = torch.zeros(n, KV, D, dtype=torch.float64)
    vals[:, :, :vdim] = (p[:, 3 + nq + nk:] + vb).view(n, KV, vdim) * 1.5
    for pool, rows in ((kv.k_pool, keys), (kv.v_pool, vals)):
        flat = pool.view(-1)[kv.entry_offset:].view(-1, KV, kv.page_size, D)
        got = torch.stack([flat[int(kv.page_table[0, (start + t) // kv.page_size]), :, (start + t) % kv.page_size] for t in range(n)])
        assert helpers.rel_err(got, rows) <= tol and bool((got[:, :, rows[0, 0].nonzero().numel():] == 0).all())


def portions_of(total, cuts):
    cuts = [c for c in cuts if c < total]
    return [slice(a, b) for a, b in zip([0] + cuts, cuts + [total])]


@pytest.mark.parametrize("H, dim, vdim, lens", [(3, 24, 12, [70, 1, 33]), (1, 5, 7, [20, 3]), (2, 64, 96, [130, 17]), (2, 200, 40, [40]), (4, 128, 64, [5, 1, 2])])
def test_constant_decay_walk(H, dim, vdim, lens):
    g = torch.Generator().manual_seed(H + dim)
    decay = [0.9, 0.3, 0.995, 0.6][:H]
    width = 2 * H * dim + 2 * H * vdim
    seqs = [torch.randn(n, 2 + width, generator=g) for n in lens]
    gain = torch.randn(H * vdim, generator=g)
    wants = []
    for s in seqs:
        z = s[:, 2:].double()
        q, k, v, gate = z.split([H * dim, H * dim, H * vdim, H * vdim], dim=1)
        o = pb.decay_walk(pb.silu(q).view(-1, H, dim), pb.silu(k).view(-1, H, dim), pb.silu(v).view(-1, H, vdim), decay).reshape(len(s), -1)
        wants.append(pb.unit_rms(o, 1e-5) * gain.double() * torch.sigmoid(gate) * 1.7)
    slots = [3, 0, 5][:len(lens)]
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 6e-3)):
        for cuts in ([], [1, 2, 19]):
            state = torch.zeros(6, H * dim * vdim + 3, device="cuda")[:, :H * dim * vdim]
            got = [[] for _ in lens]
            for part in portions_of(max(lens), cuts):
                live = [i for i, n in enumerate(lens) if n > part.start]
                rows = [seqs[i][part] for i in live]
                step = step_of([len(r) for r in rows], [slots[i] for i in live])
                out = torch.empty(sum(len(r) for r in rows), H * vdim, dtype=dtype, device="cuda")
                kernels.decay_attention(torch.cat(rows).cuda(), 2, 2 + 2 * H * dim + H * vdim,
                                        torch.tensor(decay, device="cuda"), gain.cuda(), 1e-5, 1.7, state, step, H, dim, vdim, out)
                for i, o in zip(live, out.float().cpu().split([len(r) for r in rows])):
                    got[i].append(o)
            for i in range(len(lens)):
                assert helpers.rel_err(torch.cat(got[i]), wants[i]) <= tol, (dtype, cuts, i)


@pytest.mark.parametrize("H, dim, vdim, lens, cap", [(3, 20, 28, [70, 1, 33], 12.0), (1, 5, 7, [20, 3], 2.0), (2, 64, 130, [130, 17], 14.0), (1, 200, 33, [40], 9.0),
                                                     (2, 4, 6, [2400, 2049, 7], 16.0), (4, 128, 64, [5, 1, 2], 6.0), (1, 8, 300, [30], 5.0)])
def test_matrix_memory_walk(H, dim, vdim, lens, cap):
    """Runs beyond a round of the scan (2,048 tokens), portions, unequal sequences, slots out of order; forget gates from a few
    tokens' memory to thousands'."""
    g = torch.Generator().manual_seed(H + dim)
    width = 2 * H * (dim + vdim + 1)
    seqs = [torch.randn(n, 2 + width, generator=g) for n in lens]
    gain, ib = torch.randn(H * vdim, generator=g), torch.randn(H, generator=g)
    fb = torch.linspace(0.0, 9.0, H) if H > 1 else torch.tensor([4.0])
    wants = []
    for s in seqs:
        q, k, v, gate, zi, zf = s[:, 2:].double().split([H * dim, H * dim, H * vdim, H * vdim, H, H], dim=1)
        i = cap * torch.tanh((zi + ib.double()) / cap)
        f = torch.nn.functional.logsigmoid(cap * torch.tanh((zf + fb.double()) / cap))
        o = pb.memory_walk(q.reshape(-1, H, dim) * dim ** -0.5, k.reshape(-1, H, dim), v.reshape(-1, H, vdim), i, f)
        wants.append(pb.unit_rms(o, 1e-5).reshape(len(s), -1) * gain.double() * torch.sigmoid(gate))
    slots = [3, 0, 5][:len(lens)]
    n_S = H * dim * (vdim + 1)
    for dtype, tol in ((torch.float32, 2e-4), (torch.bfloat16, 8e-3)):
        for cuts in ([], [1, 2, 6, 19]):
            state = torch.zeros(6, n_S + H + 3, device="cuda")[:, :n_S + H]
            got = [[] for _ in lens]
            for part in portions_of(max(lens), cuts):
                live = [i for i, n in enumerate(lens) if n > part.start]
                rows = [seqs[i][part] for i in live]
                step = step_of([len(r) for r in rows], [slots[i] for i in live])
                out = torch.empty(sum(len(r) for r in rows), H * vdim, dtype=dtype, device="cuda")
                c = 2
                cols = []
                for size in (H * dim, H * dim, H * vdim, H * vdim, H, H):
                    cols.append(c)
                    c += size
                kernels.matrix_memory(torch.cat(rows).cuda(), *cols, ib.cuda(), fb.cuda(), cap, gain.cuda(), 1e-5, state, step, H, dim, vdim, out)
                for i, o in zip(live, out.float().cpu().split([len(r) for r in rows])):
                    got[i].append(o)
            for i in range(len(lens)):
                assert helpers.rel_err(torch.cat(got[i]), wants[i]) <= tol, (dtype, cuts, i, helpers.rel_err(torch.cat(got[i]), wants[i]))


@pytest.mark.parametrize("n, E, top, tile", [(1, 4, 1, 64), (50, 6, 2, 64), (300, 33, 3, 128), (700, 12, 1, 128), (17, 5, 5, 64)])
def test_plan_of_experts_by_token_id(n, E, top, tile):
    """The same plan as that of the ids looked up first, and the weights."""
    g = torch.Generator().manual_seed(n)
    table = torch.rand(90, E, generator=g).argsort(dim=1)[:, :top].to(torch.int32).contiguous().cuda()
    tokens = torch.randint(0, 90, (n,), generator=g).int().cuda()
    rows = kernels.moe_plan_rows(n * top, E, tile)
    make = lambda: (torch.empty(n, top, dtype=torch.int32, device="cuda"), torch.empty(rows, dtype=torch.int32, device="cuda"),
                    torch.empty(rows // tile, dtype=torch.int32, device="cuda"))
    a, b = make(), make()
    weights = torch.empty(n, top, device="cuda")
    kernels.moe_plan_table(tokens, table, 1.0 / top, weights, E, tile, *a)
    kernels.moe_plan(table[tokens.long()].contiguous(), E, tile, *b)
    assert all(torch.equal(x, y) for x, y in zip(a, b)) and bool((weights == 1.0 / top).all())
    assert torch.equal(a[1][a[0].long()].cpu(), torch.arange(n, dtype=torch.int32)[:, None].expand(n, top))
