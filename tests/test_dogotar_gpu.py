"""Dogotar through the engine against the plain implementation (tests/plain_dogotar.py): every mechanism alone, every cutting of
the work, reused pages and slots, keys far back, at page borders and at the edges of windows and chunks, the first tokens, states
that remember for long, long decoding, generation through the scheduler.  Models and weights are made here
(tests/dogotar_models.py)."""

import types

import numpy as np
import pytest
import torch

import dogotar_models as dm
import helpers
import plain_dogotar as plain

pytestmark = pytest.mark.gpu

LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}
TRACES = {"whole": helpers.trace_whole, "tail_decode": helpers.trace_tail_decode, "portions": helpers.trace_portions,
          "mixed": helpers.trace_mixed}
LENGTHS = [1, 2, 19, 53, 97, 150]


def row_error(got, want):
    """Root mean square of the difference (its mean taken off) over that of the wanted row."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    d = got - want
    d = d - d.mean()
    w = want - want.mean()
    return float(np.sqrt((d * d).mean()) / max(np.sqrt((w * w).mean()), 1e-30))


def sequences(vocab, lengths=LENGTHS, seed=100):
    return {f"r{i}": helpers.random_tokens(vocab, n, seed=seed + i) for i, n in enumerate(lengths)}


def stored(weights, dtype):
    """The weights as a checkpoint of ``dtype`` holds them, and their exact values in float64 for the oracle."""
    held = {k: v.to(torch.bfloat16 if dtype == "bfloat16" else torch.float32) for k, v in weights.items()}
    return held, {k: v.double() for k, v in held.items()}


def replay(folder, dtype, steps, *, max_tokens=None, max_live=64, page_size=16, graphs=True):
    """Logits by (request, position).  Pages nobody has written or that went back to the pool hold NaN."""
    from prefixserve_b200.engine.replay import Replayer
    rp = Replayer(folder, dtype, max_tokens or helpers.peak_tokens(steps), max_live=max_live, page_size=page_size,
                  use_graphs=graphs)
    rp.cache.poison_freed = True
    for kv in rp.cache.kv:
        if kv is not None:
            kv.fill_(float("nan"))
    outputs = {}
    for st in steps:
        out = rp.run_step(st)
        if out is not None:
            outputs[st["step"]] = out
    rp.cache.check()
    return helpers.collect(steps, outputs)


def errors(rows, truth):
    out = []
    for (rid, pos), got in rows.items():
        assert np.isfinite(got).all(), f"{rid} position {pos}: not finite"
        out.append(row_error(got, truth[rid][pos].numpy()))
    return np.asarray(out)


def assert_close(rows, truth, dtype):
    """float32: every row within the limit.  bfloat16: the read-out of a memory is a quotient that is normed, so where a head of a
    few numbers nearly cancels, the rounding of its inputs is blown up whoever computes it; 97 rows of 100 are held to the limit,
    the rest to four times that."""
    e = errors(rows, truth)
    if dtype == "float32":
        assert e.max() < LIMIT[dtype], e.max()
    else:
        assert np.quantile(e, 0.97) < LIMIT[dtype] and e.max() < 4 * LIMIT[dtype], (np.quantile(e, 0.97), e.max())


def exact_weights(which, dtype):
    return stored(dm.tensors(dm.CONFIGS[which], seed=sorted(dm.CONFIGS).index(which)), dtype)


@pytest.fixture(scope="module")
def made(tmp_path_factory):
    """(configuration name, dtype) -> (folder, float64 logits of every test sequence)."""
    out = {}
    for which, cfg in dm.CONFIGS.items():
        for dtype in ("float32", "bfloat16"):
            held, exact = exact_weights(which, dtype)
            folder = dm.write_folder(tmp_path_factory.mktemp(f"{which}-{dtype}"), cfg, held)
            truth = {rid: plain.forward(cfg, exact, toks) for rid, toks in sequences(cfg["vocab"]).items()}
            out[which, dtype] = (folder, truth)
    return out


@pytest.mark.parametrize("trace", sorted(TRACES))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(dm.CONFIGS))
def test_every_cutting_matches_the_plain_model(made, which, dtype, trace):
    """Whole prompts, a decoded tail, portions down to two tokens, and up to four requests at once over a pool that
    only holds what is live (pages and slots are used again)."""
    folder, truth = made[which, dtype]
    seqs = sequences(dm.CONFIGS[which]["vocab"])
    steps = TRACES[trace](seqs)
    rows = replay(folder, dtype, steps, max_live=4 if trace == "mixed" else 64)
    assert len(rows) == sum(len(t) for t in seqs.values())
    assert_close(rows, truth, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page_size", [1, 4, 64])
@pytest.mark.parametrize("which", ["mixed", "wide"])
def test_token_by_token_through_small_and_large_pages(made, which, dtype, page_size):
    """Every token decoded alone from the first on: prefill against token-by-token decoding, over many page borders."""
    folder, truth = made[which, dtype]
    seqs = {rid: toks for rid, toks in sequences(dm.CONFIGS[which]["vocab"]).items() if len(toks) in (2, 150)}
    steps = helpers.trace_tail_decode(seqs, tail=10 ** 6)
    rows = replay(folder, dtype, steps, page_size=page_size, max_tokens=helpers.peak_tokens(steps, page=max(page_size, 64)))
    assert_close(rows, truth, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["mixed", "attention_only"])
def test_two_slots_and_an_exact_pool_serve_six_requests(made, which, dtype):
    folder, truth = made[which, dtype]
    seqs = sequences(dm.CONFIGS[which]["vocab"])
    steps = helpers.trace_mixed(seqs, max_live=2, seed=7)
    rows = replay(folder, dtype, steps, max_live=2, page_size=4, max_tokens=helpers.peak_tokens(steps, page=4))
    assert_close(rows, truth, dtype)


def test_a_batch_gives_each_request_what_it_gets_alone(made):
    folder, _ = made["mixed", "float32"]
    seqs = sequences(131)
    together = replay(folder, "float32", helpers.trace_mixed(seqs, max_live=4, seed=3), max_live=4)
    alone = replay(folder, "float32", helpers.trace_whole(seqs))
    for key, row in alone.items():
        assert row_error(together[key], row) < 1e-5


def test_captured_steps_give_what_uncaptured_ones_give(made):
    folder, _ = made["mixed", "bfloat16"]
    seqs = sequences(131)
    steps = helpers.trace_tail_decode(seqs, tail=20)
    a, b = replay(folder, "bfloat16", steps, graphs=True), replay(folder, "bfloat16", steps, graphs=False)
    assert all(np.array_equal(a[k], b[k]) for k in a)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_of_repeated_lengths_are_captured_and_stay_right(tmp_path, dtype):
    """A prompt in portions of one length: from the second on they are replayed from a capture; chunks of the matrix memory run
    side by side in them, and the values of the first mixing layer reach the later ones inside the capture."""
    cfg = dm.CONFIGS["wide"]
    held, exact = exact_weights("wide", dtype)
    folder = dm.write_folder(tmp_path / "m", cfg, held)
    toks = helpers.random_tokens(300, 700, seed=8)
    truth = {"a": plain.forward(cfg, exact, toks)}
    steps, at = [], 0
    for i, n in enumerate((160, 160, 160, 160, 60)):
        steps.append({"step": i, "entries": [{"id": "a", "tokens": toks[at: at + n], "want": [0, n - 1]}], "end": ["a"] if i == 4 else []})
        at += n
    assert_close(replay(folder, dtype, steps), truth, dtype)


def test_pages_behind_the_window_and_before_the_chunk_go_back(tmp_path):
    from prefixserve_b200.engine.replay import Replayer
    cfg = dm.config([dm.attention(window=9), dm.parallel(dm.left(chunk=12))])
    held, _ = stored(dm.tensors(cfg, seed=1), "float32")
    rp = Replayer(dm.write_folder(tmp_path / "m", cfg, held), "float32", 1024, page_size=4)
    toks = helpers.random_tokens(61, 200, seed=3)
    rp.run_step({"step": 0, "entries": [{"id": "a", "tokens": toks[:150], "want": []}], "end": []})
    for i in range(150, 200):
        rp.run_step({"step": i, "entries": [{"id": "a", "tokens": toks[i: i + 1], "want": [0]}], "end": []})
        for group in (0, 1):
            assert len([p for p in rp.cache.page_ids(rp.slot_of["a"], group) if p >= 0]) <= 12 // 4 + 2
    rp.cache.check()


# ---- keys and states that must not be lost ----------------------------------------------------------------------

MARK, ASK = 62, 63


def echo_model(dtype, kind, reach, dim=16):
    """One layer whose attention answers the token ASK with the value of the token MARK wherever that lies and is visible: the
    key matrix is the first query head's behind a fixed permutation of the width, and ASK's embedding is MARK's under the same
    permutation (a layer norm does not care), so ASK's query is MARK's key and its score stands out among hundreds of random
    ones.  Whoever loses that one key, or sees it where the mask hides it, gives a visibly different row.  kind: "window" (an
    attention layer without a rotation) or "chunk" (a parallel layer whose right branch is silent)."""
    sizes = dict(heads=2, kv_heads=1, dim=dim, vdim=8 if dim == 16 else 32, scale=12.8 / dim, cap=40.0)
    lay = dm.attention(window=reach, rot=None, v_mix=False, **sizes) if kind == "window" else dm.parallel(dm.left(chunk=reach, **sizes), dm.right())
    cfg = dm.config([lay], vocab=64, width=32)
    w = dm.tensors(cfg, seed=11)
    p = "l0.mix." if kind == "window" else "l0.mix.left."
    turn = torch.eye(32)[torch.roll(torch.arange(32), 1)]
    w[p + "k"] = w[p + "q"][:dim] @ turn
    w["embed"][ASK] = turn @ w["embed"][MARK]
    w["l0.norm1"], w["l0.norm1.b"] = torch.ones(32), torch.zeros(32)
    w[p + "o"] *= 2.0
    for n in ("q", "k"):
        w[p + n + ".b"] *= 0.0
        w[p + n + ".norm"] = torch.ones_like(w[p + n + ".norm"])
    if kind == "chunk":
        w["l0.mix.right.o"] *= 0.0
    return cfg, *stored(w, dtype)


CUTTINGS = (
    (16, lambda s, n, m: helpers.trace_whole(s)),
    (64, lambda s, n, m: helpers.trace_tail_decode(s, tail=140)),
    (16, lambda s, n, m: helpers.trace_tail_decode(s, tail=n - m - 1)),
    (64, lambda s, n, m: helpers.trace_portions(s, sizes=(3, 2, 59, 2, 40, 7, 2, 31, 64))),
    (16, lambda s, n, m: helpers.trace_portions(s, sizes=(64, 1, 35, 100, 2))),
)


def check_echo(tmp_path, dtype, kind, reach, dim, marked, sees, misses, n=330):
    cfg, held, exact = echo_model(dtype, kind, reach, dim)
    folder = dm.write_folder(tmp_path / "m", cfg, held)
    toks = helpers.random_tokens(62, n, seed=9)
    toks[marked] = MARK
    for a in [*sees, *misses]:
        if a != marked:
            toks[a] = ASK
    truth = {"a": plain.forward(cfg, exact, toks)}
    quiet = list(toks)
    quiet[marked] = 1
    hidden = plain.forward(cfg, exact, quiet)
    diff = lambda rows: [row_error(truth["a"][i].numpy(), hidden[i].numpy()) for i in rows]
    assert min(diff(sees)) > 0.1 and (not misses or max(diff(misses)) < 1e-9), (diff(sees), diff(misses))
    for page_size, cut in CUTTINGS:
        steps = cut({"a": toks}, n, marked)
        e = errors(replay(folder, dtype, steps, page_size=page_size, max_tokens=helpers.peak_tokens(steps, page=64)), truth)
        assert e.max() < LIMIT[dtype], e.max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("marked", [0, 3, 63, 64])
@pytest.mark.parametrize("kind,dim", [("window", 16), ("window", 64), ("chunk", 64)])
def test_one_key_far_back_or_at_a_page_border_is_found(tmp_path, kind, dim, dtype, marked):
    """No mask: the marked key is a sequence's first, an early one, a page's last or a page's first (pages of 16 and of 64);
    it is asked for right behind it and hundreds of tokens later, in prompts, in portions and in single tokens."""
    check_echo(tmp_path, dtype, kind, None, dim, marked, [marked + 1, 100, 200, 329], [])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [16, 64])
@pytest.mark.parametrize("window,marked", [(40, 100), (40, 0), (64, 63), (64, 64), (33, 70), (1, 50), (17, 15), (130, 128)])
def test_a_key_just_inside_and_just_outside_the_window(tmp_path, dim, dtype, window, marked):
    """The marked key is asked for by the last query that sees it and by the first that does not, in prompts, in portions (whose
    tiles straddle the edge) and in single tokens.  A window of one token sees itself only."""
    check_echo(tmp_path, dtype, "window", window, dim, marked, [marked + window - 1], [marked + window, 329])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [16, 64])
@pytest.mark.parametrize("chunk,marked", [(40, 40), (40, 78), (64, 64), (64, 126), (33, 67), (130, 3), (17, 51), (100, 198)])
def test_a_key_is_seen_to_the_end_of_its_chunk_and_never_after(tmp_path, dim, dtype, chunk, marked):
    """Chunks are counted from a sequence's start however it is cut: the last position of the marked key's chunk sees it, the
    first of the next, one token later, does not."""
    end = (marked // chunk + 1) * chunk
    check_echo(tmp_path, dtype, "chunk", chunk, dim, marked, [end - 1], [end, 329])


def memory_model(dtype, dim=40, vdim=10):
    """A parallel layer whose memory hardly forgets, whose attention is silent, and a token (63) that opens the input gate wide:
    what it wrote outweighs everything behind it, so it shows in every later row."""
    cfg = dm.config([dm.parallel(dm.left(), dm.right(heads=2, dim=dim, vdim=vdim, cap=9.0))], vocab=64, width=32)
    w = dm.tensors(cfg, seed=21)
    w["embed"][:, 0] = 0.0
    w["embed"][63, 0] = 4.0
    w["l0.norm1"][0] = 1.0
    w["l0.norm1.b"][0] = 0.0
    w["l0.mix.right.i"] *= 0.4
    w["l0.mix.right.i"][:, 0] = 3.0
    w["l0.mix.right.i.b"] -= 2.5
    w["l0.mix.right.f.b"] += 9.0
    w["l0.mix.right.f"] *= 0.3
    w["l0.mix.left.o"] *= 0.0
    return cfg, *stored(w, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim", [(40, 10), (64, 32), (24, 136)])
def test_what_a_token_wrote_into_the_memory_shows_hundreds_of_tokens_later(tmp_path, dim, vdim, dtype):
    """A lost state, a lost exponent or a state of somebody else shows for long; portions down to two tokens, some that fill
    several chunks, single tokens, slots used again."""
    cfg, held, exact = memory_model(dtype, dim, vdim)
    folder = dm.write_folder(tmp_path / "m", cfg, held)
    seqs = sequences(63, lengths=[3, 64, 300, 180], seed=40)
    for rid, at in (("r0", 0), ("r1", 1), ("r2", 2), ("r3", 70)):
        seqs[rid][at] = 63
    truth = {rid: plain.forward(cfg, exact, toks) for rid, toks in seqs.items()}
    quiet = list(seqs["r2"])
    quiet[2] = 1
    hidden = plain.forward(cfg, exact, quiet)
    shows = [row_error(hidden[i].numpy(), truth["r2"][i].numpy()) for i in (3, 10, 50, 150, 299)]
    assert min(shows) > 0.1, shows
    for steps in (helpers.trace_whole(seqs), helpers.trace_portions(seqs, sizes=(2, 2, 3, 1, 2, 50, 2)), helpers.trace_tail_decode(seqs, tail=150),
                  helpers.trace_portions(seqs, sizes=(140, 2, 133)), helpers.trace_mixed(seqs, max_live=2, seed=1)):
        e = errors(replay(folder, dtype, steps, max_live=4), truth)
        # (a read-out that nearly cancels is blown up by the norm behind it, and its rounding with it)
        assert e.max() < 3 * LIMIT[dtype], e.max()


@pytest.mark.parametrize("which", ["mixed", "wide"])
def test_long_decoding(made, which):
    """Hundreds of single tokens behind a short prompt, several requests side by side in captured steps."""
    cfg = dm.CONFIGS[which]
    for dtype in ("float32", "bfloat16"):
        folder, _ = made[which, dtype]
        _, exact = exact_weights(which, dtype)
        seqs = sequences(cfg["vocab"], lengths=[400, 260, 333], seed=60)
        truth = {rid: plain.forward(cfg, exact, toks) for rid, toks in seqs.items()}
        steps = helpers.trace_many_live(seqs, tail=250, portion_beside=False)
        assert_close(replay(folder, dtype, steps, max_live=3), truth, dtype)


# ---- mechanisms alone -------------------------------------------------------------------------------------------

def dev(x, dtype=torch.int32):
    return torch.tensor(x, dtype=dtype).cuda()


def step_context(lengths, starts, slots=None):
    """What the ops read of a step: portions of the given lengths starting at the given absolute positions."""
    slots = slots or list(range(len(lengths)))
    positions, item_of, offsets = [], [], [0]
    for i, (n, s) in enumerate(zip(lengths, starts)):
        positions += list(range(s, s + n))
        item_of += [i] * n
        offsets.append(offsets[-1] + n)
    return types.SimpleNamespace(positions=dev(positions), token_item=dev(item_of), item_start=dev(offsets), slots=dev(slots),
                                 num_items=len(lengths), num_tokens=len(positions), max_new_tokens=max(lengths),
                                 kv_len=dev([n + s for n, s in zip(lengths, starts)]),
                                 max_kv_len=max(n + s for n, s in zip(lengths, starts)), extras={})


def paged(lengths, page):
    """A page table in a scrambled order for items that hold so many tokens, and the number of pages."""
    need = [-(-n // page) for n in lengths]
    ids = torch.randperm(sum(need), generator=torch.Generator().manual_seed(4)).tolist()
    table = torch.full((len(lengths), max(need)), -1, dtype=torch.int32)
    for i, n in enumerate(need):
        table[i, :n] = torch.tensor([ids.pop() for _ in range(n)])
    return table, sum(need)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [5, 20, 1024, 1100, 2048, 5000, 9000])
def test_layer_norms_behind_a_sum_alone(dtype, width):
    """h += pending and one or two norms of it; rows picked out leave the stream as it is; a mean far from zero."""
    from prefixserve_b200 import ops
    g = torch.Generator().manual_seed(width)
    rnd = lambda *s: torch.randn(*s, generator=g)
    h, d = rnd(7, width) + 30.0 * torch.arange(7)[:, None], (3 * rnd(7, width)).to(dtype)
    norms = [(1 + 0.2 * rnd(width), rnd(width)) for _ in range(2)]
    on = [tuple(t.cuda() for t in n) for n in norms]
    tol = 1e-4 if dtype == torch.float32 else 4e-2   # (a mean of 180 leaves float32 five digits behind the point)
    for pending in (None, d):
        want_h = h.double() + (0 if pending is None else pending.double())
        want = [plain.layer_norm(want_h, a.double(), b.double(), 1e-3) for a, b in norms]
        for k in (1, 2):
            stream = h.clone().cuda()
            xs = ops.add_layer_norm(stream, None if pending is None else pending.cuda(), on[:k], 1e-3, dtype)
            assert len(xs) == k and torch.allclose(stream.cpu().double(), want_h, atol=1e-5)
            assert all(torch.allclose(x.cpu().double(), y, atol=tol) for x, y in zip(xs, want))
        stream = h.clone().cuda()
        picked = ops.add_layer_norm(stream, None if pending is None else pending.cuda(), on[:1], 1e-3, dtype, rows=dev([5, 0, 5]))[0]
        assert torch.equal(stream.cpu(), h) and torch.allclose(picked.cpu().double(), want[0][[5, 0, 5]], atol=tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim,vdim,hq,hkv,rot,interleaved,mixed", [
    (16, 10, 4, 2, 8, False, True), (40, 24, 6, 2, None, False, False), (64, 32, 4, 2, 32, False, True), (64, 64, 3, 1, 64, False, False),
    (128, 40, 2, 1, 32, False, True), (128, 64, 4, 4, 96, False, False), (32, 16, 5, 1, 16, False, True), (256, 8, 2, 1, 128, False, True),
    (64, 64, 4, 2, 20, True, True), (7, 5, 3, 1, 4, True, False)])
@pytest.mark.parametrize("long", [False, True])
def test_normed_heads_rotation_mixing_and_append_alone(dtype, dim, vdim, hq, hkv, rot, interleaved, mixed, long):
    """Biases, a norm with a gain per head, the rotation behind it, values mixed with another layer's, queries out, keys and
    values into the token's cache row; the projection is a run of columns of a wider product."""
    from prefixserve_b200 import ops
    g = torch.Generator().manual_seed(dim + vdim)
    rnd = lambda *s: torch.randn(*s, generator=g)
    lengths, starts, page = ([600, 1, 440] if long else [5, 1, 40]), [0, 17, 3], 8
    ctx, t = step_context(lengths, starts), sum(lengths)
    qk, width, v = (hq + hkv) * dim, (hq + hkv) * dim + hkv * vdim, hkv * vdim
    wide, first = (2 * rnd(t, width + 16)).to(dtype), rnd(t, v + 24).to(dtype)
    bias, gq, gk, fb, share = rnd(width), 1 + 0.3 * rnd(dim), 1 + 0.3 * rnd(dim), rnd(v), torch.tensor([0.3])
    table, pages = paged([n + s for n, s in zip(lengths, starts)], page)
    kv = torch.zeros(pages, 1, hkv, page, dim + vdim, dtype=dtype).cuda()
    cos = sin = None
    if rot:
        angles = torch.arange(700)[:, None] * (100.0 ** (-2.0 * torch.arange(rot // 2) / rot))[None]
        cos, sin = angles.cos().float().cuda(), angles.sin().float().cuda()
    q = ops.attention_prepare_heads(wide.cuda()[:, 8: 8 + width], kv, table.cuda(), ctx, num_heads=hq, num_kv_heads=hkv, dim=dim, vdim=vdim,
                                    page_size=page, gain_q=gq.cuda(), gain_k=gk.cuda(), eps=1e-3, cos=cos, sin=sin, rotary_dim=rot,
                                    interleaved=interleaved, bias=bias.cuda(), first=first.cuda()[:, 16: 16 + v] if mixed else None,
                                    first_bias=fb.cuda() if mixed else None, share=share.cuda() if mixed else None).cpu().double()
    full, pos = wide[:, 8: 8 + width].double() + bias.double(), ctx.positions.cpu().long()

    def turned(x):
        if not rot:
            return x
        c, s = (a.double().cpu()[pos][:, None] for a in (cos, sin))
        out = x.clone()
        a, b = (x[..., 0:rot:2], x[..., 1:rot:2]) if interleaved else (x[..., : rot // 2], x[..., rot // 2: rot])
        u, w = a * c - b * s, b * c + a * s
        if interleaved:
            out[..., 0:rot:2], out[..., 1:rot:2] = u, w
        else:
            out[..., : rot // 2], out[..., rot // 2: rot] = u, w
        return out
    want_q = turned(plain.rms_norm(full[:, : hq * dim].reshape(t, hq, dim), gq.double(), 1e-3))
    want_k = turned(plain.rms_norm(full[:, hq * dim: qk].reshape(t, hkv, dim), gk.double(), 1e-3))
    want_v = full[:, qk:]
    if mixed:
        want_v = plain.mix_values(want_v, first[:, 16: 16 + v].double() + fb.double(), 0.3)
    tol = 2e-5 if dtype == torch.float32 else 5e-2
    assert torch.allclose(q, want_q, atol=tol)
    held = kv.cpu().double()
    at = table[ctx.token_item.cpu().long(), pos // page].long()
    rows = held[at, 0, :, pos % page]
    assert torch.allclose(rows[..., :dim], want_k, atol=tol) and torch.allclose(rows[..., dim:].reshape(t, v), want_v, atol=tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim,vdim,hq,hkv", [(64, 32, 4, 2), (128, 128, 4, 1), (16, 24, 3, 3), (10, 6, 4, 2), (136, 40, 2, 1), (128, 64, 8, 1)])
@pytest.mark.parametrize("window,chunk", [(None, None), (37, None), (None, 48), (64, None), (None, 200)])
def test_capped_attention_with_gate_and_factor_alone(dtype, dim, vdim, hq, hkv, window, chunk):
    """Scores near and far beyond the cap, a window or a chunk, an output gate and a factor, the result into a run of columns;
    single tokens far into a sequence (the keys split among blocks), short and long portions behind cached keys."""
    from prefixserve_b200 import ops
    g = torch.Generator().manual_seed(dim)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol, page = (2e-5 if dtype == torch.float32 else 2e-2), 16
    for lengths, starts in (([3, 300, 1, 80], [60, 150, 1100, 0]), ([1, 1, 1], [1100, 0, 47])):
        ctx, t = step_context(lengths, starts), sum(lengths)
        held = [n + s for n, s in zip(lengths, starts)]
        table, pages = paged(held, page)
        q = rnd(t, hq, dim).to(dtype)
        k, v = [rnd(n, hkv, dim).to(dtype) for n in held], [rnd(n, hkv, vdim).to(dtype) for n in held]
        kv = torch.full((pages, 1, hkv, page, dim + vdim), float("nan"), dtype=dtype)
        for i, n in enumerate(held):
            for p in range(n):
                kv[table[i, p // page], 0, :, p % page] = torch.cat([k[i][p], v[i][p]], -1)
        gate, wide = rnd(t, hq * vdim + 8).to(dtype), torch.full((t, hq * vdim + 24), 7.0, dtype=dtype, device="cuda")
        out = ops.attention_over_rows(q.cuda(), kv.cuda(), table.cuda(), ctx, num_heads=hq, num_kv_heads=hkv, dim=dim, vdim=vdim, page_size=page,
                                      scale=0.5, window=window, chunk=chunk, softcap=3.0, gate=gate.cuda()[:, 4: 4 + hq * vdim], out_scale=-1.5,
                                      out=wide[:, 8: 8 + hq * vdim])
        assert out.data_ptr() == wide[:, 8:].data_ptr() and bool((wide[:, :8] == 7.0).all()) and bool((wide[:, 8 + hq * vdim:] == 7.0).all())
        first = 0
        for i, (n, s) in enumerate(zip(lengths, starts)):
            mask = (plain.in_window(held[i], window) & plain.in_chunk(held[i], chunk))
            qq = torch.zeros(held[i], hq, dim, dtype=torch.float64)
            qq[s:] = q[first: first + n].double()
            want = plain.capped_attention(qq, k[i].double().repeat_interleave(hq // hkv, 1), v[i].double().repeat_interleave(hq // hkv, 1), 0.5, 3.0, mask)[s:]
            want = want.reshape(n, -1) * torch.sigmoid(gate[first: first + n, 4: 4 + hq * vdim].double()) * -1.5
            assert torch.allclose(out[first: first + n].cpu().double(), want, atol=tol), (i, (out[first: first + n].cpu().double() - want).abs().max())
            first += n


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,vdim", [(1, 5, 7), (3, 16, 24), (2, 64, 40), (2, 128, 128), (1, 200, 33), (2, 24, 64), (1, 136, 200), (1, 256, 264),
                                            (1, 300, 16), (1, 600, 5)])
def test_matrix_memory_alone(dtype, heads, dim, vdim):
    """Portions of many lengths in one step (chunks side by side: full ones, a short last one, exactly two), states from before,
    gates from shut to wide open, slots in any order; and the same as short steps.  The bare read-out is checked through its
    norm: a gain and a gate per channel, the result into a run of columns."""
    from prefixserve_b200 import ops
    g = torch.Generator().manual_seed(dim + vdim)
    rnd = lambda *s: torch.randn(*s, generator=g)
    whole, slots, cap, eps = [300, 1, 64, 128, 129, 2], [3, 0, 5, 1, 7, 2], 7.0, 1e-2
    width, v = 2 * heads * (dim + vdim) + 2 * heads, heads * vdim
    proj = [rnd(n, width + 8) for n in whole]
    for p in proj:
        p[:, width - 2 * heads: width] *= 6.0
        p[:, width - heads: width] += 4.0
    proj = [p.to(dtype) for p in proj]
    bi, bf, gain = rnd(heads), rnd(heads), 1 + 0.3 * rnd(v)
    want = []
    for p in proj:
        x = p[:, :width].double()
        q, k, vv, gate, zi, zf = x.split([heads * dim, heads * dim, v, v, heads, heads], -1)
        i = plain.soft_cap(zi + bi.double(), cap)
        f = torch.nn.functional.logsigmoid(plain.soft_cap(zf + bf.double(), cap))
        o = plain.matrix_memory(q.reshape(-1, heads, dim) * dim ** -0.5, k.reshape(-1, heads, dim), vv.reshape(-1, heads, vdim), i, f)
        want.append(plain.rms_norm(o, None, eps).reshape(-1, v) * gain.double() * torch.sigmoid(gate))
    floats = ops.matrix_memory_state(heads, dim, vdim)
    for cut in (lambda n: [n], lambda n: [c for c in (n // 3, n - n // 3) if c], lambda n: [2, n // 2, n - n // 2 - 2] if n > 4 else [1] * n):
        state = torch.zeros(9, floats + 8, device="cuda")
        held = state[:, 4: 4 + floats]
        at, pieces, outs = [0] * len(whole), [cut(n) for n in whole], [[] for _ in whole]
        for turn in range(max(len(c) for c in pieces)):
            live = [i for i in range(len(whole)) if turn < len(pieces[i])]
            lengths = [pieces[i][turn] for i in live]
            ctx = step_context(lengths, [at[i] for i in live], [slots[i] for i in live])
            p = torch.cat([proj[i][at[i]: at[i] + n] for i, n in zip(live, lengths)])
            wide = torch.full((sum(lengths), v + 16), 7.0, dtype=dtype, device="cuda")
            o = ops.matrix_memory(p.cuda()[:, :width], bi.cuda(), bf.cuda(), gain.cuda(), held, ctx, heads=heads, dim=dim, vdim=vdim, cap=cap,
                                  eps=eps, out=wide[:, 8: 8 + v]).cpu()
            assert bool((wide[:, :8] == 7.0).all()) and bool((wide[:, 8 + v:] == 7.0).all())
            first = 0
            for i, n in zip(live, lengths):
                outs[i].append(o[first: first + n])
                first += n
                at[i] += n
        for i in range(len(whole)):
            got = torch.cat(outs[i]).double()
            e = (got - want[i]).abs().max() / want[i].abs().max()
            assert e < (5e-5 if dtype == torch.float32 else 2e-2), (i, float(e))
        assert float(state[:, :4].abs().max()) == 0 and float(state[:, -4:].abs().max()) == 0 and float(state[[4, 6, 8]].abs().max()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,k,n", [(1, 64, 40), (8, 256, 96), (3, 40, 33), (20, 128, 200), (64, 72, 48), (100, 64, 64), (700, 256, 4096), (130, 20, 10)])
@pytest.mark.parametrize("name", ["gelu_tanh", "silu", "relu2"])
def test_product_with_an_activation_into_a_run_of_columns(dtype, rows, k, n, name):
    from prefixserve_b200 import ops
    g = torch.Generator().manual_seed(rows)
    x, w = torch.randn(rows, k, generator=g).to(dtype), (2 * torch.randn(n, k, generator=g) / k ** 0.5).to(dtype)
    z = x.double() @ w.double().T
    want = {"gelu_tanh": plain.gelu_tanh(z), "silu": z * torch.sigmoid(z), "relu2": z.clamp(min=0) ** 2}[name]
    tol = dict(atol=1e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=3e-2, rtol=2e-2)
    assert torch.allclose(ops.unary_linear(x.cuda(), w.cuda(), name).cpu().double(), want, **tol)
    for at in (8, 3):
        wide = torch.full((rows, n + 24), 7.0, dtype=dtype, device="cuda")
        ops.unary_linear(x.cuda(), w.cuda(), name, out=wide[:, at: at + n])
        assert torch.allclose(wide[:, at: at + n].cpu().double(), want, **tol)
        assert bool((wide[:, :at] == 7.0).all()) and bool((wide[:, at + n:] == 7.0).all())


# ---- generation ---------------------------------------------------------------------------------------------------

def greedy(cfg, exact, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(plain.forward(cfg, exact, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("which", ["mixed", "attention_only"])
def test_greedy_generation_through_the_entry_point_and_scheduler(made, which):
    """Prompts longer than a portion, more requests than run at once, captured decode steps: the same tokens as the
    plain model's greedy continuation (float32: a tie would have to be exact to differ)."""
    from prefixserve_b200.engine.llm import LLM
    from prefixserve_b200.sampling import SamplingParams
    folder, _ = made[which, "float32"]
    cfg = dm.CONFIGS[which]
    _, exact = exact_weights(which, "float32")
    prompts = [helpers.random_tokens(cfg["vocab"], n, seed=70 + n) for n in (1, 5, 23, 40)]
    llm = LLM(folder, dtype="float32", max_seq_len=128, num_blocks=64, max_running_requests=3, chunked_prefill_size=16)
    got = llm.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    assert got == [greedy(cfg, exact, p, 12) for p in prompts]
    assert llm.engine.runner.graph_replays > 0
    llm.engine.cache.check()
    # a second call on the same engine starts from clean slots
    assert llm.generate(prompts[:2], SamplingParams(max_tokens=5, ignore_eos=True)) == [greedy(cfg, exact, p, 5) for p in prompts[:2]]


def test_command_line_generates_from_a_dogotar_folder(made):
    import json
    import subprocess
    import sys
    folder, _ = made["parallel_only", "bfloat16"]
    out = subprocess.run([sys.executable, "-m", "prefixserve_b200", "--model", str(folder), "--prompt-ids", "5,17,3", "--max-tokens", "6",
                          "--num-blocks", "32", "--max-seq-len", "64", "--max-running-requests", "2"],
                         capture_output=True, text=True, timeout=600, cwd=str(helpers.__file__).rsplit("/tests/", 1)[0])
    assert out.returncode == 0, out.stderr[-2000:]
    first = json.loads(out.stdout.splitlines()[0])
    assert first["prompt_ids"] == [5, 17, 3] and len(first["output_ids"]) == 6


def test_a_preset_of_the_design_generates(tmp_path):
    from prefixserve_b200.config.presets import preset
    from prefixserve_b200.engine.llm import LLM
    from prefixserve_b200.sampling import SamplingParams
    from prefixserve_b200.weights import write_random_model
    folder = write_random_model(tmp_path / "m", preset("dogotar-tiny"), 0, std=0.1, gain_noise=0.1, dtype=torch.bfloat16)
    llm = LLM(folder, dtype="bfloat16", max_seq_len=64, num_blocks=32, max_running_requests=2)
    got = llm.generate([[5, 6, 7], [9]], SamplingParams(max_tokens=4, ignore_eos=True))
    assert [len(g) for g in got] == [4, 4]
