"""Vurazen through the engine against the plain implementation (tests/plain_vurazen.py): each mechanism alone, prompts whole
and token by token, portions down to two tokens, mixed batches, pages and state slots that are used again, keys just inside
and just outside a window and among the kept first tokens, at page borders and far back, sinks, states that remember hundreds
of tokens, the last inputs of a convolution at a portion's start, long decoding, sizes of several kinds, greedy generation
through the engine's own entry point and scheduler."""
import numpy as np
import pytest
import torch

import plain_vurazen as plain
from conftest import assert_logits_close, rel_err

pytestmark = pytest.mark.gpu

S, P, L, moe = plain.scan_layer, plain.parallel_layer, plain.lightning_layer, plain.moe

MIXED = plain.make_config([P(), S(mlp=moe()), L(), S(mlp=moe(ff=40, experts=5, top=3, shared_ff=33)), P(window=37, keep_first=17, mlp=None)], loop=(1, 4, 2))
ODD = plain.make_config([L(heads=5, dim=7, vdim=9, mlp=moe(ff=20, experts=6, top=1, shared_ff=9)),
                         P(heads=6, kv_heads=2, dim=14, window=11, keep_first=1, softcap=4.0, scale=0.5, rot=6, base=300.0, conv=6, rheads=3, rkv_heads=1,
                           rdim=10, rvdim=6, rconv=2, left_scale=1.3, right_scale=0.4, mlp=None),
                         S(inner=30, state=21, dt_rank=1, conv=2, mlp=plain.dense(50)),
                         P(heads=3, kv_heads=3, dim=9, window=50, keep_first=60, rot=2, conv=3, rheads=2, rkv_heads=2, rdim=17, rvdim=3, rconv=7,
                           mlp=moe(ff=12, experts=3, top=3, shared_ff=40)),
                         S(inner=44, state=70, dt_rank=9, conv=5, mlp=None)], vocab=97, width=36, eps=1e-4, scale=0.5, softcap=6.0, loop=(2, 4, 3))
ONES = plain.make_config([P(heads=1, kv_heads=1, dim=2, window=1, keep_first=0, rot=2, conv=1, rheads=1, rkv_heads=1, rdim=1, rvdim=1, rconv=1,
                            left_scale=1.0, right_scale=1.0, mlp=moe(ff=1, experts=1, top=1, shared_ff=1)),
                          S(inner=1, state=1, dt_rank=1, conv=1), L(heads=1, dim=1, vdim=1, decay=[1.0], mlp=plain.dense(1))],
                         vocab=33, width=16, scale=1.0, loop=(0, 3, 1))
# sizes in whole 16-byte pieces, heads that the tensor-core kernels take
SQUARE = plain.make_config([P(heads=8, kv_heads=2, dim=64, window=70, keep_first=5, rot=32, rheads=4, rkv_heads=4, rdim=32, rvdim=64, mlp=moe(ff=64, experts=8, top=2, shared_ff=64)),
                            S(inner=256, state=16, dt_rank=8, mlp=plain.dense(96)), L(heads=4, dim=32, vdim=64, mlp=moe(ff=32, experts=12, top=3, shared_ff=32)),
                            P(heads=4, kv_heads=4, dim=128, window=130, keep_first=70, softcap=50.0, rot=64, rheads=2, rkv_heads=1, rdim=64, rvdim=32)],
                           width=128, loop=(1, 3, 2))
# What the routed experts of the whole-model tests add to the stream is scaled down: among hundreds of random routing decisions
# some are close calls that bfloat16 rounding decides the other way; at this gain such a flip stays within the bfloat16
# tolerance. The experts at full gain are held to float32 accuracy by `test_each_mechanism_alone`.
GAIN = 0.1
CONFIGS = {"mixed": (MIXED, (6, 10), 16), "odd": (ODD, (3, 5), 8), "ones": (ONES, (1, 1), 4), "square": (SQUARE, (16, 8), 16)}


class Want:
    def __init__(self, rows, noise):
        self.rows, self.noise = np.asarray(rows), noise

    def __getitem__(self, idx):
        return Want(self.rows[idx], self.noise)


def reference(w, cfg, toks):
    exact = plain.forward(w, cfg, toks)
    with plain.bfloat16_activations():
        rounded = plain.forward(w, cfg, toks)
    return Want(exact, rel_err(rounded, exact))


def close(got, want, dtype, what):
    """float32: 1e-4 of the row's largest logit and the same argmax. bfloat16: four times the noise of 16-bit activations
    on this very model and prompt, and at least 2e-2."""
    if dtype == "float32":
        assert_logits_close(got, want.rows, dtype, what)
    else:
        err, tol = rel_err(got, want.rows), max(2e-2, 4.0 * want.noise)
        assert err <= tol, f"{what}: relative error {err:.3e} above {tol:.1e} (bfloat16; noise of rounding {want.noise:.1e})"


class Harness:
    """A model folder, the engine's model, cache, state slots and step function; `step` takes
    [(request id, tokens, wanted places)] and returns {(id, position): logits}."""

    def __init__(self, tmp, cfg, weights, dtype, page=16, pages=64, slots=4, max_tokens=512):
        from tiny_inference_engine_b200 import StepRunner, load_model, make_cache
        plain.write_model_dir(tmp, cfg, weights)
        self.model = load_model(tmp, dtype)
        self.cache, self.states = make_cache(self.model, page_size=page, num_pages=pages, max_requests=slots)
        self.runner = StepRunner(self.model, self.cache, max_tokens=max_tokens, max_seqs=8, max_logit_rows=max_tokens, states=self.states)
        self.live = {}

    def step(self, entries, end=()):
        from tiny_inference_engine_b200 import StepEntry
        batch, keys = [], []
        for rid, tokens, want in entries:
            if rid not in self.live:
                self.live[rid] = [self.cache.new_request(), 0]
            req, have = self.live[rid]
            assert self.cache.reserve(req, have + len(tokens)), "pool too small for the test"
            batch.append(StepEntry(req, list(tokens), have, list(want)))
            keys += [(rid, have + w) for w in want]
        logits = self.runner.run(batch)
        for (rid, tokens, _), e in zip(entries, batch):
            self.live[rid][1] += len(tokens)
            self.cache.advance_window(e.cache, self.live[rid][1])
        out = {}
        if logits is not None:
            host = logits.float().cpu().numpy()
            out = {k: host[i] for i, k in enumerate(keys)}
        torch.cuda.synchronize()
        self.runner.check()
        for rid in end:
            self.cache.release(self.live.pop(rid)[0])
        return out

    def whole(self, rid, tokens):
        got = self.step([(rid, tokens, range(len(tokens)))], end=[rid])
        return np.stack([got[(rid, i)] for i in range(len(tokens))])

    def in_portions(self, rid, tokens, sizes):
        rows, at, i = {}, 0, 0
        while at < len(tokens):
            n = min(sizes[i % len(sizes)], len(tokens) - at)
            rows.update(self.step([(rid, tokens[at:at + n], range(n))]))
            at, i = at + n, i + 1
        self.cache.release(self.live.pop(rid)[0])
        return np.stack([rows[(rid, j)] for j in range(len(tokens))])


def tokens_of(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


@pytest.fixture(scope="module")
def truth():
    memo = {}

    def get(name, toks):
        cfg, ranks, _ = CONFIGS[name]
        key = (name, tuple(toks))
        if key not in memo:
            memo[key] = reference(plain.random_weights(cfg, 5, ranks=ranks, expert_gain=GAIN), cfg, toks)
        return memo[key]
    return get


# ---------------------------------------------------------------------------------------------- each mechanism alone

V60 = dict(vocab=60, width=48)
SINGLE = {
    "scan": plain.make_config([S(mlp=None)], **V60),
    "scan_many_states": plain.make_config([S(inner=20, state=33, dt_rank=11, conv=3, mlp=None), S(inner=24, state=130, dt_rank=2, conv=8, mlp=None),
                                           S(inner=17, state=5, dt_rank=40, conv=1, mlp=None)], **V60),
    "scan_aligned": plain.make_config([S(inner=128, state=16, dt_rank=16, mlp=None), S(inner=64, state=24, dt_rank=8, mlp=None),
                                       S(inner=64, state=64, dt_rank=8, mlp=None), S(inner=32, state=256, dt_rank=8, mlp=None)], vocab=60, width=64),
    "attention": plain.make_config([P(right_scale=0.0, mlp=None)], **V60),
    "attention_one_kv_head_no_kept_tokens": plain.make_config([P(heads=5, kv_heads=1, dim=10, keep_first=0, rot=4, right_scale=0.0, mlp=None)], **V60),
    "attention_a_kv_head_each_whole_head_rotated": plain.make_config([P(heads=3, kv_heads=3, dim=12, rot=12, conv=2, softcap=2.0, right_scale=0.0, mlp=None)], **V60),
    "attention_heads_of_64": plain.make_config([P(heads=4, kv_heads=1, dim=64, rot=48, softcap=30.0, right_scale=0.0, mlp=None)], **V60),
    "attention_heads_of_256": plain.make_config([P(heads=2, kv_heads=1, dim=256, rot=16, right_scale=0.0, mlp=None)], **V60),
    "attention_no_taps": plain.make_config([P(heads=2, kv_heads=1, dim=64, conv=1, right_scale=0.0, mlp=None)], **V60),
    "delta": plain.make_config([P(left_scale=0.0, mlp=None)], **V60),
    "delta_large_heads": plain.make_config([P(left_scale=0.0, rheads=2, rkv_heads=1, rdim=80, rvdim=24, mlp=None), P(left_scale=0.0, rheads=6, rkv_heads=3, rdim=6, rvdim=40, mlp=None)], **V60),
    "both_halves": plain.make_config([P(mlp=None)], **V60),
    "lightning": plain.make_config([L(mlp=None)], **V60),
    "lightning_long_rows": plain.make_config([L(heads=2, dim=40, vdim=300, mlp=None), L(heads=7, dim=5, vdim=3, decay=[0.0, 0.3, 0.5, 0.9, 0.99, 0.9999, 1.0], mlp=None)], **V60),
    "dense": plain.make_config([L(mlp=plain.dense(56)), L(mlp=plain.dense(64))], **V60),
    "experts": plain.make_config([L(mlp=moe(ff=20, experts=7, top=3, shared_ff=31))], **V60),
    "experts_all_chosen": plain.make_config([S(mlp=moe(ff=12, experts=3, top=3, limit=0.3, shared_ff=12, shared_limit=3.0))], **V60),
    "passes": plain.make_config([L(mlp=None), S(mlp=None), L(mlp=None)], loop=(0, 2, 3), **V60),
    "one_pass_of_the_last_layer": plain.make_config([L(mlp=None), S(mlp=None)], loop=(1, 2, 1), **V60),
    "odd_width": plain.make_config([P(heads=2, kv_heads=1, dim=6, rot=2, rheads=3, rkv_heads=3, rdim=7, rvdim=5, mlp=plain.dense(19)), S(inner=13, state=3, dt_rank=2, mlp=moe(ff=9, experts=3, top=2, shared_ff=7))],
                                   vocab=51, width=38, eps=1e-3),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SINGLE))
def test_each_mechanism_alone(tmp_path, name, dtype):
    cfg = SINGLE[name]
    w = plain.random_weights(cfg, 3, ranks=(4, 6))
    toks = tokens_of(cfg, 61, 1)
    got = Harness(tmp_path, cfg, w, dtype).whole("a", toks)
    close(got, reference(w, cfg, toks), dtype, name)


# ---------------------------------------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_decoding_and_portions(tmp_path, truth, name, dtype):
    """The same logits at every position whether the prompt comes whole, token by token from the first token on (inputs
    before the first that are zeros, states that start empty), or in portions of several sizes down to two."""
    cfg, ranks, page = CONFIGS[name]
    w = plain.random_weights(cfg, 5, ranks=ranks, expert_gain=GAIN)
    toks = tokens_of(cfg, 150, 2)
    want = truth(name, toks)
    hs = Harness(tmp_path, cfg, w, dtype, page=page, pages=256 // page * 2)
    close(hs.whole("w", toks), want, dtype, f"{name} whole")
    close(hs.in_portions("d", toks, [1]), want, dtype, f"{name} token by token")
    close(hs.in_portions("p", toks, [2, 3, 17, 2, 1, 40, 5]), want, dtype, f"{name} portions")
    close(hs.in_portions("q", toks, [1, 1, 2, 64, 7]), want, dtype, f"{name} first tokens one by one, then portions")
    rows = hs.step([("m", toks[:101], [100])])
    for i in range(101, 150):
        rows.update(hs.step([("m", toks[i:i + 1], [0])]))
    hs.cache.release(hs.live.pop("m")[0])
    close(np.stack([rows[("m", i)] for i in range(100, 150)]), want[100:], dtype, f"{name} prompt then decoding")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "square"])
def test_mixed_batches_on_a_small_pool_with_two_state_slots(tmp_path, truth, name, dtype):
    """Requests of unequal lengths, portions of some beside single tokens of others, never more than two alive: pages and
    state slots are given back and used again, a request sits out a step now and then, and every row equals the request run alone."""
    cfg, ranks, page = CONFIGS[name]
    w = plain.random_weights(cfg, 5, ranks=ranks, expert_gain=GAIN)
    lengths = [70, 33, 2, 90, 47, 64]
    reqs = [tokens_of(cfg, n, 10 + i) for i, n in enumerate(lengths)]
    want = [truth(name, r) for r in reqs]
    hs = Harness(tmp_path, cfg, w, dtype, page=page, pages=(2 * 128) // page, slots=2)
    rows, at = {}, [0] * len(reqs)
    pending, alive, turn = list(range(len(reqs))), [], 0
    sizes = [5, 1, 2, 31, 1, 1, 16, 3]
    while pending or alive:
        while pending and len(alive) < 2:
            alive.append(pending.pop(0))
        entries, ended = [], []
        for k, i in enumerate(alive):
            if len(alive) == 2 and k == 1 and turn % 5 == 4:
                continue                                   # left out of this step, goes on later
            n = min(1 if (turn + k) % 3 == 0 else sizes[(turn + i) % len(sizes)], lengths[i] - at[i])
            entries.append((f"r{i}", reqs[i][at[i]:at[i] + n], range(n)))
            at[i] += n
            if at[i] == lengths[i]:
                ended.append(i)
        rows.update(hs.step(entries, end=[f"r{i}" for i in ended]))
        alive = [i for i in alive if i not in ended]
        turn += 1
    assert hs.states.num_free == 2 and all(p.num_free == p.num_blocks for p in hs.cache.pools)
    for i, r in enumerate(reqs):
        close(np.stack([rows[(f"r{i}", j)] for j in range(len(r))]), want[i], dtype, f"{name} request {i} in mixed batches")


# ---------------------------------------------------------------------------------------------- edges that random weights would hide

def _one_token_stands_out(w, cfg, marked, quiet=0.4):
    """Column `mark` of the embedding is zero but for token `marked`, column `const` is one number for every token: behind the
    first norm (its weights one, its biases zero) the first is a large entry for the marked token and a small one for the others,
    the second about the same for all. `quiet` scales the other columns. Returns the two columns."""
    mark, const = cfg["width"] - 2, cfg["width"] - 1
    emb = w["embed"].astype(np.float64) * quiet
    emb[:, mark], emb[:, const] = 0.0, 1.0
    emb[marked, mark] = 3.0
    w["embed"] = plain.round_bf16(emb)
    w["l0.norm1"][:], w["l0.norm1.b"][:] = 1.0, 0.0
    return mark, const


def _identity_conv(w, name):
    w[name][:] = 0.0
    w[name][:, -1] = 1.0


def _marked_tokens(cfg, n, at, seed, marked=7):
    toks = [t if t != marked else marked + 1 for t in tokens_of(cfg, n, seed)]
    toks[at] = marked
    other = list(toks)
    other[at] = marked + 2
    return toks, other


def _peaked(window, keep_first, at, n, dim, heads, kv_heads, softcap=40.0):
    """One parallel layer, its right half switched off, in which the key of the token at place `at` outweighs all other keys
    together for every later query that sees it. (The dimension that carries it is not rotated.)"""
    cfg = plain.make_config([P(heads=heads, kv_heads=kv_heads, dim=dim, window=window, keep_first=keep_first, softcap=softcap, scale=1.0, rot=dim // 4 * 2,
                               right_scale=0.0, mlp=None)], vocab=40, width=32, scale=1.0)
    w = plain.random_weights(cfg, 8, sharp=1.0)
    marked = 7
    mark, const = _one_token_stands_out(w, cfg, marked)
    p = "l0.mix.left."
    for leaf, count in (("q", heads), ("k", kv_heads)):
        w[p + leaf] = plain.round_bf16(w[p + leaf] * 0.3)
        w[p + leaf + ".b"][:] = 0.0
        _identity_conv(w, p + leaf + ".conv")
        for h in range(count):
            w[p + leaf][h * dim + dim - 1] = 0.0
            w[p + leaf][h * dim + dim - 1, const if leaf == "q" else mark] = 3.0 if leaf == "q" else 4.0
    w[p + "sink"][:] = plain.round_bf16(np.linspace(-1.0, 2.0, heads))
    toks, other = _marked_tokens(cfg, n, at, 4)
    return cfg, w, toks, other


GEOMETRIES = [(16, 4, 2, 8), (64, 2, 1, 16), (128, 8, 1, 8), (20, 3, 3, 4)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("geometry", GEOMETRIES)
def test_a_key_just_inside_and_just_outside_the_window(tmp_path, dtype, geometry):
    """A key that dominates the softmax while it is seen, on a page's first slot: the rows up to window - 1 places behind it differ
    visibly from the same rows without it, the row at window places and all later ones do not. Whole, in portions cut at the
    edge, two tokens across it, the edge rows alone, and decoded."""
    dim, heads, kv_heads, page = geometry
    window, keep, at, n = 33, 2, 48, 110
    cfg, w, toks, other = _peaked(window, keep, at, n, dim, heads, kv_heads)
    ref, moved = reference(w, cfg, toks), plain.forward(w, cfg, other)
    edge = at + window
    inside, outside = list(range(at + 1, edge)), list(range(0, at)) + list(range(edge, n))
    assert rel_err(moved[inside], ref.rows[inside]) > 0.15 and rel_err(moved[outside], ref.rows[outside]) < 1e-9
    assert all(rel_err(moved[[i]], ref.rows[[i]]) > 0.1 for i in (at + 1, edge - 1))
    hs = Harness(tmp_path, cfg, w, dtype, page=page, pages=4 * 160 // page)
    close(hs.whole("w", toks), ref, dtype, "whole")
    close(hs.in_portions("a", toks, [edge, n]), ref, dtype, "cut at the edge")
    close(hs.in_portions("b", toks, [edge - 1, 2, n]), ref, dtype, "two tokens across the edge")
    close(hs.in_portions("c", toks, [at, 1, window - 2, 1, 1, 1, n]), ref, dtype, "the rows around the edge alone")
    close(hs.in_portions("d", toks, [at - 3] + [1] * n), ref, dtype, "decoded across the edge")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("geometry", GEOMETRIES)
@pytest.mark.parametrize("keep", [5, 70])
def test_the_first_tokens_stay_and_the_next_one_does_not(tmp_path, dtype, geometry, keep):
    """The last kept token is seen by every later row, hundreds of places behind; the token after it leaves with the window. Their
    pages come back to others meanwhile: a second request runs beside and takes every page the window has passed."""
    dim, heads, kv_heads, page = geometry
    window, n = 24, 300
    hs = None
    for at, stays in ((keep - 1, True), (keep, False)):
        cfg, w, toks, other = _peaked(window, keep, at, n, dim, heads, kv_heads)
        ref, moved = reference(w, cfg, toks), plain.forward(w, cfg, other)
        late = list(range(at + window, n))
        assert (rel_err(moved[late], ref.rows[late]) > 0.15) if stays else (rel_err(moved[late], ref.rows[late]) < 1e-9)
        hs = Harness(tmp_path / str(at), cfg, w, dtype, page=page, pages=2 * 304 // page)
        close(hs.whole("w", toks), ref, dtype, f"whole, key at {at}")
        rows = hs.step([("a", toks[:at + 1], range(at + 1))])
        rows.update(hs.step([("a", toks[at + 1:200], range(199 - at)), ("x", other[:200], [])]))
        for i in range(200, n):
            rows.update(hs.step([("a", toks[i:i + 1], [0])] + ([("x", other[i:i + 1], [])] if i % 2 == 0 and i < 260 and i - 200 < 2 else [])))
        close(np.stack([rows[("a", i)] for i in range(n)]), ref, dtype, f"portions, then decoded, key at {at}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("geometry", [(64, 8, 2, 16, 1500, 64), (64, 2, 2, 8, 1000, 3), (20, 4, 2, 8, 700, 130)])
def test_many_splits_of_a_long_window_with_kept_tokens(tmp_path, dtype, geometry):
    """Single rows whose window is long enough to be cut into several splits: the kept tokens and the sink count once. The key
    that carries the rows is the last kept one."""
    dim, heads, kv_heads, page, window, keep = geometry
    n = window + keep + 120
    cfg, w, toks, other = _peaked(window, keep, keep - 1, n, dim, heads, kv_heads)
    ref = reference(w, cfg, toks)
    hs = Harness(tmp_path, cfg, w, dtype, page=page, pages=2 * (n // page + 2), max_tokens=n)
    rows = hs.step([("d", toks[:n - 40], range(n - 100, n - 40))])
    for i in range(n - 40, n):
        rows.update(hs.step([("d", toks[i:i + 1], [0])]))
    close(np.stack([rows[("d", i)] for i in range(n - 100, n)]), ref[n - 100:], dtype, "prompt, then decoded through splits")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("geometry", [(16, 4, 2, 8), (64, 4, 2, 16)])
def test_the_sink_counts_once_and_unscaled(tmp_path, dtype, geometry):
    """Scores near zero and sinks that are worth as much as the whole window: without the sink, or with the sink scaled or
    capped like a score, every row would be visibly another one."""
    dim, heads, kv_heads, page = geometry
    cfg = plain.make_config([P(heads=heads, kv_heads=kv_heads, dim=dim, window=40, keep_first=4, softcap=1.5, scale=0.02, right_scale=0.0, mlp=None)], vocab=40, width=32)
    w = plain.random_weights(cfg, 6, sharp=1.0)
    w["l0.mix.left.sink"][:] = plain.round_bf16(np.linspace(2.5, 5.0, heads))
    toks = tokens_of(cfg, 130, 5)
    ref = reference(w, cfg, toks)
    none = {k: (np.full_like(v, -80.0) if k.endswith("sink") else v) for k, v in w.items()}
    capped = {k: (1.5 * np.tanh(v / 1.5) if k.endswith("sink") else v) for k, v in w.items()}
    assert rel_err(plain.forward(none, cfg, toks)[60:], ref.rows[60:]) > 0.08 and rel_err(plain.forward(capped, cfg, toks)[60:], ref.rows[60:]) > 0.07
    hs = Harness(tmp_path, cfg, w, dtype, page=page)
    close(hs.whole("w", toks), ref, dtype, "whole")
    close(hs.in_portions("d", toks, [90] + [1] * 40), ref, dtype, "decoded")


def _far_memory(kind):
    """One layer of a recurrent kind whose state forgets slowly: what the token at place 3 wrote still decides the last rows."""
    build = {"scan": S(inner=24, state=10, dt_rank=4, mlp=None), "lightning": L(heads=2, dim=12, vdim=12, decay=[0.9995, 0.999], mlp=None),
             "delta": P(left_scale=0.0, rheads=2, rkv_heads=2, rdim=16, rvdim=12, mlp=None)}[kind]
    cfg = plain.make_config([build], vocab=40, width=32, scale=1.0)
    w = plain.random_weights(cfg, 11)
    mark, const = _one_token_stands_out(w, cfg, 7)
    p = "l0.mix." + ("right." if kind == "delta" else "")
    scale_rows = lambda leaf, c, rows=slice(None): w[p + leaf].__setitem__(rows, plain.round_bf16(w[p + leaf][rows] * c))
    if kind == "scan":
        _identity_conv(w, p + "conv")
        w[p + "conv.b"][:] = 0.0
        scale_rows("in", 0.1, slice(0, 24))
        w[p + "in"][:24, mark], w[p + "in"][:24, const] = 0.0, 0.25
        w[p + "in"][:24:2, mark] = 4.0      # every second channel: what the marked token writes points elsewhere than the rest
        w[p + "dt"][:], w[p + "dt.b"][:], w[p + "A_log"][:], w[p + "D"][:] = 0.0, -2.0, -6.0, 0.0
        scale_rows("x", 0.5)
    elif kind == "lightning":
        for leaf in ("q", "k", "v"):
            scale_rows(leaf, 0.1 if leaf != "v" else 1.0)
        w[p + "k"][:, mark], w[p + "k"][:, const] = 4.0, 0.0
        w[p + "q"][:, const] = 2.0
    else:
        for leaf in ("q", "k", "v"):
            _identity_conv(w, p + leaf + ".conv")
        w[p + "A_log"][:], w[p + "dt_bias"][:] = -4.0, -5.0
        w[p + "a2"] = plain.round_bf16(w[p + "a2"] * 0.1)
        w[p + "b"][:] = 0.0
        w[p + "b"][:, const], w[p + "b"][:, mark] = -3.0, 4.0
        w[p + "v"][:, mark] = 3.0
        for leaf in ("q", "k"):      # the marked key and every query share a direction
            w[p + leaf][::4, const if leaf == "q" else mark] = 6.0
    w[p + "o"] = plain.round_bf16(w[p + "o"] * (0.15 if kind == "scan" else 3.0))
    return (cfg, w) + _marked_tokens(cfg, 400, 3, 12)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["scan", "lightning", "delta"])
def test_a_state_remembers_a_token_hundreds_back(tmp_path, dtype, kind):
    """The state is carried through a prompt portion, through another, and through decoding, and a second request in another
    slot in between does not touch it."""
    cfg, w, toks, other = _far_memory(kind)
    want, moved = reference(w, cfg, toks), plain.forward(w, cfg, other)
    assert rel_err(moved[-5:], want.rows[-5:]) > 5e-2      # a token 396 back is still felt
    hs = Harness(tmp_path, cfg, w, dtype, pages=64, max_tokens=512)
    close(hs.whole("w", toks), want, dtype, "whole")
    rows = hs.step([("a", toks[:130], range(130))])
    rows.update(hs.step([("x", other[:77], [])]))                       # another request takes another slot
    rows.update(hs.step([("a", toks[130:300], range(170)), ("x", other[77:78], [])]))
    for i in range(300, 400):
        rows.update(hs.step([("a", toks[i:i + 1], [0])] + ([("x", other[78 + i - 300:79 + i - 300], [])] if i % 2 else [])))
    close(np.stack([rows[("a", i)] for i in range(400)]), want, dtype, "portions, then decoding beside another request")


@pytest.mark.parametrize("taps", [2, 4, 7])
def test_a_convolutions_last_inputs_come_from_the_slot_at_a_portions_start(tmp_path, taps):
    """Taps that weigh the oldest input most: a portion's first rows must read the inputs of the portions before (of one, two or
    three tokens, shorter than the taps) from the request's slot, and a sequence's first rows zeros, also in a slot that another
    request has just left. All three kinds of convolution: q and k of attention, the delta rule's, the scan's."""
    cfg = plain.make_config([P(conv=taps, rconv=taps, mlp=None), S(conv=taps, mlp=None)], vocab=40, width=32)
    w = plain.random_weights(cfg, 13)
    for name in w:
        if name.endswith(".conv"):
            w[name] = np.ascontiguousarray(w[name][:, ::-1])
    a, b = tokens_of(cfg, 60, 1), tokens_of(cfg, 45, 2)
    hs = Harness(tmp_path, cfg, w, "float32", slots=1)
    close(hs.in_portions("a", a, [7, 1, 2, 1, 1, 3, 13]), reference(w, cfg, a), "float32", "first request")
    close(hs.in_portions("b", b, [1, 2, 5, 9]), reference(w, cfg, b), "float32", "second request in the same slot")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_captured_steps_and_slots_used_again(tmp_path, truth, dtype):
    """Three requests decode together for 200 steps (steps of one token each are captured as graphs and replayed), end at
    different times, and a fourth takes over a slot and pages that were just given back."""
    cfg, ranks, page = CONFIGS["mixed"]
    w = plain.random_weights(cfg, 5, ranks=ranks, expert_gain=GAIN)
    reqs = [tokens_of(cfg, n, 20 + i) for i, n in enumerate([230, 215, 260, 120])]
    want = [truth("mixed", r) for r in reqs]
    hs = Harness(tmp_path, cfg, w, dtype, page=page, pages=3 * 272 // page, slots=3)
    rows = hs.step([(f"r{i}", reqs[i][:12 + i], range(12 + i)) for i in range(3)])
    at = [12, 13, 14, 0]
    alive = [0, 1, 2]
    while alive:
        ended = [i for i in alive if at[i] + 1 == len(reqs[i])]
        rows.update(hs.step([(f"r{i}", reqs[i][at[i]:at[i] + 1], [0]) for i in alive], end=[f"r{i}" for i in ended]))
        for i in alive:
            at[i] += 1
        alive = [i for i in alive if i not in ended]
        if ended and at[3] == 0:                          # the newcomer's prompt rides beside the others' single tokens
            rows.update(hs.step([("r3", reqs[3][:40], range(40))] + [(f"r{i}", reqs[i][at[i]:at[i] + 1], [0]) for i in alive]))
            for i in alive:
                at[i] += 1
            at[3] = 40
            alive.append(3)
    assert hs.runner.graph_replays > 100, "decode steps of this model are meant to be captured"
    for i, r in enumerate(reqs):
        close(np.stack([rows[(f"r{i}", j)] for j in range(len(r))]), want[i], dtype, f"request {i}")


# ---------------------------------------------------------------------------------------------- the engine's own entry points

def test_greedy_generation_through_the_engine_and_its_scheduler(tmp_path):
    from tiny_inference_engine_b200 import SamplingParams, ServingConfig, load_engine
    cfg, ranks, page = CONFIGS["mixed"]
    w = plain.random_weights(cfg, 5, ranks=ranks, expert_gain=GAIN)
    plain.write_model_dir(tmp_path, cfg, w)
    prompts = [tokens_of(cfg, n, 30 + i) for i, n in enumerate([19, 3, 41, 1, 27])]
    want = [plain.generate(w, cfg, p, 24) for p in prompts]
    engine = load_engine(tmp_path, dtype="float32", num_pages=40, page_size=page, serving=ServingConfig(max_seqs=3, max_tokens_per_step=16))
    assert engine.generate(prompts[0], SamplingParams(max_tokens=24)) == want[0]
    assert engine.generate_batch(prompts, SamplingParams(max_tokens=24)) == want
    tight = load_engine(tmp_path, dtype="float32", num_pages=9, page_size=page, serving=ServingConfig(max_seqs=3, max_tokens_per_step=16))
    assert tight.generate_batch(prompts, SamplingParams(max_tokens=24)) == want


def test_the_command_line_generates_the_plain_greedy_tokens(tmp_path, capsys):
    from tiny_inference_engine_b200.cli.main import main
    cfg, ranks, page = CONFIGS["odd"]
    w = plain.random_weights(cfg, 5, ranks=ranks, expert_gain=GAIN)
    plain.write_model_dir(tmp_path, cfg, w)
    prompt = tokens_of(cfg, 21, 77)
    assert main(["generate", "-m", str(tmp_path), "-p", " ".join(map(str, prompt)), "--temp", "0", "--max-tokens", "12",
                 "--dtype", "float32", "--kv-mem", "64M", "--max-tokens-per-step", "8", "--max-seqs", "2"]) == 0
    assert [int(t) for t in capsys.readouterr().out.split()] == plain.generate(w, cfg, prompt, 12)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_of_a_vurazen_model(tmp_path, truth, dtype):
    from test_replay_gpu import Replay
    cfg, ranks, page = CONFIGS["odd"]
    w = plain.random_weights(cfg, 5, ranks=ranks, expert_gain=GAIN)
    plain.write_model_dir(tmp_path / "m", cfg, w)
    reqs = [tokens_of(cfg, n, 40 + i) for i, n in enumerate([100, 37, 64, 2, 81])]
    want = [truth("odd", r) for r in reqs]
    V = cfg["vocab"]
    rp = Replay(tmp_path / "m", dtype, tmp_path / "out", max_tokens=4 * 128, page_size=page)
    try:
        got = rp.step([("a", reqs[0][:50], range(50)), ("b", reqs[1], range(37))], end=["b"]).reshape(87, V)
        close(got[:50], want[0][:50], dtype, "a, first portion")
        close(got[50:], want[1], dtype, "b whole beside it")
        got = rp.step([("c", reqs[2][:2], [1]), ("a", reqs[0][50:51], [0]), ("d", reqs[3], [0, 1])], end=["d"]).reshape(4, V)
        noise = max(x.noise for x in want)
        close(got, Want(np.stack([want[2].rows[1], want[0].rows[50], want[3].rows[0], want[3].rows[1]]), noise), dtype, "three requests, one step")
        assert rp.step([("e", reqs[4][:80], [])]) is None
        got = rp.step([("e", reqs[4][80:], [0]), ("a", reqs[0][51:], range(49)), ("c", reqs[2][2:], [61])], end=["a", "c", "e"]).reshape(51, V)
        close(got, Want(np.concatenate([want[4].rows[80:81], want[0].rows[51:], want[2].rows[63:64]]), noise), dtype, "the rest")
    finally:
        rp.close()


# ---------------------------------------------------------------------------------------------- sizes drawn at random

def _random_config(seed):
    """A configuration with every size, count, constant and the order of layers drawn from what the design allows."""
    r = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(r.integers(len(xs)))]
    aligned = seed % 3 == 0                                # every third draw: sizes in whole 16-byte pieces

    def mlp():
        kind = pick("none", "dense", "moe", "moe")
        if kind == "none":
            return None
        if kind == "dense":
            return plain.dense(pick(24, 50, 64))
        experts = pick(1, 2, 5, 8, 12)
        return moe(ff=pick(8, 20, 32), experts=experts, top=int(r.integers(1, min(experts, 6) + 1)), limit=pick(0.4, 2.0), shared_ff=pick(8, 27), shared_limit=pick(0.5, 3.0))
    layers = []
    for i in range(int(r.integers(2, 6))):
        kind = pick("scan", "parallel", "parallel", "lightning")
        if kind == "scan":
            layers.append(S(inner=pick(32, 64, 128) if aligned else pick(10, 27, 40, 60), state=pick(16, 24) if aligned else pick(1, 5, 16, 40, 100), dt_rank=pick(1, 4, 8, 13),
                            conv=pick(1, 2, 3, 4, 6), mlp=mlp()))
        elif kind == "lightning":
            heads = pick(1, 2, 5)
            layers.append(L(heads=heads, dim=pick(16, 32) if aligned else pick(3, 8, 20, 40), vdim=pick(16, 64) if aligned else pick(3, 10, 36),
                            decay=r.uniform(0.3, 0.9999, heads).tolist(), mlp=mlp()))
        else:
            kv, rkv, dim = pick(1, 2, 3), pick(1, 2), pick(64, 128) if aligned else pick(4, 10, 20, 48)
            layers.append(P(heads=kv * pick(1, 2, 4), kv_heads=kv, dim=dim, window=pick(1, 2, 5, 16, 33, 64, 400), keep_first=pick(0, 1, 4, 17, 64),
                            softcap=pick(2.0, 10.0, 50.0), scale=pick(None, 0.3), rot=pick(0, 2, dim // 4 * 2, dim // 2 * 2), base=pick(100.0, 1e4, 5e5), conv=pick(1, 2, 4, 5),
                            rheads=rkv * pick(1, 2, 3), rkv_heads=rkv, rdim=pick(16, 32) if aligned else pick(4, 12, 40), rvdim=pick(16, 64) if aligned else pick(3, 12, 36),
                            rconv=pick(1, 2, 4, 5), left_scale=pick(0.5, 1.0), right_scale=pick(0.4, 1.3), mlp=mlp()))
    start = int(r.integers(0, len(layers)))
    loop = None if r.random() < 0.3 else (start, int(r.integers(start + 1, len(layers) + 1)), pick(1, 2, 3))
    cfg = plain.make_config(layers, vocab=pick(33, 97, 160, 301), width=pick(24, 36, 64, 72, 128), eps=pick(1e-6, 1e-5, 1e-3), scale=pick(0.7, 1.0, 8.0),
                            softcap=pick(5.0, 30.0), loop=loop)
    return cfg, (pick(1, 3, 8, 24), pick(1, 5, 16)), pick(4, 8, 16, 32)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(15))
def test_configurations_drawn_at_random(tmp_path, seed, dtype):
    cfg, ranks, page = _random_config(seed)
    w = plain.random_weights(cfg, 100 + seed, ranks=ranks, expert_gain=GAIN)
    a, b = tokens_of(cfg, 83, seed), tokens_of(cfg, 31, 50 + seed)
    want_a, want_b = reference(w, cfg, a), reference(w, cfg, b)
    hs = Harness(tmp_path, cfg, w, dtype, page=page, pages=2 * 128 // page, slots=2)
    close(hs.whole("w", a), want_a, dtype, f"seed {seed} whole")
    rows = hs.step([("a", a[:29], range(29)), ("b", b[:2], range(2))])
    rows.update(hs.step([("a", a[29:31], range(2)), ("b", b[2:], range(29))], end=["b"]))
    rows.update(hs.step([("a", a[31:70], range(39))]))
    for i in range(70, 83):
        rows.update(hs.step([("a", a[i:i + 1], [0])]))
    close(np.stack([rows[("a", i)] for i in range(83)]), want_a, dtype, f"seed {seed} in portions beside another request, then decoded")
    close(np.stack([rows[("b", i)] for i in range(31)]), want_b, dtype, f"seed {seed} the other request")


# ---------------------------------------------------------------------------------------------- kernels alone

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D", [50, 320, 5000])
def test_the_layer_norm_adds_up_to_four_terms_in_float(dtype, D):
    from tiny_inference_engine_b200 import ops
    g = torch.Generator(device="cuda").manual_seed(1)
    T = 37
    draw = lambda *shape: torch.randn(*shape, device="cuda", generator=g)
    x, a, b, part, other = 5.0 + draw(T, D), draw(T, D).to(dtype), draw(T, D).to(dtype), draw(3, T, D), draw(T, D)
    w, bias, vec = draw(D), draw(D), draw(D)
    terms = ops.ScaledSum([(a, 0.6), (ops.SplitSum(part.reshape(-1), 3, T, D), 0.9), (b, 1.0), (a, -0.25)])
    want_x = x.double() + 0.35 * a.double() + 0.9 * part.double().sum(0) + b.double()
    norm = lambda v: (v - v.mean(-1, keepdim=True)) / (((v - v.mean(-1, keepdim=True)) ** 2).mean(-1, keepdim=True) + 1e-3).sqrt() * w.double() + bias.double()
    tol = 2e-5 if dtype == torch.float32 else 6e-2
    out, x1 = torch.empty(T, D, device="cuda", dtype=dtype), x.clone()
    ops.add_layer_norm(x1, terms, w, bias, 1e-3, out)
    assert (x1.double() - want_x).abs().max() < 1e-5 and (out.double() - norm(want_x)).abs().max() < tol
    rows = torch.tensor([5, 0, 36], device="cuda", dtype=torch.int32)
    x2, some = x.clone(), torch.empty(3, D, device="cuda", dtype=dtype)
    ops.add_layer_norm(x2, a, w, bias, 1e-3, some, rows=rows)
    assert torch.equal(x2, x)            # with rows the stream stays as it is
    assert (some.double() - norm(x.double() + a.double())[rows.long()]).abs().max() < tol
    x3 = x.clone()
    ops.stream_add(x3, terms, dtype, other=other, vec=vec)
    assert (x3.double() - (want_x + other.double() + vec.double())).abs().max() < 1e-5


def test_decays_close_to_one_do_not_drift_in_float32():
    """A channel that forgets over many thousands of tokens: the sum it holds stays within rounding of the exact one. (4,096 adds
    of half a unit each, to either side, are about 3e-6; decays that err to one side by one unit would be 1e-4.)"""
    from tiny_inference_engine_b200 import ops
    T, I, N = 4096, 16, 8
    g = torch.Generator(device="cuda").manual_seed(2)
    x = torch.rand(T, I, device="cuda", generator=g)
    raw = torch.rand(T, I, device="cuda", generator=g) - 3.0
    low = torch.ones(T, 24, device="cuda")
    A = -torch.logspace(-5, -1, N, device="cuda")[None].repeat(I, 1)
    a2 = (A.double() * 1.4426950408889634).float()
    state = torch.zeros(1, I * N, device="cuda")
    z = torch.full((T, I), 30.0, device="cuda")
    out, zero = torch.empty(T, I, device="cuda"), torch.zeros(I, device="cuda")

    class Ctx:
        query_start = torch.tensor([0, T], device="cuda", dtype=torch.int32)
        state_slots = torch.tensor([0], device="cuda", dtype=torch.int32)
        S, multi_seqs = 1, 1
    ops.selective_scan(x, z, low, 8, 16, raw, zero, a2, zero, state, Ctx, out)
    dt = torch.nn.functional.softplus(raw.double())
    want = torch.zeros(I, N, dtype=torch.float64, device="cuda")
    for t in range(T):
        want = torch.exp(dt[t][:, None] * A.double()) * want + (dt[t] * x[t].double())[:, None]
    assert ((state.view(I, N).double() - want).abs() / want.abs()).max() < 1e-5
    assert ((out[-1].double() / 30.0 - want.sum(1)).abs() / want.sum(1)).max() < 1e-5


def test_rotation_keeps_its_precision_at_large_positions():
    """A key at position 100,003 turned in double precision: neighbouring pairs, dimensions past the rotated ones untouched, the
    value as it was before the rotation."""
    from tiny_inference_engine_b200 import ops
    from tiny_inference_engine_b200.config.spec import PartSpec
    from tiny_inference_engine_b200.parts import build_part
    g = torch.Generator(device="cuda").manual_seed(3)
    pos = torch.tensor([0, 1, 777, 100003], device="cuda", dtype=torch.int32)
    proj = torch.randn(4, 48, device="cuda", generator=g)
    k, v = (torch.zeros(1, 1, 8, 16, device="cuda") for _ in range(2))
    q = torch.empty(4, 32, device="cuda")
    turns = build_part("position", PartSpec("rope", {"theta": 50.0, "head_dim": 16, "rotary_dim": 10}), torch.float32).turns_table()

    class Ctx:
        seq_of_row = torch.arange(4, device="cuda", dtype=torch.int32)
        query_start = torch.arange(5, device="cuda", dtype=torch.int32)
        state_slots = torch.full((4,), -1, device="cuda", dtype=torch.int32)
        positions, multi_seqs = pos, 0
    slots = torch.arange(4, device="cuda", dtype=torch.int32)
    ops.conv_rope_append(proj, 0, 32, torch.ones(1, 48, device="cuda"), None, None, 0, Ctx, turns, slots, k, v, q, 2, 1, 16)
    heads = proj.double().cpu().numpy().reshape(4, 3, 16)
    want = plain.rotate_pairs(heads, pos.cpu().numpy(), 50.0, 10)
    assert np.abs(q.cpu().numpy().reshape(4, 2, 16) - want[:, :2]).max() < 2e-6
    assert np.abs(k[0, 0, :4].cpu().numpy() - want[:, 2]).max() < 2e-6
    assert torch.equal(v[0, 0, :4], proj[:, 32:])
