"""Sebalorn through the engine against the plain implementation (tests/plain_sebalorn.py): each mechanism alone, prompts whole
and token by token, portions down to two tokens, mixed batches, pages and state slots that are used again, keys far back and at
page borders, through splits, sinks, states that remember hundreds of tokens, long decoding, sizes of several kinds, greedy
generation through the engine's own entry point and scheduler, and the kernels alone."""
import numpy as np
import pytest
import torch

import plain_sebalorn as plain
from conftest import assert_logits_close, rel_err

pytestmark = pytest.mark.gpu

LA, A, R = plain.latent_layer, plain.attention_layer, plain.retention_layer

MIXED = plain.make_config([A(), LA(), R(), LA(heads=5, mlp=plain.dense(40)), A(heads=3, kv_heads=1, dim=20, vdim=20, rot=20, mlp=None)], loop=(1, 4, 2))
ODD = plain.make_config([R(heads=5, dim=7, vdim=9, rot=6, base=300.0, mlp=plain.dense(21)),
                         LA(heads=6, dim=5, rot_dim=2, vdim=7, kv_rank=11, q_rank=9, base=50.0, scale=0.5, mlp=None),
                         A(heads=6, kv_heads=2, dim=14, vdim=6, rot=6, base=300.0, scale=0.4, mlp=plain.dense(50)),
                         A(heads=3, kv_heads=3, dim=9, vdim=66, rot=2, mlp=plain.dense(3)),
                         LA(heads=1, dim=18, rot_dim=34, vdim=3, kv_rank=50, q_rank=7, mlp=plain.dense(44)),
                         R(heads=3, dim=44, vdim=70, rot=10, mlp=None)], vocab=97, width=36, eps=1e-4, scale=0.5, softcap=6.0, loop=(2, 4, 3))
# (A read-out of one value is its sign behind the norm over its head, which any rounding can turn where it is close to zero: such
# heads are held to float32 accuracy alone, below.)
ONES = plain.make_config([A(heads=1, kv_heads=1, dim=2, vdim=1, rot=2, mlp=plain.dense(1)), LA(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=2, q_rank=2),
                          R(heads=1, dim=2, vdim=6, rot=2, decay=[1.0], mlp=None)], vocab=33, width=16, scale=1.0, loop=(0, 3, 1))
# sizes in whole 16-byte pieces, heads that the tensor-core kernels take
SQUARE = plain.make_config([A(heads=8, kv_heads=2, dim=64, vdim=64, rot=32, mlp=plain.dense(96)), LA(heads=8, dim=32, rot_dim=16, vdim=24, kv_rank=64, q_rank=40, mlp=plain.dense(256)),
                            R(heads=4, dim=32, vdim=64, rot=32, mlp=plain.dense(128)), LA(heads=40, dim=16, rot_dim=32, vdim=16, kv_rank=96, q_rank=64),
                            A(heads=4, kv_heads=4, dim=128, vdim=64, rot=128)], width=128, loop=(1, 4, 2))
CONFIGS = {"mixed": (MIXED, 16), "odd": (ODD, 8), "ones": (ONES, 4), "square": (SQUARE, 16)}


class Want:
    """Exact rows, and how far 16-bit activations move this model's logits on this prompt (worked out when first asked for): the
    largest of their own rounding and of three draws of random errors of the same size, since a small model may happen to be
    much touchier than one run shows."""

    def __init__(self, rows, noise):
        self.rows, self._noise = np.asarray(rows), noise

    @property
    def noise(self):
        if callable(self._noise):
            self._noise = self._noise()
        return self._noise

    def __getitem__(self, idx):
        return Want(self.rows[idx], lambda: self.noise)


def reference(w, cfg, toks):
    exact = plain.forward(w, cfg, toks)

    def noise():
        errs = []
        for draw in (None, 1, 2, 3):
            with plain.bfloat16_activations(draw):
                errs.append(rel_err(plain.forward(w, cfg, toks), exact))
        return max(errs)
    return Want(exact, noise)


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
        cfg, _ = CONFIGS[name]
        key = (name, tuple(toks))
        if key not in memo:
            memo[key] = reference(plain.random_weights(cfg, 5), cfg, toks)
        return memo[key]
    return get


# ---------------------------------------------------------------------------------------------- each mechanism alone

V60 = dict(vocab=60, width=48)
SINGLE = {
    "latent": plain.make_config([LA(mlp=None)], **V60),
    "latent_one_head_no_rotated_part": plain.make_config([LA(heads=1, rot_dim=0, mlp=None)], **V60),
    "latent_mostly_rotated": plain.make_config([LA(heads=4, dim=2, rot_dim=20, kv_rank=8, q_rank=30, base=100.0, mlp=None)], **V60),
    "latent_tensor_core_sizes": plain.make_config([LA(heads=4, dim=16, rot_dim=16, vdim=24, kv_rank=48, q_rank=16, mlp=None)], **V60),
    "latent_more_heads_than_a_tile_has_rows": plain.make_config([LA(heads=35, dim=8, rot_dim=16, vdim=8, kv_rank=32, q_rank=24, mlp=None)], **V60),
    "latent_three_heads_a_large_latent": plain.make_config([LA(heads=3, dim=32, rot_dim=32, vdim=40, kv_rank=288, q_rank=72, mlp=None)], **V60),
    "attention": plain.make_config([A(mlp=None)], **V60),
    "attention_one_kv_head": plain.make_config([A(heads=5, kv_heads=1, dim=10, vdim=10, rot=4, mlp=None)], **V60),
    "attention_a_kv_head_each_whole_head_rotated": plain.make_config([A(heads=3, kv_heads=3, dim=12, vdim=30, rot=12, mlp=None)], **V60),
    "attention_no_rotation": plain.make_config([A(rot=0, mlp=None)], **V60),
    "attention_heads_of_64": plain.make_config([A(heads=4, kv_heads=1, dim=64, vdim=64, rot=48, mlp=None)], **V60),
    "attention_values_smaller_than_keys": plain.make_config([A(heads=4, kv_heads=2, dim=128, vdim=40, rot=16, mlp=None)], **V60),
    "attention_values_larger_than_keys": plain.make_config([A(heads=4, kv_heads=2, dim=64, vdim=96, rot=16, mlp=None)], **V60),
    "attention_heads_of_256": plain.make_config([A(heads=2, kv_heads=1, dim=256, vdim=256, rot=16, mlp=None)], **V60),
    "retention": plain.make_config([R(mlp=None)], **V60),
    "retention_part_rotated": plain.make_config([R(heads=2, dim=40, vdim=300, rot=14, mlp=None), R(heads=7, dim=6, vdim=3, rot=2, decay=[0.0, 0.3, 0.5, 0.9, 0.99, 0.9999, 1.0], mlp=None)], **V60),
    "retention_aligned": plain.make_config([R(heads=4, dim=32, vdim=64, rot=16, mlp=None), R(heads=2, dim=128, vdim=128, rot=128, mlp=None)], **V60),
    "retention_no_rotation": plain.make_config([R(rot=0, mlp=None)], **V60),
    "retention_long_values": plain.make_config([R(heads=1, dim=16, vdim=640, rot=8, mlp=None)], **V60),
    "retention_values_of_one": plain.make_config([R(heads=2, dim=1, vdim=1, rot=0, mlp=None), R(heads=1, dim=2, vdim=1, rot=2, decay=[1.0], mlp=None)], **V60),
    "dense": plain.make_config([R(mlp=plain.dense(56)), R(mlp=plain.dense(64)), R(mlp=plain.dense(19))], **V60),
    "dense_wide": plain.make_config([R(mlp=plain.dense(1024))], vocab=60, width=256),
    "passes": plain.make_config([R(mlp=None), A(mlp=None), R(mlp=None)], loop=(0, 2, 3), **V60),
    "one_pass_of_the_last_layer": plain.make_config([R(mlp=None), LA(mlp=None)], loop=(1, 2, 1), **V60),
    "a_pass_behind_a_layer_with_both_halves": plain.make_config([R(), LA()], loop=(1, 2, 2), **V60),
    "no_cap": plain.make_config([R()], softcap=None, **V60),
    "odd_width": plain.make_config([A(heads=2, kv_heads=1, dim=6, vdim=5, rot=2, mlp=plain.dense(19)), LA(heads=2, dim=3, rot_dim=4, vdim=5, kv_rank=9, q_rank=5), R(heads=2, dim=5, vdim=3, rot=4)],
                                   vocab=51, width=38, eps=1e-3),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SINGLE))
def test_each_mechanism_alone(tmp_path, name, dtype):
    cfg = SINGLE[name]
    if name == "retention_values_of_one" and dtype == "bfloat16":
        return
    w = plain.random_weights(cfg, 3)
    toks = tokens_of(cfg, 61, 1)
    want = reference(w, cfg, toks)
    hs = Harness(tmp_path, cfg, w, dtype)
    close(hs.whole("a", toks), want, dtype, name)
    close(hs.in_portions("b", toks, [30, 2] + [1] * 40), want, dtype, f"{name}, a portion, two tokens, then decoded")


# ---------------------------------------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_decoding_and_portions(tmp_path, truth, name, dtype):
    """The same logits at every position whether the prompt comes whole, token by token from the first token on (states
    that start empty), or in portions of several sizes down to two."""
    cfg, page = CONFIGS[name]
    w = plain.random_weights(cfg, 5)
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
    cfg, page = CONFIGS[name]
    w = plain.random_weights(cfg, 5)
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


# ---------------------------------------------------------------------------------------------- what random weights would hide

MARK, QUIET = 7, 0.4


def _one_token_stands_out(w, cfg):
    """Column `mark` of the embedding is zero but for token MARK, column `const` is one number for every token: behind the first
    norm (its weight one) the first is a large entry for the marked token and a small one for the others, the second about the
    same for all. Returns the two columns."""
    mark, const = cfg["width"] - 2, cfg["width"] - 1
    emb = w["embed"].astype(np.float64) * QUIET
    emb[:, mark], emb[:, const] = 0.0, 1.0
    emb[MARK, mark] = 3.0
    w["embed"] = plain.round_bf16(emb)
    w["l0.norm1"][:] = 0.0
    return mark, const


def _marked_tokens(cfg, n, at, seed):
    toks = [t if t != MARK else MARK + 1 for t in tokens_of(cfg, n, seed)]
    toks[at] = MARK
    other = list(toks)
    other[at] = MARK + 2
    return toks, other


def _peaked(kind, geometry, at, n):
    """One layer in which the key of the token at place `at` outweighs all other keys together for every later query. (What carries
    it is not rotated, so the distance does not matter.)"""
    if kind == "attention":
        dim, vdim, heads, kv_heads = geometry
        cfg = plain.make_config([A(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=dim // 4 * 2, scale=1.0, mlp=None)], vocab=40, width=32, scale=1.0)
    else:
        dim, rd, vdim, heads, rank, q_rank = geometry
        cfg = plain.make_config([LA(heads=heads, dim=dim, rot_dim=rd, vdim=vdim, kv_rank=rank, q_rank=q_rank, scale=1.0, mlp=None)], vocab=40, width=32, scale=1.0)
    w = plain.random_weights(cfg, 8, sharp=1.0)
    mark, const = _one_token_stands_out(w, cfg)
    p = "l0.mix."
    if kind == "attention":
        for leaf, count in (("q", heads), ("k", kv_heads)):
            w[p + leaf] = plain.round_bf16(w[p + leaf] * 0.2)
            w[p + leaf + ".norm"][:] = plain.round_bf16(4.0 / dim ** 0.5 if leaf == "k" else 3.0 / dim ** 0.5)
            for h in range(count):
                w[p + leaf][h * dim + dim - 1] = 0.0
                w[p + leaf][h * dim + dim - 1, const if leaf == "q" else mark] = 4.0
    else:
        for leaf in ("dq", "dkv"):
            w[p + leaf] = plain.round_bf16(w[p + leaf] * 0.3)
            w[p + leaf][0] = 0.0
            w[p + leaf][0, const if leaf == "dq" else mark] = 4.0
            w[p + leaf + ".norm"][:] = 1.0
        w[p + "uq"], w[p + "uk"] = plain.round_bf16(w[p + "uq"] * 0.3), plain.round_bf16(w[p + "uk"] * 0.3)
        for h in range(heads):      # the first unrotated dimension of every head: a constant in q, the marked token's channel in k
            w[p + "uq"][h * (dim + rd)], w[p + "uk"][h * dim] = 0.0, 0.0
            w[p + "uq"][h * (dim + rd), 0], w[p + "uk"][h * dim, 0] = plain.round_bf16(5.0 / q_rank ** 0.5), plain.round_bf16(5.0 / rank ** 0.5)
        w[p + "sink"][:] = plain.round_bf16(np.linspace(-1.0, 2.0, heads))
    return (cfg, w) + _marked_tokens(cfg, n, at, 4)


FAR = [("attention", (16, 12, 4, 2), 8), ("attention", (64, 64, 4, 1), 16), ("attention", (128, 48, 8, 4), 8),
       ("latent", (6, 4, 5, 3, 12, 10), 8), ("latent", (16, 16, 24, 4, 48, 24), 16), ("latent", (8, 16, 8, 34, 32, 16), 8)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,geometry,page", FAR)
@pytest.mark.parametrize("at", [0, 15, 16])
def test_a_key_hundreds_back_at_a_pages_border(tmp_path, dtype, kind, geometry, page, at):
    """A key that carries the softmax of every later row, on the sequence's first place, a page's last and a page's first: in a
    prompt, in portions, and decoded through splits. The rows ahead of it do not see it."""
    n = 330
    cfg, w, toks, other = _peaked(kind, geometry, at, n)
    ref, moved = reference(w, cfg, toks), plain.forward(w, cfg, other)
    assert rel_err(moved[at + 1:], ref.rows[at + 1:]) > 0.15 and min(rel_err(moved[[i]], ref.rows[[i]]) for i in (at + 1, n - 1)) > 0.1
    assert at == 0 or rel_err(moved[:at], ref.rows[:at]) < 1e-9
    hs = Harness(tmp_path, cfg, w, dtype, page=page, pages=2 * 336 // page)
    close(hs.whole("w", toks), ref, dtype, "whole")
    close(hs.in_portions("p", toks, [at + 1, 2, 90, 17, 2, n]), ref, dtype, "in portions")
    close(hs.in_portions("d", toks, [290] + [1] * 40), ref, dtype, "decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,geometry,page", [FAR[0], FAR[1], FAR[3], FAR[4]])
def test_many_splits_of_a_long_context(tmp_path, dtype, kind, geometry, page):
    """Single rows over a context that is cut into several splits: each key, and a sink, counts once."""
    n = 1250
    cfg, w, toks, _ = _peaked(kind, geometry, 601, n)
    ref = reference(w, cfg, toks)
    hs = Harness(tmp_path, cfg, w, dtype, page=page, pages=n // page + 2, max_tokens=n)
    rows = hs.step([("d", toks[:n - 25], range(n - 60, n - 25))])
    for i in range(n - 25, n):
        rows.update(hs.step([("d", toks[i:i + 1], [0])]))
    close(np.stack([rows[("d", i)] for i in range(n - 60, n)]), ref[n - 60:], dtype, "prompt, then decoded through splits")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("geometry", [(6, 4, 5, 3, 12, 10), (16, 16, 24, 4, 48, 24), (8, 16, 8, 34, 32, 16)])
def test_the_sink_counts_once_and_unscaled(tmp_path, dtype, geometry):
    """Scores near zero and sinks that are worth as much as all keys together: without the sink, with the sink scaled like a score,
    or with it counted twice, every row would be visibly another one."""
    dim, rd, vdim, heads, rank, q_rank = geometry
    cfg = plain.make_config([LA(heads=heads, dim=dim, rot_dim=rd, vdim=vdim, kv_rank=rank, q_rank=q_rank, scale=0.02, mlp=None)], vocab=40, width=32, scale=1.0)
    w = plain.random_weights(cfg, 6, sharp=1.0)
    w["l0.mix.o"] = plain.round_bf16(w["l0.mix.o"] * 6.0)
    w["l0.mix.sink"][:] = plain.round_bf16(np.linspace(4.0, 6.0, heads))
    toks = tokens_of(cfg, 330, 5)
    ref = reference(w, cfg, toks)
    for change in (lambda s: np.full_like(s, -80.0), lambda s: 0.02 * s, lambda s: s + np.float32(np.log(2.0))):
        moved = plain.forward({k: (change(v) if k.endswith("sink") else v) for k, v in w.items()}, cfg, toks)
        assert rel_err(moved[60:], ref.rows[60:]) > 0.05
    hs = Harness(tmp_path, cfg, w, dtype)
    close(hs.whole("w", toks), ref, dtype, "whole")
    close(hs.in_portions("d", toks, [1, 2, 250] + [1] * 80), ref, dtype, "first tokens, a portion, then decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(2, 12, 12, 4), (2, 64, 32, 32)])
def test_a_state_remembers_a_token_hundreds_back(tmp_path, dtype, sizes):
    """The state is carried through a prompt portion, through another, and through decoding, and a second request in another
    slot in between does not touch it. What the marked token wrote still decides the last rows."""
    heads, dim, vdim, rot = sizes
    cfg = plain.make_config([R(heads=heads, dim=dim, vdim=vdim, rot=rot, decay=[0.9995, 0.999], mlp=None)], vocab=40, width=32, scale=1.0)
    w = plain.random_weights(cfg, 11)
    mark, const = _one_token_stands_out(w, cfg)
    for leaf, col in (("q", const), ("k", mark)):      # along what is not rotated
        w["l0.mix." + leaf] = plain.round_bf16(w["l0.mix." + leaf] * 0.1)
        for h in range(heads):
            w["l0.mix." + leaf][h * dim + rot:(h + 1) * dim, col] = 4.0
    w["l0.mix.o"] = plain.round_bf16(w["l0.mix.o"] * 3.0)
    toks, other = _marked_tokens(cfg, 400, 3, 12)
    want, moved = reference(w, cfg, toks), plain.forward(w, cfg, other)
    assert rel_err(moved[-5:], want.rows[-5:]) > 0.1
    hs = Harness(tmp_path, cfg, w, dtype, pages=64, max_tokens=512)
    close(hs.whole("w", toks), want, dtype, "whole")
    rows = hs.step([("a", toks[:130], range(130))])
    rows.update(hs.step([("x", other[:77], [])]))                       # another request takes another slot
    rows.update(hs.step([("a", toks[130:300], range(170)), ("x", other[77:78], [])]))
    for i in range(300, 400):
        rows.update(hs.step([("a", toks[i:i + 1], [0])] + ([("x", other[78 + i - 300:79 + i - 300], [])] if i % 2 else [])))
    close(np.stack([rows[("a", i)] for i in range(400)]), want, dtype, "portions, then decoding beside another request")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_captured_steps_and_slots_used_again(tmp_path, truth, dtype):
    """Three requests decode together for 200 steps (steps of one token each are captured as graphs and replayed), end at
    different times, and a fourth takes over a slot and pages that were just given back."""
    cfg, page = CONFIGS["mixed"]
    w = plain.random_weights(cfg, 5)
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
    cfg, page = CONFIGS["mixed"]
    w = plain.random_weights(cfg, 5)
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
    cfg, page = CONFIGS["odd"]
    w = plain.random_weights(cfg, 5)
    plain.write_model_dir(tmp_path, cfg, w)
    prompt = tokens_of(cfg, 21, 77)
    assert main(["generate", "-m", str(tmp_path), "-p", " ".join(map(str, prompt)), "--temp", "0", "--max-tokens", "12",
                 "--dtype", "float32", "--kv-mem", "64M", "--max-tokens-per-step", "8", "--max-seqs", "2"]) == 0
    assert [int(t) for t in capsys.readouterr().out.split()] == plain.generate(w, cfg, prompt, 12)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_of_a_sebalorn_model(tmp_path, truth, dtype):
    from test_replay_gpu import Replay
    cfg, page = CONFIGS["odd"]
    w = plain.random_weights(cfg, 5)
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
    layers = []
    for i in range(int(r.integers(2, 6))):
        mlp = pick(None, plain.dense(pick(8, 24, 50, 64, 160)), plain.dense(pick(72, 33)))
        kind = pick("latent", "latent", "attention", "retention")
        base = pick(100.0, 1e4, 5e5)
        if kind == "latent":
            layers.append(LA(heads=pick(1, 2, 4, 7), dim=pick(16, 32) if aligned else pick(1, 6, 20), rot_dim=pick(16, 32) if aligned else pick(2, 6, 24),
                             vdim=pick(16, 64) if aligned else pick(3, 10, 36), kv_rank=pick(16, 80, 144) if aligned else pick(4, 13, 40, 100),
                             q_rank=pick(16, 64) if aligned else pick(3, 12, 50), base=base, scale=pick(None, 0.3), mlp=mlp))
        elif kind == "attention":
            kv, dim = pick(1, 2, 3), pick(64, 128) if aligned else pick(4, 10, 20, 48)
            layers.append(A(heads=kv * pick(1, 2, 4), kv_heads=kv, dim=dim, vdim=pick(dim, dim // 2, 80) if aligned else pick(3, 16, dim), rot=pick(0, 2, dim // 4 * 2, dim // 2 * 2),
                            base=base, scale=pick(None, 0.3), mlp=mlp))
        else:
            heads, dim = pick(1, 2, 5), pick(16, 32) if aligned else pick(3, 8, 20, 40)
            layers.append(R(heads=heads, dim=dim, vdim=pick(16, 64) if aligned else pick(3, 10, 36), rot=pick(2, dim // 4 * 2, dim // 2 * 2), base=base,
                            decay=r.uniform(0.3, 0.9999, heads).tolist(), mlp=mlp))
    start = int(r.integers(0, len(layers)))
    loop = None if r.random() < 0.3 else (start, int(r.integers(start + 1, len(layers) + 1)), pick(1, 2, 3))
    cfg = plain.make_config(layers, vocab=pick(33, 97, 160, 301), width=pick(24, 36, 64, 72, 128), eps=pick(1e-6, 1e-5, 1e-3), scale=pick(0.7, 1.0, 8.0),
                            softcap=pick(5.0, 30.0), loop=loop)
    return cfg, pick(4, 8, 16, 32)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(15))
def test_configurations_drawn_at_random(tmp_path, seed, dtype):
    cfg, page = _random_config(seed)
    w = plain.random_weights(cfg, 100 + seed)
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

def _draw(seed):
    g = torch.Generator(device="cuda").manual_seed(seed)
    return lambda *shape: torch.randn(*shape, device="cuda", generator=g)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D", [50, 320, 5000])
def test_the_rms_norm_adds_up_to_four_terms_in_float(dtype, D):
    from tiny_inference_engine_b200 import ops
    draw, T = _draw(1), 37
    x, a, b, part, w = draw(T, D), draw(T, D).to(dtype), draw(T, D).to(dtype), draw(3, T, D), draw(D)
    terms = ops.ScaledSum([(a, 1.0), (ops.SplitSum(part.reshape(-1), 3, T, D), 0.9), (b, 1.0), (a, -0.25)])
    want_x = x.double() + 0.75 * a.double() + 0.9 * part.double().sum(0) + b.double()
    norm = lambda v: v / ((v ** 2).mean(-1, keepdim=True) + 1e-3).sqrt() * w.double()
    tol = 2e-5 if dtype == torch.float32 else 6e-2
    out, x1 = torch.empty(T, D, device="cuda", dtype=dtype), x.clone()
    ops.add_terms_rmsnorm(x1, terms, w, 1e-3, out)
    assert (x1.double() - want_x).abs().max() < 1e-5 and (out.double() - norm(want_x)).abs().max() < tol
    rows = torch.tensor([5, 0, 36], device="cuda", dtype=torch.int32)
    x2, some = x.clone(), torch.empty(3, D, device="cuda", dtype=dtype)
    ops.add_terms_rmsnorm(x2, terms, w, 1e-3, some, rows=rows)
    assert torch.equal(x2, x)            # with rows the stream stays as it is
    assert (some.double() - norm(want_x)[rows.long()]).abs().max() < tol


@pytest.mark.parametrize("T,N,K", [(1, 256, 512), (8, 6144, 2048), (8, 96, 64), (40, 384, 1024), (100, 256, 4096), (130, 1024, 192), (300, 100, 72), (700, 3072, 256), (1024, 8224, 128)])
def test_the_squared_relu_in_a_products_epilogue(T, N, K):
    """Every tiling: tokens on the narrow side with k whole or in splits, 128-row tiles, pairs of SMs."""
    from tiny_inference_engine_b200 import ops
    draw = _draw(T)
    a, w = draw(T, K).to(torch.bfloat16), (draw(N, K) / K ** 0.5).to(torch.bfloat16)
    want = torch.relu(a.double() @ w.double().t()) ** 2
    out = torch.full((T, N), float("nan"), device="cuda", dtype=torch.bfloat16)
    ops.bound_gemm(w, silu=ops.SQUARED_RELU)(a, out)
    assert ((out.double() - want).abs() <= 1e-2 * want + 1e-4).all()
    f32 = torch.full((T, N), float("nan"), device="cuda")
    ops.bound_gemm(w, silu=ops.SQUARED_RELU)(a, f32)
    assert ((f32.double() - want).abs() <= 2e-4 * want + 1e-5).all()
    # operands that only the CUDA cores take, and float32
    for dtype, tol in ((torch.bfloat16, 2e-2), (torch.float32, 2e-5)):
        a2, w2 = draw(9, 37).to(dtype), draw(33, 37).to(dtype)
        o2 = torch.empty(9, 33, device="cuda", dtype=dtype)
        ops.bound_gemm(w2, silu=ops.SQUARED_RELU)(a2, o2)
        ref = torch.relu(a2.double() @ w2.double().t()) ** 2
        assert ((o2.double() - ref).abs() <= tol * ref + tol).all()


def _rotations(theta, rot):
    from tiny_inference_engine_b200.config.spec import PartSpec
    from tiny_inference_engine_b200.parts import build_part
    for pairing in ("halves", "neighbours"):
        for angles in ("float32", "float64"):
            part = build_part("position", PartSpec("rope", {"theta": theta, "head_dim": max(rot, 2), "rotary_dim": rot, "pairing": pairing, "angles": angles}), torch.float32)
            yield part, (plain.rotate_neighbours if pairing == "neighbours" else plain.rotate_halves), (3e-6 if angles == "float64" else 2e-2)


POSITIONS = [0, 1, 777, 100003]


@pytest.mark.parametrize("dim,rot", [(16, 10), (16, 16), (32, 8), (6, 2)])
def test_rotations_in_both_pairings_and_at_large_positions(dim, rot):
    """q and k of rope_split (k times a factor), rope in place, and the step ahead of grouped-query attention: dimensions past the
    rotated ones pass. Angles in double keep their precision at position 100,003; float products lose some."""
    from tiny_inference_engine_b200 import ops
    draw, H, nv = _draw(3), 3, 20
    pos = torch.tensor(POSITIONS, device="cuda", dtype=torch.int32)
    q_off, k_off, v_off = 0, 96, 192
    proj = draw(4, 232)
    section = lambda off, n: proj[:, off:off + n].double().cpu().numpy()
    for part, rotate, tol in _rotations(50.0, rot):
        table, neighbours = part.rotation()
        want_q = rotate(section(q_off, H * dim).reshape(4, H, dim), POSITIONS, 50.0, rot)
        want_k = rotate(section(k_off, H * dim).reshape(4, H, dim), POSITIONS, 50.0, rot)
        qn, kn, vn = torch.empty(4, H * dim, device="cuda"), torch.empty(4, H * dim, device="cuda"), torch.empty(4, nv, device="cuda")
        ops.rope_split(proj, q_off, k_off, v_off, H, dim, table, pos, 0.5, qn, kn, vn, neighbours)
        assert np.abs(qn.cpu().numpy().reshape(4, H, dim) - want_q).max() < tol
        assert np.abs(kn.cpu().numpy().reshape(4, H, dim) - 0.5 * want_k).max() < tol
        assert torch.equal(vn, proj[:, v_off:v_off + nv])
        x = proj[:, :H * dim].clone()
        part.apply(x, pos, H, dim)
        assert np.abs(x.cpu().numpy().reshape(4, H, dim) - want_q).max() < tol
        y, kc, vc = proj.clone(), torch.zeros(1, H, 8, dim, device="cuda"), torch.zeros(1, H, 8, 4, device="cuda")
        ops.qkv_span_prep(y, q_off, k_off, v_off, None, None, None, None, None, 1e-6, table, pos, torch.arange(4, device="cuda", dtype=torch.int32), kc, vc,
                          H, H, dim, 4, neighbours=neighbours)
        assert np.abs(y[:, :H * dim].cpu().numpy().reshape(4, H, dim) - want_q).max() < tol
        assert np.abs(kc[0, :, :4].permute(1, 0, 2).cpu().numpy() - want_k).max() < tol


def test_the_latents_rotated_parts_in_both_pairings():
    from tiny_inference_engine_b200 import ops
    draw, rank, rot, q_rank, H, dim = _draw(4), 12, 10, 8, 3, 5
    pos = torch.tensor(POSITIONS, device="cuda", dtype=torch.int32)
    proj, q = draw(4, 40), draw(4, H * (dim + rot))
    ones = torch.ones(64, device="cuda")
    for part, rotate, tol in _rotations(50.0, rot):
        table, neighbours = part.rotation()
        cq, kc, folded = torch.empty(4, q_rank, device="cuda"), torch.zeros(1, 1, 8, rank + rot, device="cuda"), torch.zeros(4, H * (rank + rot), device="cuda")
        ops.latent_prep(proj, 0, q_rank, 8, rank, rot, ones[:q_rank], ones[:rank], 1e-6, table, pos, torch.arange(4, device="cuda", dtype=torch.int32), cq, kc, neighbours)
        ops.latent_query_rot(q, dim, rot, table, pos, folded, rank, H, neighbours)
        want = rotate(proj[:, 8 + rank:8 + rank + rot].double().cpu().numpy()[:, None], POSITIONS, 50.0, rot)[:, 0]
        assert np.abs(kc[0, 0, :4, rank:].cpu().numpy() - want).max() < tol
        assert np.abs(kc[0, 0, :4, :rank].cpu().numpy() - plain.unit_rms(proj[:, 8:8 + rank].cpu().numpy(), 1e-6)).max() < 1e-5
        want = rotate(q.double().cpu().numpy().reshape(4, H, dim + rot)[:, :, dim:], POSITIONS, 50.0, rot)
        assert np.abs(folded.cpu().numpy().reshape(4, H, rank + rot)[:, :, rank:] - want).max() < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,vdim", [(3, 20), (4, 64), (2, 640), (1, 7)])
def test_heads_normed_without_a_weight_and_gated(dtype, H, vdim):
    from tiny_inference_engine_b200 import ops
    draw, T = _draw(5), 21
    o, wide = draw(T, H * vdim), draw(T, H * vdim + 16).to(dtype)
    gate, out = wide[:, 8:8 + H * vdim], torch.empty(T, H * vdim, device="cuda", dtype=dtype)
    unit = (o.view(T, H, vdim).double() / ((o.view(T, H, vdim).double() ** 2).mean(-1, keepdim=True) + 1e-4).sqrt()).view(T, -1)
    tol = 1e-5 if dtype == torch.float32 else 3e-2
    for act, f in ((ops.GATE_SILU, torch.nn.functional.silu), (ops.GATE_SIGMOID, torch.sigmoid)):
        ops.head_norm_gate(o, gate, None, 1e-4, out, H, vdim, act)
        assert (out.double() - unit * f(gate.double())).abs().max() < tol
    y = draw(T, H * vdim).to(dtype)
    want = y.double() * torch.sigmoid(wide[:, :H].double()).repeat_interleave(vdim, dim=1)
    ops.head_gate_mul(y, wide[:, :H], H, vdim)
    assert (y.double() - want).abs().max() < tol
