"""Grouped-query attention whose values are its keys, in a window beside which the first tokens stay visible:

    q, k   = h Wq^T + bq, h Wk^T + bk                       one product, the weights stacked (`qk_bias`)
    q, k   = conv(q), conv(k)                               a short causal convolution over time per channel (`conv_taps`)
    v      = k                                              as it leaves the convolution, before the rotation
    q, k   = pairs (2i, 2i+1) of the first `rotary_dim` dimensions of each head turned by position * theta^(-2i/rotary_dim)
    k, v  -> cache pages
    s      = scale * q . k;  s <- cap * tanh(s / cap)       (`softcap`, 0: none)
    p      = exp(s) / (exp(sink_h) + sum exp(s))            over j <= i with i - j < window or j < keep_first; `sink`: a learned
                                                            number per head, neither scaled nor capped, without a key or value
    out    = (p v) Wo^T

Every size and constant is a parameter and each option can be left out (`window` 0: every j <= i). The convolution's last
`conv_taps - 1` inputs (with their bias) are a request's state, float32; the kept tokens' pages stay in the cache beside the
window's. Convolution, angles (double), scores, cap, softmax and sink are float32 whatever the compute dtype; on the tensor
cores the softmax weights enter the value product as two bfloat16 terms.
"""
from __future__ import annotations

import math

import torch

from .. import ops
from ..errors import InvalidArgument
from ..weights.loader import TensorNeed
from .attention import MAX_SPLITS, NUM_SMS, TMA_DECODE_TABLE_ENTRIES, decode_splits
from .base import CacheNeed, Mixer, StateNeed, build_part, register_part, to_compute


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


class ConvKeyAttention(Mixer):
    launches_only = False
    graph_safe = True       # the kernels read the step from device tensors only and skip sequences without a slot

    def __init__(self, spec, dtype, prefix: str = ""):
        p = spec.params
        self.prefix = prefix + p.get("prefix", "")
        self.hidden = int(p["hidden_size"])
        self.heads, self.kv_heads, self.dim = int(p["num_heads"]), int(p["num_kv_heads"]), int(p["head_dim"])
        self.scale = float(p["scale"]) if p.get("scale") is not None else 1.0 / math.sqrt(self.dim)
        self.window = int(p.get("window") or 0)
        self.keep_first = int(p.get("keep_first") or 0) if self.window > 0 else 0
        self.softcap = float(p.get("softcap") or 0.0)
        self.taps = int(p.get("conv_taps", 1))
        self.has_bias, self.has_sink = bool(p.get("qk_bias", False)), bool(p.get("sink", False))
        if self.heads <= 0 or self.kv_heads <= 0 or self.heads % self.kv_heads:
            raise InvalidArgument(f"{self.heads} heads are not a multiple of {self.kv_heads} kv heads")
        if self.dim <= 0 or not 1 <= self.taps <= 16 or self.window < 0 or self.keep_first < 0 or self.softcap < 0:
            raise InvalidArgument(f"attention: bad sizes dim={self.dim} taps={self.taps} (1 to 16) window={self.window} kept={self.keep_first}")
        self.dtype = dtype
        self.position = build_part("position", p["position"], dtype, prefix=self.prefix) if p.get("position") else None
        if self.position is not None:
            self.scale *= float(self.position.score_scale())
        self.q_dim, self.k_dim = self.heads * self.dim, self.kv_heads * self.dim
        self.k_off = _up8(self.q_dim)                   # columns of the stacked product
        self.channels = self.k_off + self.k_dim         # what the convolution's kernels walk: q, (padding,) k
        self.width = self.k_off + _up8(self.k_dim)
        self.sink = None

    def _name(self, leaf):
        return self.prefix + leaf

    def needs(self):
        D, n = self.hidden, self._name
        t = {n("q"): TensorNeed((self.q_dim, D)), n("k"): TensorNeed((self.k_dim, D)), n("o"): TensorNeed((D, self.q_dim)),
             n("q.conv"): TensorNeed((self.q_dim, self.taps)), n("k.conv"): TensorNeed((self.k_dim, self.taps))}
        if self.has_bias:
            t.update({n("q.b"): TensorNeed((self.q_dim,), "norm"), n("k.b"): TensorNeed((self.k_dim,), "norm")})
        if self.has_sink:
            t[n("sink")] = TensorNeed((self.heads,), "norm")
        if self.position is not None:
            t.update(self.position.needs())
        return t

    def bind(self, get):
        n = self._name
        device = get(n("q")).device
        stacked = torch.zeros((self.width, self.hidden), dtype=self.dtype, device=device)
        conv = torch.zeros((self.taps, self.channels), dtype=torch.float32, device=device)      # a tap of every channel side by side
        bias = torch.zeros(self.channels, dtype=torch.float32, device=device) if self.has_bias else None
        for leaf, off, rows in (("q", 0, self.q_dim), ("k", self.k_off, self.k_dim)):
            stacked[off:off + rows] = to_compute(get(n(leaf)), self.dtype)
            conv[:, off:off + rows] = get(n(leaf + ".conv")).to(torch.float32).t()
            if self.has_bias:
                bias[off:off + rows] = get(n(leaf + ".b")).to(torch.float32)
        self.gemm_in = ops.bound_gemm(stacked, split_many=False)
        self.w_in = self.gemm_in.w
        self.conv_w, self.bias = conv, bias
        self.gemm_o = ops.bound_gemm(to_compute(get(n("o")), self.dtype).contiguous(), split_many=True)
        self.w_o = self.gemm_o.w
        self.sink = get(n("sink")).to(torch.float32).contiguous() if self.has_sink else None
        if self.position is not None:
            self.position.bind(get)
        self._capacity = None

    def cache_need(self):
        return CacheNeed("window" if self.window > 0 else "full", self.kv_heads, self.dim, self.window, keep_first=self.keep_first)

    def state_need(self):
        return StateNeed(((self.taps - 1) * self.channels,), torch.float32) if self.taps > 1 else None

    def forward(self, h, ctx, cache, state):
        T, H, G, dim = h.shape[0], self.heads, self.kv_heads, self.dim
        g = ctx.groups[cache.group]
        if not cache.writes:
            raise InvalidArgument("this attention computes its own keys and values: it cannot read another entry's cache")
        if self.taps > 1 and state is None:
            raise InvalidArgument("a convolution over time needs state slots (make the cache with `make_cache`)")
        proj = ctx.ws.rows("cattn.proj", T, self.width, self.dtype)
        self.gemm_in(h, proj)
        turns = None
        if self.position is not None and not self.position.is_identity:
            if not hasattr(self.position, "turns_table"):
                raise InvalidArgument("this attention takes a rotation by a table of frequencies (or none) as its position encoding")
            turns = self.position.turns_table()
        q = ctx.ws.rows("cattn.q", T, self.q_dim, self.dtype)
        ops.conv_rope_append(proj, 0, self.k_off, self.conv_w, self.bias, state, 0, ctx, turns, g.slots, cache.k, cache.v, q, H, G, dim)
        attn = ctx.ws.rows("cattn.out", T, self.q_dim, self.dtype)
        options = dict(window=self.window, keep_first=self.keep_first, softcap=self.softcap, sink=self.sink)
        index = (ctx.query_start, ctx.context_lens, g.block_tables)
        tensor_cores = ops.attention_decode_tma_takes(q, H, G, dim, cache.k.shape[2])
        n = ctx.multi_rows
        if n > 0 and tensor_cores:
            ops.attention_prompt_kept(q, cache.k, cache.v, attn, *index, ctx.multi_seqs, ctx.multi_max_queries, H, G, dim, self.scale, **options)
        elif n > 0:
            ops.attention_kept_rows(q[:n], cache.k, cache.v, attn[:n], ctx.seq_of_row[:n], *index, H, G, dim, dim, self.scale, **options)
        if ctx.single_count > 0:
            self._attend_single(q, attn, ctx, g, cache, index, options, tensor_cores)
        out = ctx.ws.rows("cattn.mixed", T, self.hidden, self.dtype)
        if self._capacity is None:
            self._capacity = ops.partial_capacity(ctx.ws.max_rows, self.gemm_o.N, self.gemm_o.K)
        return self.gemm_o(attn, out, lambda m: ctx.ws.flat("cattn.mixed.partial", m, torch.float32, self._capacity))

    def _attend_single(self, q, attn, ctx, g, cache, index, options, tensor_cores):
        """Sequences that bring one token: the keys they see in splits (on the tensor cores the kept keys come on top of the
        first split's own)."""
        H, G, dim, page, n = self.heads, self.kv_heads, self.dim, cache.k.shape[2], ctx.single_count
        longest = ctx.single_max_context if self.window <= 0 else min(ctx.single_max_context, self.window)
        kept_tiles = -(-self.keep_first // 64)
        cap = (TMA_DECODE_TABLE_ENTRIES // (64 // min(page, 64)) - 1 - kept_tiles) * 64      # what the kernel's table of pages holds
        if tensor_cores and cap >= 64:
            split_keys, max_splits = decode_splits(longest, n, G, page, ctx.single_contexts if self.window <= 0 else None)
            if split_keys > cap:
                split_keys, max_splits = cap, max(1, -(-longest // cap))
            if max_splits <= MAX_SPLITS:
                scratch = ctx.ws.flat("attn.split", ops.attention_split_scratch_floats(ctx.max_seqs, H, dim, MAX_SPLITS), torch.float32)
                counters = ctx.ws.zeros("attn.counters", ctx.max_seqs * G, torch.int32)
                cluster = max_splits in ops.CLUSTER_SPLITS and n * G * max_splits <= 2 * NUM_SMS
                ops.attention_decode_kept(q, cache.k, cache.v, attn, *index, H, G, dim, self.scale, ctx.multi_seqs, n, split_keys, max_splits,
                                          scratch, counters, cluster=cluster, **options)
                return
        longest += self.keep_first
        # splits enough to fill the SMs a few times over, none shorter than 32 keys; a row's sums depend on the batch by their order only
        want = max(1, (4 * NUM_SMS) // max(1, n * G))
        split_keys = max(32, -(-math.ceil(longest / want) // 32) * 32)
        while math.ceil(longest / split_keys) > MAX_SPLITS:
            split_keys *= 2
        max_splits = max(1, math.ceil(longest / split_keys))
        scratch = ctx.ws.flat("cattn.split", ops.attention_split_scratch_floats(ctx.max_seqs, H, dim, MAX_SPLITS), torch.float32)
        ops.attention_kept_split(q, cache.k, cache.v, attn, *index, H, G, dim, dim, self.scale, ctx.single_seqs, n, split_keys, max_splits,
                                 scratch, **options)


register_part("mixer", "conv_key_attention", ConvKeyAttention, replace=True)
