"""A plain, slow Vurazen in numpy: whole sequences, no cache, no state carried between calls, one function per mechanism.
Arithmetic is float64 on the stored values. Nothing here imports the engine package: the tests compare the two.

A Vurazen model lists its layers in any order. A layer has ONE norm (mean and variance, weight and bias), whose output
both its sublayers read: x <- x + (mixer(norm x) + ff(norm x)); a layer may have no feed-forward. Layers start .. stop-1
may run several times in a row with the same weights; ahead of every pass but the first the embedding's output joins the
stream again, and ahead of every pass a vector of that pass does. Mixers:

  mamba1      a selective scan: a diagonal state per channel whose decay depends on the token, behind a short convolution;
  parallel    two mixers on the same input, summed with one factor each. Left: attention whose queries and keys pass a
              short convolution, whose values are the unrotated keys, in a window beside which the first tokens stay
              visible, with capped scores and a learned sink per head. Right: a delta rule with a decay per key channel;
  lightning   linear attention with a constant decay per head and one norm over all heads.

Feed-forwards: `dense` (relu(gate) * up) and `moe` (the `top` largest router logits, softmax over those alone, clamped
experts, and a shared expert for every token). The logits are capped.
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np

EXPERT_SLOPE = 1.702
UNIT_EPS = 1e-6


# --------------------------------------------------------------------------- small functions

def f64(a):
    return np.asarray(a, dtype=np.float64)


def sigmoid(z):
    z = f64(z)
    return np.exp(np.minimum(z, 0.0)) / (1.0 + np.exp(-np.abs(z)))


def softplus(z):
    return np.logaddexp(0.0, z)


def silu(z):
    return z * sigmoid(z)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    x = f64(x)
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def capped(s, cap):
    return s if not cap else cap * np.tanh(s / cap)


def round_bf16(x):
    a = np.ascontiguousarray(x, dtype=np.float32)
    bits = a.view(np.uint32).astype(np.uint64)
    rounded = ((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16) << 16
    return rounded.astype(np.uint32).view(np.float32).reshape(np.shape(x))


_act = None       # with `bfloat16_activations()`: rounds what a 16-bit pipeline would keep in 16 bits


class bfloat16_activations:
    """Within this context the outputs of `linear`, of the norms and of other steps that feed a matrix product are rounded
    to bfloat16 (the weights of the tests are bfloat16 values already): the distance to the exact result is the noise that
    a pipeline with 16-bit activations cannot avoid, which is what a tolerance for such a pipeline is measured against."""

    def __enter__(self):
        global _act
        _act = lambda y: round_bf16(y).astype(np.float64)

    def __exit__(self, *exc):
        global _act
        _act = None


def kept(y):
    return y if _act is None else _act(y)


def linear(x, w, b=None):
    y = f64(x) @ f64(w).T
    return kept(y if b is None else y + f64(b))


def layer_norm(x, w, name, eps):
    """(x - mean) / sqrt(mean of squared deviations + eps) * weight + bias (`<name>.b`)."""
    x = f64(x)
    d = x - x.mean(axis=-1, keepdims=True)
    return kept(d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * f64(w[name]) + f64(w[name + ".b"]))


def short_conv(u, taps, bias=None):
    """Causal convolution over time per channel: y_t = sum_j taps[:, j] u_(t - n + 1 + j), zeros before the start."""
    u, taps = f64(u), f64(taps)
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, u.shape[1])), u], axis=0)
    y = sum(taps[:, j][None, :] * padded[j:j + u.shape[0]] for j in range(n))
    return y if bias is None else y + f64(bias)


# --------------------------------------------------------------------------- the selective scan

def selective_scan(x, dt, A, B, C, D):
    """S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;  y_c = sum_n S[c, n] C_n + D_c x_c. S starts at zero."""
    n, channels = x.shape
    S = np.zeros(A.shape)
    y = np.zeros((n, channels))
    for t in range(n):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def scan_mixer(h, w, p, mx):
    inner, rank, N = mx["inner"], mx["dt_rank"], mx["state"]
    both = linear(h, w[p + "in"])
    x, z = both[:, :inner], both[:, inner:]
    x = kept(silu(short_conv(x, w[p + "conv"], w[p + "conv.b"])))
    low = linear(x, w[p + "x"])
    dt = softplus(f64(low[:, :rank]) @ f64(w[p + "dt"]).T + f64(w[p + "dt.b"]))
    y = selective_scan(x, dt, -np.exp(f64(w[p + "A_log"])), low[:, rank:rank + N], low[:, rank + N:], f64(w[p + "D"]))
    return linear(kept(y * silu(z)), w[p + "o"])


# --------------------------------------------------------------------------- attention with kept first tokens

def rotate_pairs(x, positions, base, dims):
    """x [n, heads, dim]: pairs (2i, 2i+1) of the first `dims` dimensions turned by position * base^(-2i/dims)."""
    x = f64(x).copy()
    for i in range(dims // 2):
        a = f64(positions) * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        u, v = x[:, :, 2 * i].copy(), x[:, :, 2 * i + 1].copy()
        x[:, :, 2 * i], x[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return x


def window_mask(n, size, keep_first):
    """Position i sees j <= i with i - j < size or j < keep_first."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_with_sink(scores, visible, sink):
    """Row-wise softmax over the visible entries with exp(sink) as one more term of the denominator."""
    s = np.where(visible, scores, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - m))


def window_attention(h, w, p, mx):
    n, H, G, dim = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"]
    q = kept(short_conv(linear(h, w[p + "q"], w[p + "q.b"]), w[p + "q.conv"])).reshape(n, H, dim)
    k = kept(short_conv(linear(h, w[p + "k"], w[p + "k.b"]), w[p + "k.conv"])).reshape(n, G, dim)
    v = k
    rot = mx["rot"]
    q = kept(rotate_pairs(q, np.arange(n), rot["base"], rot["dims"]))
    k = kept(rotate_pairs(k, np.arange(n), rot["base"], rot["dims"]))
    see = window_mask(n, mx["mask"]["size"], mx["mask"]["keep_first"])
    out = np.zeros((n, H, dim))
    for head in range(H):
        g = head // (H // G)
        s = capped(float(mx["scale"]) * (q[:, head] @ k[:, g].T), mx["softcap"])
        out[:, head] = softmax_with_sink(s, see, float(f64(w[p + "sink"])[head])) @ v[:, g]
    return linear(kept(out.reshape(n, H * dim)), w[p + "o"])


# --------------------------------------------------------------------------- the delta rule

def delta_recurrence(q, k, v, beta, g):
    """Per head: S <- g * S (rows: key channels); u = beta (v - S^T k); S <- S + k u^T; o = S^T q. S starts at zero.
    q, k, g [n, H, dim]; v [n, H, vdim]; beta [n, H]."""
    n, H, dim = q.shape
    out = np.zeros(v.shape)
    for head in range(H):
        S = np.zeros((dim, v.shape[2]))
        for t in range(n):
            S = g[t, head][:, None] * S
            u = beta[t, head] * (v[t, head] - S.T @ k[t, head])
            S = S + np.outer(k[t, head], u)
            out[t, head] = S.T @ q[t, head]
    return out


def delta_mixer(h, w, p, mx, eps):
    n, H, G, dim, vdim = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    conv = lambda leaf: silu(short_conv(linear(h, w[p + leaf]), w[p + leaf + ".conv"]))
    unit = lambda x: x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + UNIT_EPS)
    q = unit(conv("q").reshape(n, G, dim)) * dim ** -0.5
    k = unit(conv("k").reshape(n, G, dim))
    v = conv("v").reshape(n, H, vdim)
    each = lambda x: np.repeat(x, H // G, axis=1)
    beta = sigmoid(linear(h, w[p + "b"]))
    a = f64(linear(h, w[p + "a1"])) @ f64(w[p + "a2"]).T + f64(w[p + "dt_bias"])
    g = np.exp(-np.exp(f64(w[p + "A_log"]))[None, :, None] * softplus(a).reshape(n, H, dim))
    o = delta_recurrence(each(q), each(k), v, beta, g)
    gate = sigmoid(f64(linear(h, w[p + "g1"])) @ f64(w[p + "g2"]).T)
    o = (unit_rms(o, eps) * f64(w[p + "norm"])).reshape(n, H * vdim) * gate
    return linear(kept(o), w[p + "o"])


def parallel_mixer(h, w, p, mx, eps):
    left = window_attention(h, w, p + "left.", mx["left"])
    right = delta_mixer(h, w, p + "right.", mx["right"], eps)
    return float(mx["left_scale"]) * left + float(mx["right_scale"]) * right


# --------------------------------------------------------------------------- linear attention with constant decays

def constant_decay_recurrence(q, k, v, decay):
    """Per head: S <- decay S + k v^T; o = S^T q. S starts at zero. q, k [n, H, dim]; v [n, H, vdim]; decay [H]."""
    n, H, dim = q.shape
    out = np.zeros(v.shape)
    for head in range(H):
        S = np.zeros((dim, v.shape[2]))
        for t in range(n):
            S = decay[head] * S + np.outer(k[t, head], v[t, head])
            out[t, head] = S.T @ q[t, head]
    return out


def lightning_mixer(h, w, p, mx, eps):
    n, H, dim, vdim = h.shape[0], mx["heads"], mx["dim"], mx["vdim"]
    q = silu(linear(h, w[p + "q"])).reshape(n, H, dim)
    k = silu(linear(h, w[p + "k"])).reshape(n, H, dim)
    v = silu(linear(h, w[p + "v"])).reshape(n, H, vdim)
    o = constant_decay_recurrence(q, k, v, [float(d) for d in mx["decay"]]).reshape(n, H * vdim)
    o = unit_rms(o, eps) * f64(w[p + "norm"]) * sigmoid(linear(h, w[p + "g"]))
    return linear(kept(o), w[p + "o"])


# --------------------------------------------------------------------------- feed-forwards

def dense_mlp(h, w, p):
    return linear(kept(np.maximum(linear(h, w[p + "gate"]), 0.0) * linear(h, w[p + "up"])), w[p + "down"])


def route(logits, top):
    """The `top` largest logits of a row (ties to the lower index) and the softmax over those alone."""
    order = sorted(range(len(logits)), key=lambda e: (-logits[e], e))[:top]
    z = np.array([logits[e] for e in order])
    e = np.exp(z - z.max())
    return order, e / e.sum()


def expert(h, w, p, limit):
    g = np.minimum(linear(h, w[p + "gate"]), limit)
    u = np.clip(linear(h, w[p + "up"]), -limit, limit)
    return linear(kept(g * sigmoid(EXPERT_SLOPE * g) * (u + 1.0)), w[p + "down"])


def moe_mlp(h, w, p, mlp, margins=None):
    z = f64(h) @ f64(w[p + "router"]).T + f64(w[p + "router.b"])
    top = mlp["router"]["top"]
    out = f64(expert(h, w, p + "shared.", float(mlp["shared"]["limit"]))).copy()
    for t in range(h.shape[0]):
        chosen, weights = route(z[t], top)
        if margins is not None and top < z.shape[1]:
            s = np.sort(z[t])[::-1]
            margins.append(float(s[top - 1] - s[top]))
        for e, c in zip(chosen, weights):
            out[t] += c * expert(h[t:t + 1], w, f"{p}e{e}.", float(mlp["expert"]["limit"]))[0]
    return out


# --------------------------------------------------------------------------- the model

def run_order(cfg):
    """[(layer, number of the pass if a pass of the loop starts here, else None)]."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def forward(w, cfg, tokens, layers_out=None, margins=None):
    """Logits [n, vocab] of a whole sequence from position 0."""
    eps = float(cfg["norm"]["eps"])
    x0 = f64(w["embed"])[list(tokens)] * float(cfg["embedding"]["scale"])
    x = x0.copy()
    for i, starts in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if starts is not None:
            if starts > 0:
                x = x + x0
            x = x + f64(w["loop.step"])[starts]
        h = layer_norm(x, w, p + "norm1", eps)
        mx, kind = layer["mixer"], layer["type"]
        if kind == "mamba1":
            y = scan_mixer(h, w, p + "mix.", mx)
        elif kind == "parallel":
            y = parallel_mixer(h, w, p + "mix.", mx, eps)
        else:
            y = lightning_mixer(h, w, p + "mix.", mx, eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            y = y + (dense_mlp(h, w, p + "mlp.") if mlp["kind"] == "dense" else moe_mlp(h, w, p + "mlp.", mlp, margins))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return capped(f64(layer_norm(x, w, "final.norm", eps)) @ f64(w["head"]).T, cfg["logit_softcap"])


def generate(w, cfg, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(w, cfg, toks)[-1])))
    return toks[len(prompt):]


# --------------------------------------------------------------------------- configurations and weights for the tests

def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=6, top=2, limit=1.5, shared_ff=20, shared_limit=1.0):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top},
            "shared": {"ff": shared_ff, "limit": shared_limit}}


def scan_layer(inner=48, state=12, dt_rank=5, conv=4, mlp="dense"):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}, "mlp": dense() if mlp == "dense" else mlp}


def parallel_layer(heads=4, kv_heads=2, dim=16, window=20, keep_first=3, softcap=20.0, scale=None, rot=8, base=10000.0, conv=4, rheads=4,
                   rkv_heads=2, rdim=12, rvdim=20, rconv=4, left_scale=0.7, right_scale=1.2, mlp="dense"):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "softcap": softcap,
            "scale": float(scale if scale is not None else dim ** -0.5), "mask": {"size": window, "keep_first": keep_first},
            "rot": {"base": base, "dims": rot}}
    right = {"heads": rheads, "kv_heads": rkv_heads, "dim": rdim, "vdim": rvdim, "conv": rconv}
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale},
            "mlp": dense() if mlp == "dense" else mlp}


def lightning_layer(heads=3, dim=12, vdim=20, decay=None, mlp="dense"):
    decay = [float(d) for d in (decay if decay is not None else np.exp(-np.exp(np.linspace(-0.5, -6.0, heads))))]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": dense() if mlp == "dense" else mlp}


def make_config(layers, vocab=160, width=64, eps=1e-5, scale=3.0, softcap=25.0, loop=None):
    cfg = {"architecture": "Vurazen", "embedding": {"scale": scale}, "layers": layers, "logit_softcap": softcap, "norm": {"eps": eps},
           "vocab": vocab, "width": width}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def tensor_shapes(cfg, ranks=(6, 10)):
    """ranks: the inner sizes of a right mixer's decay and gate projections."""
    D = cfg["width"]
    s = {"embed": (cfg["vocab"], D), "head": (cfg["vocab"], D)}
    if cfg.get("loop"):
        s["loop.step"] = (cfg["loop"]["times"], D)

    def norm(name):
        s[name], s[name + ".b"] = (D,), (D,)

    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        norm(p + "norm1")
        m = p + "mix."
        if layer["type"] == "mamba1":
            I, N, r = mx["inner"], mx["state"], mx["dt_rank"]
            s[m + "in"], s[m + "conv"], s[m + "conv.b"] = (2 * I, D), (I, mx["conv"]), (I,)
            s[m + "x"], s[m + "dt"], s[m + "dt.b"] = (r + 2 * N, I), (I, r), (I,)
            s[m + "A_log"], s[m + "D"], s[m + "o"] = (I, N), (I,), (D, I)
        elif layer["type"] == "lightning":
            nqk, nv = mx["heads"] * mx["dim"], mx["heads"] * mx["vdim"]
            s[m + "q"], s[m + "k"], s[m + "v"], s[m + "g"], s[m + "o"], s[m + "norm"] = (nqk, D), (nqk, D), (nv, D), (nv, D), (D, nv), (nv,)
        else:
            lf, rt = mx["left"], mx["right"]
            a, nq, nk = m + "left.", lf["heads"] * lf["dim"], lf["kv_heads"] * lf["dim"]
            s[a + "q"], s[a + "k"], s[a + "q.b"], s[a + "k.b"] = (nq, D), (nk, D), (nq,), (nk,)
            s[a + "q.conv"], s[a + "k.conv"] = (nq, lf["conv"]), (nk, lf["conv"])
            s[a + "sink"], s[a + "o"] = (lf["heads"],), (D, nq)
            b, H, dim, vdim = m + "right.", rt["heads"], rt["dim"], rt["vdim"]
            nqk, nv = rt["kv_heads"] * dim, H * vdim
            for leaf, n in (("q", nqk), ("k", nqk), ("v", nv)):
                s[b + leaf], s[b + leaf + ".conv"] = (n, D), (n, rt["conv"])
            s[b + "b"], s[b + "A_log"], s[b + "norm"] = (H, D), (H,), (vdim,)
            s[b + "a1"], s[b + "a2"], s[b + "dt_bias"] = (ranks[0], D), (H * dim, ranks[0]), (H * dim,)
            s[b + "g1"], s[b + "g2"], s[b + "o"] = (ranks[1], D), (nv, ranks[1]), (D, nv)
        mlp = layer.get("mlp")
        if mlp is not None:
            q = p + "mlp."
            units = [q] if mlp["kind"] == "dense" else [f"{q}e{e}." for e in range(mlp["router"]["experts"])]
            ff = mlp["ff"] if mlp["kind"] == "dense" else mlp["expert"]["ff"]
            sizes = [(u, ff) for u in units]
            if mlp["kind"] == "moe":
                s[q + "router"], s[q + "router.b"] = (mlp["router"]["experts"], D), (mlp["router"]["experts"],)
                sizes.append((q + "shared.", mlp["shared"]["ff"]))
            for u, n in sizes:
                s[u + "gate"], s[u + "up"], s[u + "down"] = (n, D), (n, D), (D, n)
    norm("final.norm")
    return s


def random_weights(cfg, seed, ranks=(6, 10), sharp=3.0, expert_gain=1.0):
    """float32 weights that bfloat16 holds exactly (so that both dtypes load the same model). Matrices are N(0, 1/in);
    attention's queries and keys are `sharp` times larger so that attention is not flat and a key that is lost or misplaced
    moves the logits; decays and step sizes are spread between fast and slow channels. `expert_gain` scales what the routed
    experts add: a router's close call that 16-bit rounding decides the other way then stays inside a 16-bit tolerance."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg, ranks).items():
        leaf = name.split(".")[-1]
        if name == "embed":
            t = rng.standard_normal(shape)
        elif name == "loop.step":
            t = rng.standard_normal(shape) * 0.7
        elif leaf in ("norm1", "norm"):
            t = 1.0 + rng.standard_normal(shape) * 0.1
        elif name.endswith("right.b"):
            t = rng.standard_normal(shape) / np.sqrt(shape[-1])
        elif name.endswith("dt.b"):
            t = rng.uniform(-6.0, 0.5, shape)
        elif name.endswith("router.b"):
            t = rng.standard_normal(shape)
        elif leaf == "b":
            t = rng.standard_normal(shape) * 0.3
        elif leaf == "conv":
            t = rng.standard_normal(shape) * 0.5
            t[:, -1] += 0.7
        elif leaf == "sink":
            t = rng.uniform(-1.0, 3.0, shape)
        elif leaf == "A_log":
            t = rng.uniform(-2.0, 1.5, shape)
        elif leaf == "dt_bias":
            t = rng.uniform(-5.0, 0.5, shape)
        elif leaf == "D":
            t = rng.standard_normal(shape)
        else:
            t = rng.standard_normal(shape) / np.sqrt(shape[-1])
            if leaf in ("q", "k") and ".left." in name:
                t = t * sharp
            if leaf == "router":
                t = t * 3.0
            if leaf == "down" and ".mlp.e" in name:
                t = t * expert_gain
        w[name] = round_bf16(np.asarray(t, dtype=np.float32))
    return w


def write_safetensors(path, tensors, bf16=True):
    """One file: 8-byte little-endian header length, JSON header, data. bf16 stores the upper 16 bits."""
    header, blobs, off = {}, [], 0
    for name, t in tensors.items():
        shape = list(np.shape(t))
        a = np.ascontiguousarray(t, dtype=np.float32).reshape(-1)
        if bf16:
            data = (a.view(np.uint32) >> 16).astype("<u2").tobytes()
            dt = "BF16"
        else:
            data = a.astype("<f4").tobytes()
            dt = "F32"
        header[name] = {"dtype": dt, "shape": shape, "data_offsets": [off, off + len(data)]}
        blobs.append(data)
        off += len(data)
    hj = json.dumps(header).encode()
    hj += b" " * (-len(hj) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(hj)))
        f.write(hj)
        for b in blobs:
            f.write(b)


def write_model_dir(path, cfg, weights, bf16=True):
    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(path / "model.safetensors", weights, bf16=bf16)
