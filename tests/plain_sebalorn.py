"""A plain, slow Sebalorn in numpy: whole sequences, no cache, no state carried between calls, one function per mechanism.
Arithmetic is float64 on the stored values. Nothing here imports the engine package: the tests compare the two.

A Sebalorn model lists its layers in any order. A layer has ONE RMS norm (its weight stored as the distance from one), whose
output both its sublayers read: x <- x + mixer(n(x)) + ff(n(x)); a layer may have no feed-forward. Layers start .. stop-1 may
run several times in a row with the same weights; ahead of every pass a vector of that pass joins the stream. Mixers:

  latent_attention  queries and key/value pairs through normed latents, one rotated key part for all heads, a learned sink per
                    head in the softmax, a gate per output channel;
  attention         grouped-query attention whose q and k are normed over all heads at once, a part of each head rotated, a
                    gate per head;
  retention         linear attention over rotated q and k with a constant decay per head, unit heads and a SiLU gate.

Feed-forward: down(max(up h, 0)^2). The embedding is scaled, the logits are capped.
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np


# --------------------------------------------------------------------------- small functions

def f64(a):
    return np.asarray(a, dtype=np.float64)


def sigmoid(z):
    z = f64(z)
    return np.exp(np.minimum(z, 0.0)) / (1.0 + np.exp(-np.abs(z)))


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
    a pipeline with 16-bit activations cannot avoid, which is what a tolerance for such a pipeline is measured against. With
    `draw`, random relative errors of up to 2^-9 (half a unit of bfloat16) take the place of the rounding."""

    def __init__(self, draw=None):
        self.draw = draw

    def __enter__(self):
        global _act
        if self.draw is None:
            _act = lambda y: round_bf16(y).astype(np.float64)
        else:
            rng = np.random.default_rng(self.draw)
            _act = lambda y: f64(y) * (1.0 + rng.uniform(-2.0 ** -9, 2.0 ** -9, np.shape(y)))

    def __exit__(self, *exc):
        global _act
        _act = None


def kept(y):
    return y if _act is None else _act(y)


def linear(x, w):
    return kept(f64(x) @ f64(w).T)


def norm_one_plus(x, w, eps):
    return kept(unit_rms(x, eps) * (1.0 + f64(w)))


def norm_plain(x, w, eps):
    return kept(unit_rms(x, eps) * f64(w))


# --------------------------------------------------------------------------- rotations, softmax

def _turned(u, v, positions, base, dims, i):
    a = f64(positions) * float(base) ** (-2.0 * i / dims)
    c, s = np.cos(a)[:, None], np.sin(a)[:, None]
    return u * c - v * s, v * c + u * s


def rotate_neighbours(x, positions, base, dims):
    """x [n, heads, dim]: 2i with 2i + 1, i < dims / 2; dimensions from `dims` on pass."""
    x, y = f64(x), f64(x).copy()
    for i in range(dims // 2):
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = _turned(x[:, :, 2 * i], x[:, :, 2 * i + 1], positions, base, dims, i)
    return y


def rotate_halves(x, positions, base, dims):
    """x [n, heads, dim]: i with i + dims / 2, i < dims / 2; dimensions from `dims` on pass."""
    x, y, half = f64(x), f64(x).copy(), dims // 2
    for i in range(half):
        y[:, :, i], y[:, :, i + half] = _turned(x[:, :, i], x[:, :, i + half], positions, base, dims, i)
    return y


def causal_softmax(scores, sink=None):
    """Row-wise over j <= i; with `sink`, exp(sink) is one more term of every denominator."""
    n = scores.shape[0]
    s = np.where(np.tril(np.ones((n, n), dtype=bool)), scores, -np.inf)
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    total = e.sum(axis=-1, keepdims=True)
    return e / (total if sink is None else total + np.exp(sink - m))


# --------------------------------------------------------------------------- mixers

def latent_mixer(h, w, p, mx, eps):
    n, H, dim, rd, vd, rank = h.shape[0], mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    at, rot = np.arange(n), mx["rot"]
    q = linear(norm_plain(linear(h, w[p + "dq"]), w[p + "dq.norm"], eps), w[p + "uq"]).reshape(n, H, dim + rd)
    low = linear(h, w[p + "dkv"])
    c = norm_plain(low[:, :rank], w[p + "dkv.norm"], eps)
    r = kept(rotate_neighbours(low[:, None, rank:], at, rot["base"], rd))[:, 0]
    k = linear(c, w[p + "uk"]).reshape(n, H, dim)
    v = linear(c, w[p + "uv"]).reshape(n, H, vd)
    qr = kept(rotate_neighbours(q[:, :, dim:], at, rot["base"], rd))
    out = np.zeros((n, H, vd))
    for head in range(H):
        s = (q[:, head, :dim] @ k[:, head].T + qr[:, head] @ r.T) * float(mx["scale"])
        out[:, head] = causal_softmax(s, float(f64(w[p + "sink"])[head])) @ v[:, head]
    gated = kept(out).reshape(n, H * vd) * sigmoid(linear(h, w[p + "g"]))
    return linear(kept(gated), w[p + "o"])


def attention_mixer(h, w, p, mx, eps):
    n, H, G, dim, vd = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    at, rot = np.arange(n), mx["rot"]
    q = unit_rms(linear(h, w[p + "q"]), eps) * f64(w[p + "q.norm"])
    k = unit_rms(linear(h, w[p + "k"]), eps) * f64(w[p + "k.norm"])
    q = kept(rotate_halves(q.reshape(n, H, dim), at, rot["base"], rot["dims"]))
    k = kept(rotate_halves(k.reshape(n, G, dim), at, rot["base"], rot["dims"]))
    v = linear(h, w[p + "v"]).reshape(n, G, vd)
    gate = sigmoid(linear(h, w[p + "g"]))
    out = np.zeros((n, H, vd))
    for head in range(H):
        g = head // (H // G)
        out[:, head] = kept(causal_softmax(float(mx["scale"]) * (q[:, head] @ k[:, g].T)) @ v[:, g]) * gate[:, head:head + 1]
    return linear(kept(out.reshape(n, H * vd)), w[p + "o"])


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


def retention_mixer(h, w, p, mx, eps):
    n, H, dim, vd = h.shape[0], mx["heads"], mx["dim"], mx["vdim"]
    at, rot = np.arange(n), mx["rot"]
    q = rotate_halves(linear(h, w[p + "q"]).reshape(n, H, dim), at, rot["base"], rot["dims"])
    k = rotate_halves(linear(h, w[p + "k"]).reshape(n, H, dim), at, rot["base"], rot["dims"]) * dim ** -0.5
    v = linear(h, w[p + "v"]).reshape(n, H, vd)
    o = unit_rms(constant_decay_recurrence(q, k, v, [float(d) for d in mx["decay"]]), eps)
    return linear(kept(o.reshape(n, H * vd) * silu(linear(h, w[p + "g"]))), w[p + "o"])


MIXERS = {"latent_attention": latent_mixer, "attention": attention_mixer, "retention": retention_mixer}


def dense_mlp(h, w, p):
    return linear(kept(np.maximum(linear(h, w[p + "up"]), 0.0) ** 2), w[p + "down"])


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


def forward(w, cfg, tokens, layers_out=None):
    """Logits [n, vocab] of a whole sequence from position 0."""
    eps = float(cfg["norm"]["eps"])
    x = f64(w["embed"])[list(tokens)] * float(cfg["embedding"]["scale"])
    for i, starts in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if starts is not None:
            x = x + f64(w["loop.step"])[starts]
        h = norm_one_plus(x, w[p + "norm1"], eps)
        y = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + dense_mlp(h, w, p + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return capped(f64(norm_one_plus(x, w["final.norm"], eps)) @ f64(w["head"]).T, cfg.get("logit_softcap"))


def generate(w, cfg, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(w, cfg, toks)[-1])))
    return toks[len(prompt):]


# --------------------------------------------------------------------------- configurations and weights for the tests

def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def latent_layer(heads=3, dim=10, rot_dim=6, vdim=14, kv_rank=24, q_rank=20, base=10000.0, scale=None, mlp="dense"):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                                  "scale": float(scale if scale is not None else (dim + rot_dim) ** -0.5),
                                                  "rot": {"base": base, "dims": rot_dim}}, "mlp": dense() if mlp == "dense" else mlp}


def attention_layer(heads=4, kv_heads=2, dim=16, vdim=12, rot=8, base=10000.0, scale=None, mlp="dense"):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(scale if scale is not None else dim ** -0.5),
                                           "rot": {"base": base, "dims": rot}}, "mlp": dense() if mlp == "dense" else mlp}


def retention_layer(heads=3, dim=12, vdim=20, rot=12, base=10000.0, decay=None, mlp="dense"):
    decay = [float(d) for d in (decay if decay is not None else 1.0 - 2.0 ** -np.linspace(1.5, 9.0, heads))]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": rot}},
            "mlp": dense() if mlp == "dense" else mlp}


def make_config(layers, vocab=160, width=64, eps=1e-5, scale=3.0, softcap=25.0, loop=None):
    cfg = {"architecture": "Sebalorn", "embedding": {"scale": scale}, "layers": layers, "logit_softcap": softcap, "norm": {"eps": eps},
           "vocab": vocab, "width": width}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def tensor_shapes(cfg):
    D = cfg["width"]
    s = {"embed": (cfg["vocab"], D), "head": (cfg["vocab"], D), "final.norm": (D,)}
    if cfg.get("loop"):
        s["loop.step"] = (cfg["loop"]["times"], D)
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        m, H, dim, vd = p + "mix.", mx["heads"], mx["dim"], mx["vdim"]
        s[p + "norm1"], s[m + "o"] = (D,), (D, H * vd)
        if layer["type"] == "latent_attention":
            rd, rank, qr = mx["rot_dim"], mx["kv_rank"], mx["q_rank"]
            s[m + "dq"], s[m + "dq.norm"], s[m + "uq"] = (qr, D), (qr,), (H * (dim + rd), qr)
            s[m + "dkv"], s[m + "dkv.norm"] = (rank + rd, D), (rank,)
            s[m + "uk"], s[m + "uv"], s[m + "sink"], s[m + "g"] = (H * dim, rank), (H * vd, rank), (H,), (H * vd, D)
        elif layer["type"] == "attention":
            G = mx["kv_heads"]
            s[m + "q"], s[m + "k"], s[m + "v"], s[m + "g"] = (H * dim, D), (G * dim, D), (G * vd, D), (H, D)
            s[m + "q.norm"], s[m + "k.norm"] = (H * dim,), (G * dim,)
        else:
            s[m + "q"], s[m + "k"], s[m + "v"], s[m + "g"] = (H * dim, D), (H * dim, D), (H * vd, D), (H * vd, D)
        mlp = layer.get("mlp")
        if mlp is not None:
            s[p + "mlp.up"], s[p + "mlp.down"] = (mlp["ff"], D), (D, mlp["ff"])
    return s


def random_weights(cfg, seed, sharp=2.0):
    """float32 weights that bfloat16 holds exactly (so that both dtypes load the same model). Matrices are N(0, 1/in);
    attention's query projections are `sharp` times larger so that attention is not flat and a key that is lost or misplaced
    moves the logits."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        kind = cfg["layers"][int(name.split(".")[0][1:])]["type"] if ".mix." in name else ""
        if name == "embed":
            t = rng.standard_normal(shape)
        elif name == "loop.step":
            t = rng.standard_normal(shape) * 0.7
        elif leaf == "norm1" or name == "final.norm":
            t = rng.standard_normal(shape) * 0.2
        elif leaf == "norm":
            t = 1.0 + rng.standard_normal(shape) * 0.2
            if name.endswith("q.norm") and not name.endswith("dq.norm"):
                t = t * sharp
        elif leaf == "sink":
            t = rng.uniform(-1.0, 3.0, shape)
        else:
            t = rng.standard_normal(shape) / np.sqrt(shape[-1])
            if leaf == "uq":
                t = t * sharp
            if leaf == "down":
                t = t * 0.6
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
