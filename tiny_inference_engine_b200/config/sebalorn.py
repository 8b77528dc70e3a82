"""Sebalorn: a decoder whose configuration lists its layers in any order. A layer has ONE RMS norm, its weight stored as the
distance from one; its mixer and, unless its `mlp` is null, its feed-forward both read that norm's output and join the residual
stream side by side. The embedding is multiplied by `embedding.scale`, the logits are capped. Mixers:

  latent_attention  queries through a normed latent; keys and values from one normed latent per token and one rotated key part
                    (neighbouring dimensions pair up) that all heads share; a learned sink per head; a gate per output channel;
  attention         grouped-query attention: one RMS norm over the whole q (and k) projection, the first `rot.dims` dimensions of
                    each head rotated in halves, a gate per head;
  retention         linear attention with a constant decay per head over rotated q and k (keys times dim^(-1/2)), each head's
                    read-out divided by its root mean square, a SiLU gate.

Feed-forward: `dense`, down(max(up h, 0)^2). `loop` runs layers start .. stop-1 `times` times in a row with the same weights, each
pass with a cache and a state of its own; ahead of pass t the vector `loop.step`[t] joins the stream. config.json:

    {"architecture": "Sebalorn", "vocab": V, "width": D, "norm": {"eps": e}, "embedding": {"scale": c}, "logit_softcap": s,
     "loop": {"start": a, "stop": b, "times": n},                                                   (optional)
     "layers": [{"type": "latent_attention", "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale",
                                                       "rot": {"base", "dims"}}, "mlp": ...},
                {"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "rot": {"base", "dims"}}, "mlp": ...},
                {"type": "retention", "mixer": {"heads", "dim", "vdim", "decay": [...], "rot": {"base", "dims"}}, "mlp": ...}],
     with "mlp": {"kind": "dense", "ff"} | null}

Tensors: `embed`, `head`, `final.norm`, `loop.step` [times, D], and per layer i `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.up|down`.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from ..errors import LoadError, UnsupportedError
from .registry import Architecture, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry

DEFAULT_MAX_POSITIONS = 1 << 17
MIXERS = ("latent_attention", "attention", "retention")
_SIZES = {"latent_attention": ("heads", "dim", "vdim", "kv_rank", "q_rank"), "attention": ("heads", "kv_heads", "dim", "vdim"),
          "retention": ("heads", "dim", "vdim")}


@dataclass
class SebalornConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_softcap: float                              # 0: the logits as they are
    layers: list = field(default_factory=list)        # the configuration's own dictionaries, validated
    loop: dict | None = None                          # {"start", "stop", "times"} or None
    max_positions: int = DEFAULT_MAX_POSITIONS

    def to_dict(self) -> dict:
        d = {"architecture": "Sebalorn", "embedding": {"scale": self.embedding_scale}, "layers": self.layers,
             "logit_softcap": self.logit_softcap, "norm": {"eps": self.eps}, "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            d["loop"] = dict(self.loop)
        return d

    def run_layers(self) -> tuple[list[int], dict[int, int]]:
        """(layer index of every run entry in order, {entry at which a pass of the loop starts: number of the pass})."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n)), {}
        a, b, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        order, starts = list(range(a)), {}
        for t in range(times):
            starts[len(order)] = t
            order += list(range(a, b))
        return order + list(range(b, n)), starts


def _req(d, key: str, where: str):
    if not isinstance(d, dict) or key not in d:
        raise LoadError(f"config.json: {where} has no '{key}'")
    return d[key]


def _int(v, what: str, least: int = 1) -> int:
    if not isinstance(v, int) or isinstance(v, bool) or v < least:
        raise LoadError(f"config.json: {what} must be an integer of at least {least}, got {v!r}")
    return v


def _number(v, what: str) -> float:
    if not isinstance(v, (int, float)) or isinstance(v, bool):
        raise LoadError(f"config.json: {what} must be a number, got {v!r}")
    return float(v)


def _rot_dims(mx: dict) -> int:
    return int((mx.get("rot") or {}).get("dims", 0))


def _check_mixer(kind: str, mx: dict, where: str) -> None:
    for key in _SIZES[kind]:
        _int(_req(mx, key, where), f"{where}.{key}")
    rot = mx.get("rot")
    if rot is not None:
        dims = _int(_req(rot, "dims", where + "'s rot"), f"{where} rot.dims", 0)
        if dims and not _number(_req(rot, "base", where + "'s rot"), f"{where} rot.base") > 0:
            raise LoadError(f"config.json: {where}: rot.base must be positive")
    dims = _rot_dims(mx)
    if kind == "latent_attention":
        part = _int(_req(mx, "rot_dim", where), f"{where}.rot_dim", 0)
        if dims != part or dims % 2:
            raise LoadError(f"config.json: {where}: rot.dims {dims} must be even and the whole rotated part ({part})")
    elif dims % 2 or dims > mx["dim"]:
        raise LoadError(f"config.json: {where}: rot.dims {dims} must be even and at most dim {mx['dim']}")
    if kind == "attention" and mx["heads"] % mx["kv_heads"]:
        raise LoadError(f"config.json: {where}: {mx['heads']} heads are not a multiple of {mx['kv_heads']} kv heads")
    if kind == "retention":
        decay = _req(mx, "decay", where)
        if not isinstance(decay, list) or len(decay) != mx["heads"]:
            raise LoadError(f"config.json: {where}: 'decay' must list a number for each of the {mx['heads']} heads")
        for d in decay:
            _number(d, f"{where}.decay")
    else:
        _number(_req(mx, "scale", where), where + ".scale")


def _check_mlp(mlp, where: str) -> None:
    if mlp is None:
        return
    w = where + "'s mlp"
    kind = _req(mlp, "kind", w)
    if kind != "dense":
        raise UnsupportedError(f"config.json: {where} has a feed-forward of kind '{kind}' (supported: dense, or null for none)")
    _int(_req(mlp, "ff", w), f"{w}.ff")


def parse_sebalorn_config(j: dict) -> SebalornConfig:
    top = "the configuration"
    layers = _req(j, "layers", top)
    if not isinstance(layers, list) or not layers:
        raise LoadError("config.json: 'layers' must be a non-empty list")
    for i, layer in enumerate(layers):
        where = f"layer {i}"
        kind = _req(layer, "type", where)
        if kind not in MIXERS:
            raise UnsupportedError(f"config.json: {where} has type '{kind}' (supported: {', '.join(MIXERS)})")
        _check_mixer(kind, _req(layer, "mixer", where), where + "'s mixer")
        _check_mlp(layer.get("mlp"), where)
    loop = j.get("loop")
    if loop is not None:
        a, b, times = (_req(loop, k, "'loop'") for k in ("start", "stop", "times"))
        if not all(isinstance(v, int) and not isinstance(v, bool) for v in (a, b, times)) or not 0 <= a < b <= len(layers) or times < 1:
            raise LoadError(f"config.json: loop start={a!r} stop={b!r} times={times!r} does not name layers of this model")
        loop = {"start": a, "stop": b, "times": times}
    scale = (j.get("embedding") or {}).get("scale")
    cap = j.get("logit_softcap")
    return SebalornConfig(vocab=_int(_req(j, "vocab", top), "vocab"), width=_int(_req(j, "width", top), "width"),
                          eps=_number(_req(_req(j, "norm", top), "eps", "'norm'"), "norm.eps"),
                          embedding_scale=1.0 if scale is None else _number(scale, "embedding.scale"),
                          logit_softcap=0.0 if cap is None else _number(cap, "logit_softcap"), layers=layers, loop=loop,
                          max_positions=int(j.get("max_positions", DEFAULT_MAX_POSITIONS)))


def sebalorn_spec(c: SebalornConfig) -> ModelSpec:
    D = c.width

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm_one_plus", {"name": name, "size": D, "eps": c.eps})

    def rotation(mx: dict, head_dim: int, pairing: str) -> PartSpec | None:
        dims = _rot_dims(mx)
        return PartSpec("rope", {"theta": float(mx["rot"]["base"]), "head_dim": head_dim, "rotary_dim": dims, "pairing": pairing,
                                 "angles": "float64"}) if dims else None

    layers = []
    for i, layer in enumerate(c.layers):
        p, mx, kind = f"l{i}.", layer["mixer"], layer["type"]
        sizes = {"prefix": p + "mix.", "hidden_size": D, "num_heads": mx["heads"], "head_dim": mx["dim"], "value_dim": mx["vdim"], "eps": c.eps}
        if kind == "latent_attention":
            mixer = PartSpec("latent_attention", {**sizes, "rot_dim": mx["rot_dim"], "kv_rank": mx["kv_rank"], "q_rank": mx["q_rank"],
                                                  "scale": float(mx["scale"]), "sink": True, "output_gate": "channel",
                                                  "position": rotation(mx, mx["rot_dim"], "neighbours")})
        elif kind == "attention":
            mixer = PartSpec("gated_window_attention", {**sizes, "num_kv_heads": mx["kv_heads"], "scale": float(mx["scale"]), "span_norm": True,
                                                        "output_gate": "head", "position": rotation(mx, mx["dim"], "halves") or PartSpec("none")})
        else:
            mixer = PartSpec("constant_decay_attention", {**sizes, "decay": [float(d) for d in mx["decay"]], "activation": None,
                                                          "position": rotation(mx, mx["dim"], "halves"), "k_scale": float(mx["dim"]) ** -0.5,
                                                          "norm_per_head": True, "norm_weight": False, "gate": "silu"})
        mlp = layer.get("mlp")
        ffn = None if mlp is None else PartSpec("squared_relu_mlp", {"prefix": p + "mlp.", "hidden_size": D, "intermediate_size": mlp["ff"]})
        layers.append(LayerSpec(prefix=p, block=PartSpec("shared_norm", {}), mixer=mixer, mixer_norm=norm(p + "norm1"), ffn=ffn, ffn_norm=None))
    order, starts = c.run_layers()
    passes = c.loop["times"] if c.loop is not None else 0
    run_order = tuple(RunEntry(l, before=PartSpec("pass_vector", {"name": "loop.step", "index": starts[i], "passes": passes,
                                                                  "hidden_size": D}) if i in starts else None)
                      for i, l in enumerate(order))
    return ModelSpec(architecture="Sebalorn", hidden_size=D, vocab_size=c.vocab, max_positions=c.max_positions,
                     embedding=PartSpec("token_embedding", {"name": "embed", "vocab_size": c.vocab, "hidden_size": D, "scale": c.embedding_scale}),
                     layers=tuple(layers), run_order=run_order, final_norm=norm("final.norm"),
                     head=PartSpec("lm_head", {"name": "head", "tied": False, "vocab_size": c.vocab, "hidden_size": D, "softcap": c.logit_softcap}))


register_architecture(Architecture(name="Sebalorn", parse_config=parse_sebalorn_config, build_spec=sebalorn_spec,
                                   model_types=("sebalorn",)), replace=True)
