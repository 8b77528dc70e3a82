"""Vurazen: a decoder whose configuration lists its layers in any order. A layer has ONE norm (mean and variance, weight and
bias); its mixer and, unless its `mlp` is null, its feed-forward both read that norm's output and join the residual stream
side by side. The embedding is multiplied by `embedding.scale`, the logits are capped. Mixers:

  mamba1     a selective scan: a diagonal state per channel whose decay depends on the token, behind a short convolution;
  parallel   two mixers on the same input, `left_scale * left + right_scale * right`. left: grouped-query attention whose q
             and k have biases and pass a short convolution, whose values are its keys ahead of the rotation, in a window of
             `mask.size` positions beside which the first `mask.keep_first` stay visible, with capped scores and a learned
             sink per head; right: a gated delta rule with a decay per key channel (config/dugazen.py's recurrence);
  lightning  linear attention with a constant decay per head and one norm over all heads.

Feed-forwards: `dense` (relu(gate) * up) and `moe` (the `top` largest router logits, with a bias, softmax over those alone,
clamped experts, and a shared expert for every token). `loop` runs layers start .. stop-1 `times` times in a row with the
same weights, each pass with a cache and a state of its own; ahead of every pass but the first the embedding's output joins
the stream again, and ahead of pass t the vector `loop.step`[t]. config.json:

    {"architecture": "Vurazen", "vocab": V, "width": D, "norm": {"eps": e}, "embedding": {"scale": c}, "logit_softcap": s,
     "loop": {"start": a, "stop": b, "times": n},                                                   (optional)
     "layers": [{"type": "mamba1", "mixer": {"inner", "state", "dt_rank", "conv"}, "mlp": ...},
                {"type": "parallel", "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap", "conv",
                                                        "rot": {"base", "dims"}, "mask": {"size", "keep_first"}},
                                               "right": {"heads", "kv_heads", "dim", "vdim", "conv"},
                                               "left_scale", "right_scale"}, "mlp": ...},
                {"type": "lightning", "mixer": {"heads", "dim", "vdim", "decay": [...]}, "mlp": ...}],
     with "mlp": {"kind": "dense", "ff"} | {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top"},
                                            "shared": {"ff", "limit"}} | null}

Tensors: `embed`, `head`, `final.norm` (+ `.b`), `loop.step` [times, D], and per layer i `l<i>.norm1` (+ `.b`), `l<i>.mix.*`,
`l<i>.mlp.*`. The inner sizes of a right mixer's two-step projections (a1/a2, g1/g2) are not in config.json: they are read
from the checkpoint's tensor shapes, or given to `parse_vurazen_config`.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from ..errors import LoadError, UnsupportedError
from .registry import Architecture, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry

# Constants that the design fixes.
EXPERT_SLOPE = 1.702       # an expert's unit: y = g * sigmoid(EXPERT_SLOPE * g) * (u + EXPERT_UP_SHIFT)
EXPERT_UP_SHIFT = 1.0
UNIT_EPS = 1e-6            # inside the root of the delta rule's unit norms
DEFAULT_RANK = 16          # inner size of a1/a2 and g1/g2 when no checkpoint says (random weights)
DEFAULT_MAX_POSITIONS = 1 << 17
MIXERS = ("mamba1", "parallel", "lightning")


@dataclass
class VurazenConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_softcap: float                              # 0: the logits as they are
    layers: list = field(default_factory=list)        # the configuration's own dictionaries, validated
    loop: dict | None = None                          # {"start", "stop", "times"} or None
    ranks: dict = field(default_factory=dict)          # layer index -> (decay rank, gate rank) of a right mixer
    max_positions: int = DEFAULT_MAX_POSITIONS

    def to_dict(self) -> dict:
        d = {"architecture": "Vurazen", "embedding": {"scale": self.embedding_scale}, "layers": self.layers,
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


def _sizes(mx: dict, where: str, keys) -> None:
    for key in keys:
        _int(_req(mx, key, where), f"{where}.{key}")
    if "kv_heads" in keys and mx["heads"] % mx["kv_heads"]:
        raise LoadError(f"config.json: {where}: {mx['heads']} heads are not a multiple of {mx['kv_heads']} kv heads")


def _check_mixer(kind: str, mx: dict, where: str) -> None:
    if kind == "mamba1":
        _sizes(mx, where, ("inner", "state", "dt_rank", "conv"))
    elif kind == "lightning":
        _sizes(mx, where, ("heads", "dim", "vdim"))
        decay = _req(mx, "decay", where)
        if not isinstance(decay, list) or len(decay) != mx["heads"]:
            raise LoadError(f"config.json: {where}: 'decay' must list a number for each of the {mx['heads']} heads")
        for d in decay:
            _number(d, f"{where}.decay")
    else:
        left, right = _req(mx, "left", where), _req(mx, "right", where)
        lw = where + " left"
        _sizes(left, lw, ("heads", "kv_heads", "dim", "vdim", "conv"))
        if left["vdim"] != left["dim"]:
            raise LoadError(f"config.json: {lw}: the values are the keys, but vdim {left['vdim']} differs from dim {left['dim']}")
        _number(_req(left, "scale", lw), lw + ".scale")
        if left.get("softcap") is not None:
            _number(left["softcap"], lw + ".softcap")
        mask = left.get("mask")
        if mask is not None:
            _int(_req(mask, "size", lw + "'s mask"), f"{lw} mask.size")
            _int(mask.get("keep_first", 0), f"{lw} mask.keep_first", 0)
        rot = left.get("rot")
        if rot is not None:
            dims = _int(_req(rot, "dims", lw + "'s rot"), f"{lw} rot.dims", 0)
            if dims % 2 or dims > left["dim"]:
                raise LoadError(f"config.json: {lw}: rot.dims {dims} must be even and at most dim {left['dim']}")
            if dims and not _number(_req(rot, "base", lw + "'s rot"), f"{lw} rot.base") > 0:
                raise LoadError(f"config.json: {lw}: rot.base must be positive")
        _sizes(right, where + " right", ("heads", "kv_heads", "dim", "vdim", "conv"))
        for key in ("left_scale", "right_scale"):
            _number(_req(mx, key, where), f"{where}.{key}")


def _check_mlp(mlp, where: str) -> None:
    if mlp is None:
        return
    w = where + "'s mlp"
    kind = _req(mlp, "kind", w)
    if kind == "dense":
        _int(_req(mlp, "ff", w), f"{w}.ff")
    elif kind == "moe":
        r = _req(mlp, "router", w)
        experts = [("expert", _req(mlp, "expert", w))] + ([("shared", mlp["shared"])] if mlp.get("shared") is not None else [])
        for name, ex in experts:
            _int(_req(ex, "ff", f"{w} {name}"), f"{w}.{name}.ff")
            _number(_req(ex, "limit", f"{w} {name}"), f"{w}.{name}.limit")
        E, top = _int(_req(r, "experts", w + " router"), f"{w}.router.experts"), _int(_req(r, "top", w + " router"), f"{w}.router.top")
        if top > E:
            raise LoadError(f"config.json: {where}: cannot choose {top} of {E} experts")
    else:
        raise UnsupportedError(f"config.json: {where} has a feed-forward of kind '{kind}' (supported: dense, moe)")


def parse_vurazen_config(j: dict, ranks: dict | None = None) -> VurazenConfig:
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
    return VurazenConfig(vocab=_int(_req(j, "vocab", top), "vocab"), width=_int(_req(j, "width", top), "width"),
                         eps=_number(_req(_req(j, "norm", top), "eps", "'norm'"), "norm.eps"),
                         embedding_scale=1.0 if scale is None else _number(scale, "embedding.scale"),
                         logit_softcap=0.0 if cap is None else _number(cap, "logit_softcap"), layers=layers, loop=loop,
                         ranks=dict(ranks or {}), max_positions=int(j.get("max_positions", DEFAULT_MAX_POSITIONS)))


def ranks_from_shapes(shapes: dict) -> dict:
    """layer index -> (rows of `l<i>.mix.right.a1`, rows of `l<i>.mix.right.g1`) from a checkpoint's tensor shapes."""
    out = {}
    for name, shape in shapes.items():
        parts = name.split(".")
        if len(parts) == 4 and parts[1:] == ["mix", "right", "a1"] and parts[0][:1] == "l" and parts[0][1:].isdigit():
            g1 = shapes.get(f"{parts[0]}.mix.right.g1")
            if g1 is not None:
                out[int(parts[0][1:])] = (int(shape[0]), int(g1[0]))
    return out


def vurazen_spec(c: VurazenConfig) -> ModelSpec:
    D = c.width

    def norm(name: str) -> PartSpec:
        return PartSpec("layer_norm", {"name": name, "size": D, "eps": c.eps})

    def experts(p: str, mlp: dict) -> PartSpec:
        unit = {"hidden_size": D, "slope": EXPERT_SLOPE, "up_shift": EXPERT_UP_SHIFT}
        routed = PartSpec("routed_experts", {
            **unit, "prefix": p + "mlp.", "intermediate_size": mlp["expert"]["ff"], "limit": float(mlp["expert"]["limit"]),
            "num_experts": mlp["router"]["experts"], "top": mlp["router"]["top"], "score": "softmax", "router_bias": True, "renorm": True})
        shared = mlp.get("shared")
        if shared is None:
            return routed
        return PartSpec("feed_forward_sum", {"parts": [routed, PartSpec("clamped_glu", {
            **unit, "prefix": p + "mlp.shared.", "intermediate_size": shared["ff"], "limit": float(shared["limit"])})]})

    layers = []
    for i, layer in enumerate(c.layers):
        p, mx, kind = f"l{i}.", layer["mixer"], layer["type"]
        if kind == "mamba1":
            mixer = PartSpec("selective_scan", {"prefix": p + "mix.", "hidden_size": D, "inner_size": mx["inner"], "dt_rank": mx["dt_rank"],
                                                "state_size": mx["state"], "conv_taps": mx["conv"]})
        elif kind == "lightning":
            mixer = PartSpec("constant_decay_attention", {"prefix": p + "mix.", "hidden_size": D, "num_heads": mx["heads"], "head_dim": mx["dim"],
                                                          "value_dim": mx["vdim"], "decay": [float(d) for d in mx["decay"]], "eps": c.eps})
        else:
            lf, rt = mx["left"], mx["right"]
            rot, mask = lf.get("rot") or {}, lf.get("mask") or {}
            dims = int(rot.get("dims", 0))
            left = PartSpec("conv_key_attention", {
                "prefix": p + "mix.left.", "hidden_size": D, "num_heads": lf["heads"], "num_kv_heads": lf["kv_heads"], "head_dim": lf["dim"],
                "scale": float(lf["scale"]), "softcap": float(lf.get("softcap") or 0.0), "conv_taps": lf["conv"], "qk_bias": True, "sink": True,
                "window": mask.get("size", 0), "keep_first": mask.get("keep_first", 0),
                "position": PartSpec("rope", {"theta": float(rot["base"]), "head_dim": lf["dim"], "rotary_dim": dims}) if dims else None})
            decay_rank, gate_rank = c.ranks.get(i, c.ranks.get(str(i), (DEFAULT_RANK, DEFAULT_RANK)))
            right = PartSpec("channel_gated_delta", {
                "prefix": p + "mix.right.", "hidden_size": D, "num_heads": rt["heads"], "num_kv_heads": rt["kv_heads"], "head_dim": rt["dim"],
                "value_dim": rt["vdim"], "conv_taps": rt["conv"], "unit_eps": UNIT_EPS, "eps": c.eps, "decay_rank": decay_rank,
                "gate_rank": gate_rank})
            mixer = PartSpec("mixer_sum", {"parts": [(left, float(mx["left_scale"])), (right, float(mx["right_scale"]))]})
        mlp = layer.get("mlp")
        if mlp is None:
            ffn = None
        elif mlp["kind"] == "dense":
            ffn = PartSpec("swiglu", {"prefix": p + "mlp.", "hidden_size": D, "intermediate_size": mlp["ff"], "activation": "relu",
                                      "gate": "gate", "up": "up", "down": "down"})
        else:
            ffn = experts(p, mlp)
        layers.append(LayerSpec(prefix=p, block=PartSpec("shared_norm", {}), mixer=mixer, mixer_norm=norm(p + "norm1"), ffn=ffn, ffn_norm=None))
    order, starts = c.run_layers()
    passes = c.loop["times"] if c.loop is not None else 0
    run_order = tuple(RunEntry(l, before=PartSpec("pass_vector", {"name": "loop.step", "index": starts[i], "passes": passes, "hidden_size": D,
                                                                  "add_origin": starts[i] > 0}) if i in starts else None)
                      for i, l in enumerate(order))
    return ModelSpec(architecture="Vurazen", hidden_size=D, vocab_size=c.vocab, max_positions=c.max_positions,
                     embedding=PartSpec("token_embedding", {"name": "embed", "vocab_size": c.vocab, "hidden_size": D, "scale": c.embedding_scale}),
                     layers=tuple(layers), run_order=run_order, final_norm=norm("final.norm"),
                     head=PartSpec("lm_head", {"name": "head", "tied": False, "vocab_size": c.vocab, "hidden_size": D, "softcap": c.logit_softcap}))


register_architecture(Architecture(name="Vurazen", parse_config=parse_vurazen_config, build_spec=vurazen_spec,
                                   model_types=("vurazen",), shapes_to_config=ranks_from_shapes), replace=True)
