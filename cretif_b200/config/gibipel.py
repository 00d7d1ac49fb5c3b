"""Typed configuration of the Gibipel decoder, read from config.json, and its ModelSpec.

A Gibipel checkpoint's config.json names its class with ``"architecture": "Gibipel"`` and
describes the model as a list of layers, each with sizes of its own:

=====================  ========================================================================
key                    meaning
=====================  ========================================================================
vocab, width           vocabulary and residual width
norm.eps               eps of every RMS norm of the model
embedding.scale        factor on the embedding's rows
logit_scale            factor on the logits
layers[i].type         ``parallel``
layers[i].mixer        left: heads, kv_heads, dim, vdim, scale, mask {size (the window), pool (the
                       block of tokens that is seen as one beyond it)}, rot {base, dims, scaling
                       {factor, low, high, original} (optional)};
                       right: heads, dim, vdim, gate_cap; left_scale, right_scale
layers[i].mlp          ``{"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k,
                       "identity": I, "groups": {"count", "keep"}}, "shared": {"ff": Fs}}``
                       (identity, groups and shared optional), or null
max_positions          (optional) longest sequence; the design itself has no limit
=====================  ========================================================================

The norms stand on the sublayers' outputs, ``x += norm1(mixer(x))``, ``x += norm2(ff(x))``, and
have one weight for all channels, as has the final norm.  A layer's mixer is two side by side:
attention with biases, norms over the whole query and key projections, a rotation with stretched
wavelengths, a window with pooled blocks before it and a learned term per head in the softmax's
denominator; and a matrix memory with exponential gates.  The feed-forward's experts are chosen by
softmax scores with a correction, in groups that are scored by their best; the router's last outputs
are identities.  The output matrix is a tensor of its own.  Tensors are named ``l<i>.mix.left.*``,
``l<i>.mix.right.*``, ``l<i>.mlp.*`` (``e<n>.gate/up/down``, ``router``, ``correction``,
``shared.gate/up/down``), ``l<i>.norm1/2``, ``embed``, ``final.norm`` and ``head``.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List

from .registry import ConfigError, register_architecture
from .spec import BranchSpec, LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MIXER_TYPES = ("parallel",)
DEFAULT_MAX_POSITIONS = 1 << 20
WEIGHT_SUM_EPS = 1e-20                   # added to the sum of a token's chosen scores


@dataclass
class GibipelConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    layers: List[Dict[str, Any]] = field(default_factory=list)
    max_positions: int = DEFAULT_MAX_POSITIONS
    architecture: str = "Gibipel"

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab,
                             "width": self.width, "norm": {"eps": self.eps},
                             "embedding": {"scale": self.embedding_scale},
                             "logit_scale": self.logit_scale,
                             "layers": [dict(l) for l in self.layers]}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        return d


def _positive_int(where: str, d: Any, key: str) -> int:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise ConfigError(f"{where}: {key} must be a positive integer, got {v!r}")
    return v


def _number(where: str, d: Any, key: str, positive: bool = False) -> float:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and not v > 0):
        raise ConfigError(f"{where}: {key} must be a {'positive ' if positive else ''}number, "
                          f"got {v!r}")
    return float(v)


def _check_left(where: str, m: Any) -> None:
    heads = _positive_int(where, m, "heads")
    g = _positive_int(where, m, "kv_heads")
    if heads % g:
        raise ConfigError(f"{where}: heads ({heads}) must be a multiple of kv_heads ({g})")
    dim = _positive_int(where, m, "dim")
    _positive_int(where, m, "vdim")
    _number(where, m, "scale", positive=True)
    _positive_int(where + ".mask", m.get("mask"), "size")
    _positive_int(where + ".mask", m.get("mask"), "pool")
    rot = m.get("rot")
    _number(where + ".rot", rot, "base", positive=True)
    dims = _positive_int(where + ".rot", rot, "dims")
    if dims > dim or dims % 2:
        raise ConfigError(f"{where}: rot.dims ({dims}) must be even and at most dim ({dim})")
    sc = rot.get("scaling")
    if sc is not None:
        for key in ("factor", "low", "high", "original"):
            _number(where + ".rot.scaling", sc, key, positive=True)
        if not sc["low"] < sc["high"]:
            raise ConfigError(f"{where}: rot.scaling.low must be below rot.scaling.high")


def _check_right(where: str, m: Any) -> None:
    for key in ("heads", "dim", "vdim"):
        _positive_int(where, m, key)
    _number(where, m, "gate_cap", positive=True)


def _check_mlp(i: int, mlp: Any) -> None:
    where = f"layers[{i}].mlp"
    if mlp is None:
        return
    if not isinstance(mlp, dict) or mlp.get("kind", "moe") != "moe":
        raise ConfigError(f"{where}.kind must be 'moe', got {mlp!r}")
    _positive_int(where + ".expert", mlp.get("expert"), "ff")
    router = mlp.get("router")
    n = _positive_int(where + ".router", router, "experts")
    top = _positive_int(where + ".router", router, "top")
    ident = router.get("identity")
    if ident is not None:
        if isinstance(ident, bool) or not isinstance(ident, int) or ident < 0:
            raise ConfigError(f"{where}.router: identity must be an integer not below zero, got "
                              f"{ident!r}")
        n += ident
    if top > n:
        raise ConfigError(f"{where}.router: top ({top}) exceeds the router's outputs ({n})")
    groups = router.get("groups")
    if groups is not None:
        count = _positive_int(where + ".router.groups", groups, "count")
        keep = _positive_int(where + ".router.groups", groups, "keep")
        if n % count or keep > count or keep * (n // count) < top:
            raise ConfigError(f"{where}.router.groups: {n} outputs do not form {count} equal "
                              f"groups of which {keep} hold {top} experts")
    if mlp.get("shared") is not None:
        _positive_int(where + ".shared", mlp["shared"], "ff")


def gibipel_config_from_dict(raw: Dict[str, Any]) -> GibipelConfig:
    missing = [k for k in ("vocab", "width", "layers", "norm", "embedding", "logit_scale")
               if k not in raw]
    if missing:
        raise ConfigError(f"config.json lacks required keys: {missing}")
    vocab = _positive_int("config", raw, "vocab")
    width = _positive_int("config", raw, "width")
    eps = _number("norm", raw["norm"], "eps", positive=True)
    layers = raw["layers"]
    if not isinstance(layers, list) or not layers:
        raise ConfigError("layers must be a non-empty list")
    for i, layer in enumerate(layers):
        if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
            raise ConfigError(f"layers[{i}].type must be one of {MIXER_TYPES}, got "
                              f"{layer.get('type') if isinstance(layer, dict) else layer!r}")
        m = layer.get("mixer")
        if not isinstance(m, dict):
            raise ConfigError(f"layers[{i}].mixer must be an object")
        for side, check in (("left", _check_left), ("right", _check_right)):
            if not isinstance(m.get(side), dict):
                raise ConfigError(f"layers[{i}].mixer.{side} must be an object")
            check(f"layers[{i}].mixer.{side}", m[side])
            _number(f"layers[{i}].mixer", m, side + "_scale")
        _check_mlp(i, layer.get("mlp"))
    max_positions = raw.get("max_positions", DEFAULT_MAX_POSITIONS)
    if isinstance(max_positions, bool) or not isinstance(max_positions, int) or max_positions <= 0:
        raise ConfigError(f"max_positions must be a positive integer, got {max_positions!r}")
    return GibipelConfig(vocab=vocab, width=width, eps=eps,
                         embedding_scale=_number("embedding", raw["embedding"], "scale"),
                         logit_scale=_number("config", raw, "logit_scale"),
                         layers=[dict(l) for l in layers], max_positions=max_positions,
                         architecture=str(raw.get("architecture", "Gibipel")))


def _mixer_spec(m: Dict[str, Any], eps: float) -> PartSpec:
    left, right = m["left"], m["right"]
    rot = left["rot"]
    position = {"kind": "rotary", "theta": float(rot["base"]), "rotary_dim": int(rot["dims"]),
                "pairing": "half"}
    if rot.get("scaling") is not None:
        position["scaling"] = {k: float(rot["scaling"][k])
                               for k in ("factor", "low", "high", "original")}
    p, r = "mix.left.", "mix.right."
    attention = {
        "num_heads": left["heads"], "num_kv_heads": left["kv_heads"], "head_dim": left["dim"],
        "value_dim": left["vdim"], "scale": float(left["scale"]), "window": int(left["mask"]["size"]),
        "pool": int(left["mask"]["pool"]), "position": position, "sink": p + "sink",
        "qk_norm": {"eps": eps, "q": p + "q.norm", "k": p + "k.norm"},
        "bias": {"q": p + "q.b", "k": p + "k.b", "v": p + "v.b"},
        "names": {"q": p + "q", "k": p + "k", "v": p + "v", "o": p + "o"}}
    memory = {
        "num_heads": right["heads"], "head_dim": right["dim"], "value_dim": right["vdim"],
        "gate_cap": float(right["gate_cap"]), "eps": eps,
        "names": {"q": r + "q", "k": r + "k", "v": r + "v", "gate": r + "g", "i": r + "i",
                  "i_bias": r + "i.b", "f": r + "f", "f_bias": r + "f.b", "norm": r + "norm",
                  "o": r + "o"}}
    return PartSpec("parallel", {"sides": [
        {"name": "left", "kind": "attention", "params": attention, "scale": float(m["left_scale"])},
        {"name": "right", "kind": "matrix_memory", "params": memory,
         "scale": float(m["right_scale"])}]})


def _mlp_spec(mlp: Dict[str, Any]) -> PartSpec:
    router = mlp["router"]
    params: Dict[str, Any] = {
        "num_experts": router["experts"], "top": router["top"],
        "identities": int(router.get("identity") or 0), "intermediate_size": mlp["expert"]["ff"],
        "activation": "silu", "weight_on": "output", "scores": "softmax",
        "correction": "mlp.correction", "renormalize": True, "sum_eps": WEIGHT_SUM_EPS,
        "names": {"router": "mlp.router", "gate": "mlp.e{e}.gate", "up": "mlp.e{e}.up",
                  "down": "mlp.e{e}.down"}}
    if router.get("groups") is not None:
        params["groups"] = {"count": int(router["groups"]["count"]),
                            "keep": int(router["groups"]["keep"]), "score": "best"}
    if mlp.get("shared") is not None:
        params["shared"] = {"intermediate_size": int(mlp["shared"]["ff"]),
                            "names": {"gate": "mlp.shared.gate", "up": "mlp.shared.up",
                                      "down": "mlp.shared.down"}}
    return PartSpec("routed_experts", params)


def build_gibipel_spec(cfg: GibipelConfig) -> ModelSpec:
    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"eps": cfg.eps, "name": name, "scalar": True})

    layers: List[LayerSpec] = []
    for i, layer in enumerate(cfg.layers):
        branches = [BranchSpec("mixer", _mixer_spec(layer["mixer"], cfg.eps),
                               post_norm=norm("norm1"))]
        if layer.get("mlp") is not None:
            branches.append(BranchSpec("feed_forward", _mlp_spec(layer["mlp"]),
                                       post_norm=norm("norm2")))
        layers.append(LayerSpec(f"l{i}.", tuple(branches)))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=cfg.width,
        embedding=PartSpec("token_embedding", {"name": "embed", "scale": cfg.embedding_scale}),
        layers=layers, schedule=[ScheduleEntry(i) for i in range(len(layers))],
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"tied": False, "name": "head", "scale": cfg.logit_scale}),
        max_positions=cfg.max_positions)


register_architecture("Gibipel", gibipel_config_from_dict, build_gibipel_spec)
