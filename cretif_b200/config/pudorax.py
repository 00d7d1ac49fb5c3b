"""Typed configuration of the Pudorax decoder, read from config.json, and its ModelSpec.

A Pudorax checkpoint's config.json names its class with ``"architecture": "Pudorax"`` and
describes the model as a list of layers, each with sizes of its own:

=====================  ========================================================================
key                    meaning
=====================  ========================================================================
vocab, width           vocabulary and residual width
norm.eps               eps of every norm of the model
embedding.scale        factor on the embedding's rows
layers[i].type         ``attention`` or ``mamba2``
layers[i].mixer        attention: heads, kv_heads, dim, vdim, scale, conv (taps), rot {base, dims};
                       mamba2: heads, vdim, state, groups, norm_groups, conv (taps)
layers[i].mlp          ``{"kind": "moe", "expert": {"ff": F, "limit": c}, "router": {"experts": E,
                       "top": k}, "shared": {"ff": Fs, "limit": cs}}`` (shared optional), or null
loop                   (optional) {start, stop, times}: layers start .. stop - 1 run ``times`` times
                       in a row, each pass behind a merge of the stream with the model's input
token_side             (optional) {dim}: width of the second embedding's part of every layer
logit_softcap          (optional) c: logits leave as ``c tanh(logits / c)``
max_positions          (optional) longest sequence; the design itself has no limit
=====================  ========================================================================

The blocks are pre-norm with layer norms.  Attention: q, k and v pass a short convolution, q and k are
normed over the whole projection and rotated (the first dims channels of a head, in pairs of neighbours),
every key is seen, the heads are gated channel by channel.  mamba2: the Mamba-2 recurrence with a gated
norm.  The feed-forward's experts have clamped gates and are weighted by the softmax over the chosen
router outputs.  Behind the feed-forward every layer looks at its token once more (parts/token_side.py).
Every pass of the loop has its own cache and state.  Tensors are named ``l<i>.mix.*``, ``l<i>.mlp.*``
(``e<n>.gate/up/down``, ``router``, ``router.b``, ``shared.gate/up/down``), ``l<i>.side.gate/proj/norm``,
``l<i>.norm1/2`` (and ``.b``), ``embed``, ``side.embed``, ``loop.in``, ``final.norm`` and ``head``.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .registry import ConfigError, register_architecture
from .spec import BranchSpec, LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MIXER_TYPES = ("attention", "mamba2")
DEFAULT_MAX_POSITIONS = 1 << 20
GATE_SLOPE = 1.702                       # of an expert's gate: g sigmoid(GATE_SLOPE g)
UP_OFFSET = 1.0                          # added to an expert's other product


@dataclass
class PudoraxConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float = 1.0
    layers: List[Dict[str, Any]] = field(default_factory=list)
    loop: Optional[Dict[str, int]] = None
    token_side: Optional[int] = None     # dim
    logit_softcap: Optional[float] = None
    max_positions: int = DEFAULT_MAX_POSITIONS
    architecture: str = "Pudorax"

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab,
                             "width": self.width, "norm": {"eps": self.eps},
                             "embedding": {"scale": self.embedding_scale},
                             "layers": [dict(l) for l in self.layers]}
        if self.loop is not None:
            d["loop"] = dict(self.loop)
        if self.token_side is not None:
            d["token_side"] = {"dim": self.token_side}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        return d


def _integer(where: str, d: Any, key: str, least: int = 1) -> int:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ConfigError(f"{where}: {key} must be an integer of at least {least}, got {v!r}")
    return v


def _number(where: str, d: Any, key: str, positive: bool = False) -> float:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and not v > 0):
        raise ConfigError(f"{where}: {key} must be a {'positive ' if positive else ''}number, "
                          f"got {v!r}")
    return float(v)


def _check_attention(where: str, m: Any) -> None:
    heads, g = _integer(where, m, "heads"), _integer(where, m, "kv_heads")
    if heads % g:
        raise ConfigError(f"{where}: heads ({heads}) must be a multiple of kv_heads ({g})")
    dim = _integer(where, m, "dim")
    _integer(where, m, "vdim")
    _integer(where, m, "conv")
    _number(where, m, "scale", positive=True)
    _number(where + ".rot", m.get("rot"), "base", positive=True)
    dims = _integer(where + ".rot", m.get("rot"), "dims", least=0)
    if dims > dim or dims % 2:
        raise ConfigError(f"{where}: rot.dims ({dims}) must be even and at most dim ({dim})")


def _check_mamba2(where: str, m: Any) -> None:
    heads, vdim = _integer(where, m, "heads"), _integer(where, m, "vdim")
    groups, parts = _integer(where, m, "groups"), _integer(where, m, "norm_groups")
    _integer(where, m, "state")
    _integer(where, m, "conv")
    if heads % groups:
        raise ConfigError(f"{where}: heads ({heads}) must be a multiple of groups ({groups})")
    if heads * vdim % parts:
        raise ConfigError(f"{where}: heads x vdim ({heads * vdim}) must be a multiple of norm_groups "
                          f"({parts})")


def _check_mlp(where: str, mlp: Any) -> None:
    if mlp is None:
        return
    if not isinstance(mlp, dict) or mlp.get("kind", "moe") != "moe":
        raise ConfigError(f"{where}.kind must be 'moe', got {mlp!r}")
    n = _integer(where + ".router", mlp.get("router"), "experts")
    top = _integer(where + ".router", mlp.get("router"), "top")
    if top > n:
        raise ConfigError(f"{where}.router: top ({top}) exceeds the number of experts ({n})")
    for key in ("expert", "shared"):
        if key == "expert" or mlp.get(key) is not None:
            _integer(f"{where}.{key}", mlp.get(key), "ff")
            _number(f"{where}.{key}", mlp.get(key), "limit", positive=True)


def pudorax_config_from_dict(raw: Dict[str, Any]) -> PudoraxConfig:
    missing = [k for k in ("vocab", "width", "layers", "norm", "embedding") if k not in raw]
    if missing:
        raise ConfigError(f"config.json lacks required keys: {missing}")
    layers = raw["layers"]
    if not isinstance(layers, list) or not layers:
        raise ConfigError("layers must be a non-empty list")
    for i, layer in enumerate(layers):
        if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
            raise ConfigError(f"layers[{i}].type must be one of {MIXER_TYPES}, got "
                              f"{layer.get('type') if isinstance(layer, dict) else layer!r}")
        if not isinstance(layer.get("mixer"), dict):
            raise ConfigError(f"layers[{i}].mixer must be an object")
        check = _check_attention if layer["type"] == "attention" else _check_mamba2
        check(f"layers[{i}].mixer", layer["mixer"])
        _check_mlp(f"layers[{i}].mlp", layer.get("mlp"))
    loop = raw.get("loop")
    if loop is not None:
        start, stop = _integer("loop", loop, "start", least=0), _integer("loop", loop, "stop")
        _integer("loop", loop, "times")
        if not start < stop <= len(layers):
            raise ConfigError(f"loop: start ({start}) and stop ({stop}) must enclose layers of the "
                              f"{len(layers)} there are")
        loop = {k: loop[k] for k in ("start", "stop", "times")}
    side = raw.get("token_side")
    cap = raw.get("logit_softcap")
    max_positions = raw.get("max_positions", DEFAULT_MAX_POSITIONS)
    if isinstance(max_positions, bool) or not isinstance(max_positions, int) or max_positions <= 0:
        raise ConfigError(f"max_positions must be a positive integer, got {max_positions!r}")
    return PudoraxConfig(
        vocab=_integer("config", raw, "vocab"), width=_integer("config", raw, "width"),
        eps=_number("norm", raw["norm"], "eps", positive=True),
        embedding_scale=_number("embedding", raw["embedding"], "scale"),
        layers=[dict(l) for l in layers], loop=loop,
        token_side=None if side is None else _integer("token_side", side, "dim"),
        logit_softcap=None if cap is None else _number("config", raw, "logit_softcap", positive=True),
        max_positions=max_positions, architecture=str(raw.get("architecture", "Pudorax")))


def _attention_spec(m: Dict[str, Any], eps: float) -> PartSpec:
    p = "mix."
    rot = m["rot"]
    params: Dict[str, Any] = {
        "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
        "value_dim": m["vdim"], "scale": float(m["scale"]), "window": 0,
        "conv": {"taps": int(m["conv"]), "q": p + "q.conv", "k": p + "k.conv", "v": p + "v.conv"},
        "qk_norm": {"eps": eps, "q": p + "q.norm", "k": p + "k.norm"}, "out_gate": p + "g",
        "names": {"q": p + "q", "k": p + "k", "v": p + "v", "o": p + "o"}}
    if rot["dims"]:
        params["position"] = {"kind": "rotary", "theta": float(rot["base"]),
                              "rotary_dim": int(rot["dims"]), "pairing": "interleaved"}
    return PartSpec("attention", params)


def _mamba2_spec(m: Dict[str, Any], eps: float) -> PartSpec:
    p = "mix."
    return PartSpec("state_space", {
        "num_heads": m["heads"], "groups": m["groups"], "state_dim": m["state"],
        "value_dim": m["vdim"], "conv_taps": int(m["conv"]), "norm_groups": m["norm_groups"],
        "eps": eps,
        "names": {"in": p + "in", "conv": p + "conv", "conv_bias": p + "conv.b",
                  "dt_bias": p + "dt_bias", "A_log": p + "A_log", "D": p + "D", "norm": p + "norm",
                  "o": p + "o"}})


def _clamp(limit) -> Dict[str, float]:
    return {"limit": float(limit), "slope": GATE_SLOPE, "offset": UP_OFFSET}


def _mlp_spec(mlp: Dict[str, Any]) -> PartSpec:
    params: Dict[str, Any] = {
        "num_experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
        "intermediate_size": mlp["expert"]["ff"], "clamp": _clamp(mlp["expert"]["limit"]),
        "weight_on": "output", "scores": "softmax_chosen", "renormalize": True,
        "router_bias": "mlp.router.b",
        "names": {"router": "mlp.router", "gate": "mlp.e{e}.gate", "up": "mlp.e{e}.up",
                  "down": "mlp.e{e}.down"}}
    if mlp.get("shared") is not None:
        params["shared"] = {"intermediate_size": int(mlp["shared"]["ff"]),
                            "clamp": _clamp(mlp["shared"]["limit"]),
                            "names": {"gate": "mlp.shared.gate", "up": "mlp.shared.up",
                                      "down": "mlp.shared.down"}}
    return PartSpec("routed_experts", params)


def _schedule(cfg: PudoraxConfig) -> List[ScheduleEntry]:
    n = len(cfg.layers)
    if cfg.loop is None:
        return [ScheduleEntry(i) for i in range(n)]
    start, stop = cfg.loop["start"], cfg.loop["stop"]
    one_pass = [ScheduleEntry(i, merge_input=i == start) for i in range(start, stop)]
    return [ScheduleEntry(i) for i in range(start)] + one_pass * cfg.loop["times"] \
        + [ScheduleEntry(i) for i in range(stop, n)]


def build_pudorax_spec(cfg: PudoraxConfig) -> ModelSpec:
    def norm(name: str) -> PartSpec:
        return PartSpec("layernorm", {"eps": cfg.eps, "name": name})

    layers: List[LayerSpec] = []
    for i, layer in enumerate(cfg.layers):
        mixer = (_attention_spec if layer["type"] == "attention" else _mamba2_spec)(layer["mixer"],
                                                                                    cfg.eps)
        branches = [BranchSpec("mixer", mixer, norm=norm("norm1"))]
        if layer.get("mlp") is not None:
            branches.append(BranchSpec("feed_forward", _mlp_spec(layer["mlp"]), norm=norm("norm2")))
        if cfg.token_side is not None:
            branches.append(BranchSpec("feed_forward", PartSpec("token_side", {
                "dim": cfg.token_side, "part": i, "parts": len(cfg.layers), "vocab_size": cfg.vocab,
                "activation": "gelu_tanh",
                "names": {"table": "/side.embed", "gate": "side.gate", "proj": "side.proj"}}),
                post_norm=PartSpec("rmsnorm", {"eps": cfg.eps, "name": "side.norm"})))
        layers.append(LayerSpec(f"l{i}.", tuple(branches)))
    head: Dict[str, Any] = {"tied": False, "name": "head"}
    if cfg.logit_softcap is not None:
        head["softcap"] = cfg.logit_softcap
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=cfg.width,
        embedding=PartSpec("token_embedding", {"name": "embed", "scale": cfg.embedding_scale}),
        layers=layers, schedule=_schedule(cfg), final_norm=norm("final.norm"),
        head=PartSpec("linear_head", head), max_positions=cfg.max_positions,
        merge=None if cfg.loop is None else PartSpec("linear_merge", {"name": "loop.in"}))


register_architecture("Pudorax", pudorax_config_from_dict, build_pudorax_spec)
