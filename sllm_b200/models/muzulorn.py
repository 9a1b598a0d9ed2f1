"""Muzulorn: typed configuration and model plan.

A decoder-only model.  The embedding takes in a row of a table by the pair (token before, token), folded into buckets; the stream is
``streams`` copies that every sublayer reads as a weighted sum and mixes anew (hyper-connections; a term joins them times
``residual_mult``); norms keep their gain around zero.  A layer's mixer is softmax attention without rotation (``attention``: biased
projections, norms over the whole query and key, a query factor that grows with the position, capped scores, a learned bias by
bucketed distance; with ``kv_from`` it reads the keys and values of an earlier layer's cache), attention over a small cached latent
(``latent_attention``: queries through a latent of their own, one rotated key part for all heads, a sliding window, a sink, a gate per
output channel) or a state-space recurrence (``mamba2``).  The feed-forward (optional) is two matrices with the exact gelu between
them, or a mixture of gated experts beside a gated shared one.  The model's norm and an output head of its own follow.

This file is all that names the architecture: it reads config.json's keys (``architecture``, ``vocab``, ``width``, ``streams``,
``residual_mult``, ``norm.eps``, ``embedding.bigram.{buckets, mul_prev, mul_cur}`` and ``layers[i].{type, mixer, mlp}``), turns them
into part specifications, and registers itself.  Tensor names: ``embed``, ``bigram``, ``head``, ``final.norm`` and under ``l<i>``:
``norm1``, ``norm2``, ``hc1.{in, out, mix}``, ``hc2.*``, ``mix.*``, ``mlp.*``.
"""

from __future__ import annotations

from dataclasses import dataclass, field

from ..config.errors import ConfigError
from ..config.fields import get_float, get_int, get_str
from ..config.plan import LayerSpec, ModelPlan, PartEntry, PartSpec, RunEntry, TokenPairs
from ..config.registry import Architecture, register_architecture

NAME = "Muzulorn"
MIXER_TYPES = ("attention", "latent_attention", "mamba2")
MAX_POSITIONS = 1 << 17      # the design itself has no limit; this is the engine's (block tables and rotary tables are sized for it)


def _section(raw: dict, key: str, where: str = "config.json") -> dict:
    v = raw.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: key {key!r} must be an object")
    return v


def _check_attention(i: int, m: dict, layers: list, where: str) -> None:
    for k in ("heads", "kv_heads", "dim", "vdim", "bias_max"):
        get_int(m, k)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: heads={m['heads']} is no multiple of kv_heads={m['kv_heads']}")
    get_float(m, "scale")
    if m.get("softcap") is not None:                     # (no softcap: the scores stay as they are)
        get_float(m, "softcap")
    if m.get("q_temp") is not None:
        t = _section(m, "q_temp", where)
        get_float(t, "coef", positive=False), get_int(t, "every")
    src = m.get("kv_from")
    if src is not None:
        if isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < i:
            raise ConfigError(f"{where}.kv_from={src!r} must name an earlier layer")
        other = layers[src]
        if other.type != "attention" or other.mixer.get("kv_from") is not None:
            raise ConfigError(f"{where}.kv_from={src}: that layer has no keys and values of its own")
        for k in ("kv_heads", "dim", "vdim"):
            if other.mixer[k] != m[k]:
                raise ConfigError(f"{where}.kv_from={src}: {k} differs ({other.mixer[k]!r} there, {m[k]!r} here)")


def _check_mixer(i: int, typ: str, m: dict, layers: list) -> None:
    where = f"config.json: layers[{i}].mixer"
    if typ == "attention":
        return _check_attention(i, m, layers, where)
    if typ == "mamba2":
        for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
            get_int(m, k)
        if m["heads"] % m["groups"] or (m["heads"] * m["vdim"]) % m["norm_groups"]:
            raise ConfigError(f"{where}: groups={m['groups']} must divide heads={m['heads']}, norm_groups={m['norm_groups']} heads * vdim")
        return
    for k in ("heads", "dim", "vdim", "q_rank", "kv_rank"):
        get_int(m, k)
    get_int(m, "rot_dim", minimum=0), get_float(m, "scale")
    if m["rot_dim"] and m.get("rot") is not None:
        rot = _section(m, "rot", where)
        get_float(rot, "base")
        if get_int(rot, "dims", minimum=0) % 2 or rot["dims"] > m["rot_dim"]:
            raise ConfigError(f"{where}.rot.dims={rot['dims']} must be even and at most rot_dim={m['rot_dim']}")
    if m.get("mask") is not None:                        # (no mask: all earlier tokens)
        get_int(_section(m, "mask", where), "size")


def _check_mlp(i: int, mlp: dict) -> None:
    where = f"config.json: layers[{i}].mlp"
    kind = get_str(mlp, "kind")
    if kind == "dense":
        get_int(mlp, "ff")
    elif kind == "moe":
        get_int(_section(mlp, "expert", where), "ff")
        r = _section(mlp, "router", where)
        if get_int(r, "top") > get_int(r, "experts"):
            raise ConfigError(f"{where}.router: top={r['top']} of {r['experts']} experts cannot be chosen")
        if mlp.get("shared") is not None:
            get_int(_section(mlp, "shared", where), "ff")
    else:
        raise ConfigError(f"{where}.kind={kind!r}; this design has 'dense' and 'moe'")


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass(frozen=True)
class MuzulornConfig:
    vocab: int
    width: int
    norm_eps: float
    streams: int = 1
    residual_mult: float = 1.0
    bigram: dict | None = None       # buckets, mul_prev, mul_cur (None: the embedding's rows alone)
    layers: tuple = field(default_factory=tuple)
    architecture: str = NAME

    @classmethod
    def from_dict(cls, raw: dict) -> "MuzulornConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: key 'layers' must be a non-empty list")
        layers: list = []
        for i, entry in enumerate(layers_raw):
            if not isinstance(entry, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            typ = get_str(entry, "type")
            if typ not in MIXER_TYPES:
                raise ConfigError(f"config.json: layers[{i}].type={typ!r}; this design has {MIXER_TYPES}")
            mixer = dict(_section(entry, "mixer", f"config.json: layers[{i}]"))
            _check_mixer(i, typ, mixer, layers)
            mlp = entry.get("mlp")
            if mlp is not None:
                mlp = dict(_section(entry, "mlp", f"config.json: layers[{i}]"))
                _check_mlp(i, mlp)
            layers.append(LayerConfig(typ, mixer, mlp))
        bigram = None
        if raw.get("embedding") is not None and _section(raw, "embedding").get("bigram") is not None:
            b = _section(raw["embedding"], "bigram", "config.json: embedding")
            bigram = {"buckets": get_int(b, "buckets"), "mul_prev": get_int(b, "mul_prev", minimum=0), "mul_cur": get_int(b, "mul_cur", minimum=0)}
        return cls(vocab=get_int(raw, "vocab"), width=get_int(raw, "width"), norm_eps=get_float(_section(raw, "norm"), "eps"),
                   streams=get_int(raw, "streams"), residual_mult=get_float(raw, "residual_mult", positive=False), bigram=bigram,
                   layers=tuple(layers))

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "streams": self.streams, "residual_mult": self.residual_mult,
             "layers": [{"type": l.type, "mixer": dict(l.mixer), "mlp": dict(l.mlp) if l.mlp is not None else None}
                        for l in self.layers]}
        if self.bigram is not None:
            d["embedding"] = {"bigram": dict(self.bigram)}
        return d


def _mixer_spec(cfg: MuzulornConfig, l: LayerConfig) -> PartSpec:
    m, W, eps = l.mixer, cfg.width, cfg.norm_eps
    if l.type == "mamba2":
        return PartSpec("mamba2", dict({k: m[k] for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}, hidden_size=W, eps=eps))
    if l.type == "latent_attention":
        rot = m.get("rot") if m["rot_dim"] else None
        return PartSpec("latent_attention", {
            "hidden_size": W, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "q_rank": m["q_rank"], "kv_rank": m["kv_rank"],
            "scale": m["scale"], "eps": eps, "gate": "element", "sink": True, "rot_dim": m["rot_dim"],
            "window": m["mask"]["size"] if m.get("mask") is not None else None,
            "rotary": {"theta": rot["base"], "rotary_dim": rot["dims"], "interleaved": True, "max_positions": MAX_POSITIONS}
            if rot and rot["dims"] else None})
    return PartSpec("normed_attention", {
        "hidden_size": W, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "scale": m["scale"],
        "eps": eps, "norm_over": "projection", "bias": True, "out_bias": True, "softcap": m.get("softcap"), "q_temp": m.get("q_temp"),
        "distance_bias": m["bias_max"], "shared_kv": m.get("kv_from") is not None, "rotary": None, "max_positions": MAX_POSITIONS})


def _ffn_spec(cfg: MuzulornConfig, mlp: dict) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("plain_dense", {"hidden_size": cfg.width, "intermediate_size": mlp["ff"], "activation": "gelu"})
    return PartSpec("gated_experts", {
        "hidden_size": cfg.width, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"], "expert_ff": mlp["expert"]["ff"],
        "activation": "silu", "router_bias": True, "shared_ff": mlp["shared"]["ff"] if mlp.get("shared") is not None else 0})


def plan(cfg: MuzulornConfig) -> ModelPlan:
    norm = PartSpec("group_rmsnorm", {"size": cfg.width, "groups": 1, "eps": cfg.norm_eps, "offset": 1.0})
    hc = PartSpec("hyper_connection", {"streams": cfg.streams, "mult": cfg.residual_mult})
    layers, runs, unused = [], [], []
    for i, l in enumerate(cfg.layers):
        parts = {"mixer_norm": PartEntry("norm", norm, "norm1"), "mixer": PartEntry("mixer", _mixer_spec(cfg, l), "mix"),
                 "mixer_hc": PartEntry("shift", hc, "hc1")}
        if l.mlp is not None:
            parts.update(ffn_norm=PartEntry("norm", norm, "norm2"), ffn=PartEntry("feed_forward", _ffn_spec(cfg, l.mlp), "mlp"),
                         ffn_hc=PartEntry("shift", hc, "hc2"))
        else:
            unused += [f"l{i}.norm2", f"l{i}.hc2.in", f"l{i}.hc2.out", f"l{i}.hc2.mix"]
        layers.append(LayerSpec(prefix=f"l{i}", parts=parts, block="hyper_connected"))
        # a layer that reads another layer's keys and values borrows that run's pages (and writes none)
        runs.append(RunEntry(i, cache_from=l.mixer.get("kv_from") if l.type == "attention" else None))
    p = ModelPlan(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embedding_name="embed", layers=tuple(layers), run_list=tuple(runs), final_norm=norm, final_norm_name="final.norm",
        head_name="head", position=None, streams=cfg.streams,
        token_pairs=TokenPairs("bigram", cfg.bigram["buckets"], cfg.bigram["mul_prev"], cfg.bigram["mul_cur"]) if cfg.bigram else None,
        ignored_names=tuple(unused))
    p.validate()
    return p


def config_from_recipe(t: dict) -> dict:
    """A recipe's inline geometry carries config.json's own keys (``vocab``, ``width``, ``norm``, ``streams``, ``residual_mult``,
    ``layers``, optionally ``embedding``); a missing one raises KeyError naming it."""
    cfg = {k: t[k] for k in ("vocab", "width", "norm", "streams", "residual_mult", "layers")}
    if t.get("embedding") is not None:
        cfg["embedding"] = t["embedding"]
    cfg["architecture"] = NAME
    return cfg


register_architecture(Architecture(name=NAME, config_cls=MuzulornConfig, plan=plan, aliases=("muzulorn",),
                                   config_from_recipe=config_from_recipe), replace=True)
