"""Sezopel: typed configuration and model plan.

A decoder-only model whose looked-up embedding rows are multiplied by a constant and whose sublayers read the stream as it
is: only what a sublayer gives back is normed, x <- x + norm1(mixer(x)), x <- x + norm2(ff(x)).  Behind the feed-forward
every layer takes in a vector that belongs to the token and the layer, x <- x + norm(proj(gelu(gate(x)) * e)), e the layer's
columns of one table for the whole model.  A layer's mixer is softmax attention (``attention``: grouped-query, heads normed
without a gain and partly rotated, capped scores, one sigmoid gate per head; with ``kv_from`` it reads the keys and values of
an earlier layer's cache) or retention (``retention``: linear attention with a fixed decay per head on rotated queries and
keys, each head's output normed, gated by silu).  The feed-forward (optional) is two matrices with a squared relu between
them.  The model's norm, an output head of its own, capped logits.

This file is all that names the architecture: it reads config.json's keys (``architecture``, ``vocab``, ``width``,
``embedding.scale``, ``logit_softcap``, ``norm.eps``, ``token_side.dim`` and ``layers[i].{type, mixer, mlp}``), turns them into
part specifications, and registers itself.  Tensor names: ``embed``, ``side.embed``, ``head``, ``final.norm`` and under ``l<i>``:
``norm1``, ``norm2``, ``mix.*``, ``mlp.{up, down}``, ``side.{gate, proj, norm}``.
"""

from __future__ import annotations

from dataclasses import dataclass, field

from ..config.errors import ConfigError
from ..config.fields import get_float, get_int, get_str
from ..config.plan import LayerSpec, ModelPlan, PartEntry, PartSpec, RunEntry
from ..config.registry import Architecture, register_architecture

NAME = "Sezopel"
MIXER_TYPES = ("attention", "retention")
MAX_POSITIONS = 1 << 17      # the design itself has no limit; this is the engine's (block tables and rotary tables are sized for it)


def _section(raw: dict, key: str, where: str = "config.json") -> dict:
    v = raw.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: key {key!r} must be an object")
    return v


def _check_rot(m: dict, where: str) -> None:
    if m.get("rot") is None:                             # (no rot: queries and keys are not rotated)
        return
    rot = _section(m, "rot", where)
    get_float(rot, "base")
    if get_int(rot, "dims", minimum=0) % 2 or rot["dims"] > m["dim"]:
        raise ConfigError(f"{where}.rot.dims={rot['dims']} must be even and at most dim={m['dim']}")


def _check_mixer(i: int, typ: str, m: dict, layers: list) -> None:
    where = f"config.json: layers[{i}].mixer"
    for k in ("heads", "dim", "vdim"):
        get_int(m, k)
    _check_rot(m, where)
    if typ == "retention":
        d = m.get("decay")
        if not isinstance(d, list) or len(d) != m["heads"] or any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in d):
            raise ConfigError(f"{where}.decay must list one number per head ({m['heads']})")
        return
    if m["heads"] % get_int(m, "kv_heads"):
        raise ConfigError(f"{where}: heads={m['heads']} is no multiple of kv_heads={m['kv_heads']}")
    get_float(m, "scale")
    if m.get("softcap") is not None:                     # (no softcap: the scores stay as they are)
        get_float(m, "softcap")
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


def _check_mlp(i: int, mlp: dict) -> None:
    if get_str(mlp, "kind") != "dense":
        raise ConfigError(f"config.json: layers[{i}].mlp.kind={mlp['kind']!r}; this design has 'dense'")
    get_int(mlp, "ff")


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass(frozen=True)
class SezopelConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float = 1.0
    logit_softcap: float | None = None     # (None: the logits stay as they are)
    side_dim: int | None = None            # of the tokens' own vectors, per layer (None: no such term)
    layers: tuple = field(default_factory=tuple)
    architecture: str = NAME

    @classmethod
    def from_dict(cls, raw: dict) -> "SezopelConfig":
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
        optional = lambda section, key, get: get(_section(raw, section), key) if raw.get(section) is not None else None
        scale = optional("embedding", "scale", lambda d, k: get_float(d, k, 1.0, positive=False))
        return cls(vocab=get_int(raw, "vocab"), width=get_int(raw, "width"), norm_eps=get_float(_section(raw, "norm"), "eps"),
                   embedding_scale=1.0 if scale is None else scale,
                   logit_softcap=get_float(raw, "logit_softcap") if raw.get("logit_softcap") is not None else None,
                   side_dim=optional("token_side", "dim", get_int), layers=tuple(layers))

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "embedding": {"scale": self.embedding_scale},
             "layers": [{"type": l.type, "mixer": dict(l.mixer), "mlp": dict(l.mlp) if l.mlp is not None else None}
                        for l in self.layers]}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.side_dim is not None:
            d["token_side"] = {"dim": self.side_dim}
        return d


def _mixer_spec(cfg: SezopelConfig, l: LayerConfig) -> PartSpec:
    m, rot = l.mixer, l.mixer.get("rot")
    rotary = {"theta": rot["base"], "rotary_dim": rot["dims"], "max_positions": MAX_POSITIONS} if rot and rot["dims"] else None
    common = {"hidden_size": cfg.width, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "eps": cfg.norm_eps, "rotary": rotary}
    if l.type == "retention":
        return PartSpec("retention", dict(common, decay=tuple(float(d) for d in m["decay"])))
    return PartSpec("normed_attention", dict(
        common, kv_heads=m["kv_heads"], scale=m["scale"], softcap=m.get("softcap"), head_gain=False, head_gate=True,
        shared_kv=m.get("kv_from") is not None, max_positions=MAX_POSITIONS))


def plan(cfg: SezopelConfig) -> ModelPlan:
    norm = PartSpec("group_rmsnorm", {"size": cfg.width, "groups": 1, "eps": cfg.norm_eps})
    layers, runs = [], []
    for i, l in enumerate(cfg.layers):
        parts = {"mixer": PartEntry("mixer", _mixer_spec(cfg, l), "mix"), "mixer_post": PartEntry("norm", norm, "norm1")}
        if l.mlp is not None:
            spec = PartSpec("plain_dense", {"hidden_size": cfg.width, "intermediate_size": l.mlp["ff"], "activation": "relu2"})
            parts.update(ffn=PartEntry("feed_forward", spec, "mlp"), ffn_post=PartEntry("norm", norm, "norm2"))
        if cfg.side_dim is not None:
            spec = PartSpec("token_side", {"hidden_size": cfg.width, "dim": cfg.side_dim, "offset": i * cfg.side_dim})
            parts.update(side=PartEntry("feed_forward", spec, "side"), side_post=PartEntry("norm", norm, "side.norm"))
        layers.append(LayerSpec(prefix=f"l{i}", parts=parts, block="output_norm"))
        # a layer that reads another layer's keys and values borrows that run's pages (and writes none)
        runs.append(RunEntry(i, cache_from=l.mixer.get("kv_from") if l.type == "attention" else None))
    p = ModelPlan(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embedding_name="embed", layers=tuple(layers), run_list=tuple(runs),
        final_norm=norm, final_norm_name="final.norm", head_name="head", position=None, embedding_scale=cfg.embedding_scale,
        token_table_name="side.embed" if cfg.side_dim is not None else None,
        token_table_width=len(cfg.layers) * cfg.side_dim if cfg.side_dim is not None else 0, logit_softcap=cfg.logit_softcap,
        ignored_names=tuple(f"l{i}.norm2" for i, l in enumerate(cfg.layers) if l.mlp is None))
    p.validate()
    return p


def config_from_recipe(t: dict) -> dict:
    """A recipe's inline geometry carries config.json's own keys (``vocab``, ``width``, ``norm``, ``layers``, optionally
    ``embedding``, ``token_side``, ``logit_softcap``); a missing one raises KeyError naming it."""
    cfg = {k: t[k] for k in ("vocab", "width", "norm", "layers")}
    cfg.update({k: t[k] for k in ("embedding", "token_side", "logit_softcap") if t.get(k) is not None})
    cfg["architecture"] = NAME
    return cfg


register_architecture(Architecture(name=NAME, config_cls=SezopelConfig, plan=plan, aliases=("sezopel",),
                                   config_from_recipe=config_from_recipe), replace=True)
