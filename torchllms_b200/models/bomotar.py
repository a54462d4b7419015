"""Bomotar as an :class:`~torchllms_b200.config.registry.Architecture`.

A small decoder whose ``config.json`` lists its layers one by one; every layer names its mixer
(``parallel``) with that mixer's own sizes, and its feed-forward (``dense``, ``moe`` or none).  A layer with
``weights_of`` runs another layer's weights with a cache and a state of its own.  What the design fixes
and no file carries:

* the stream starts as the embedding table's row plus a row chosen by the pair of the token and the one
  before it (``embedding.bigram``); the head is a matrix of its own;
* a layer is ``x += m * norm1b(mixer(norm1(x)))``, ``x += m * norm2b(ff(norm2(x)))`` with ``m = residual_mult`` and plain
  weights on the RMS norms;
* ``parallel``: ``left_scale * left + right_scale * right``, both reading the same rows;
* left: causal softmax attention with grouped key/value heads, a short convolution over time on every channel
  of q, k and v, rotary positions (pairs ``i``, ``i + rot.dims / 2``; frequencies rescaled along a ramp with
  ``rot.scaling``), an element-wise sigmoid gate ahead of the output projection;
* right: the gated delta rule with a decay per head and key coordinate, short convolutions of q, k and v with
  ``silu``, unit q and k, q scaled by ``dim^-1/2``, low-rank projections for the decay and for the sigmoid output
  gate, an RMS norm per head with one shared weight;
* ``dense``: ``down(gelu_tanh(up x))``;  ``moe``: experts ``down(silu(gate x) * up x)``, softmax scores, a correction that
  steers the choice alone, groups of neighbours scored by their best choice score, weights as the softmax gives them.

This module only describes: it reads the configuration, names the generic parts with their
numbers (:func:`build_spec`), and maps the checkpoint's tensor names to the parts' own.
"""

from __future__ import annotations

import re
from dataclasses import dataclass
from typing import Any, Dict, Iterator, List, Mapping, Optional, Tuple

import torch

from ..config.model_config import ConfigError, ModelConfig, require_key
from ..config.registry import Architecture, register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PairTable, RunEntry, part
from ..weights.loader import LazyTensor

NAME = "Bomotar"

# The design has no longest sequence (rotary positions, recurrent states); tables are made this long unless
# whoever builds the engine asks for more.
DEFAULT_MAX_POSITIONS = 32768

UNIT_EPS = 1e-6               # inside the root that makes q and k of the delta rule unit vectors
PAIR_TENSOR = "bigram"


def _object(raw: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"{where}: key '{key}' must be an object")
    return value


def _positive(obj: Any, keys: Tuple[str, ...], at: str) -> None:
    for key in keys:
        if getattr(obj, key) <= 0:
            raise ConfigError(f"{at}: '{key}' must be positive, got {getattr(obj, key)}")


@dataclass(frozen=True)
class RampScaling:
    """Rotary frequencies rescaled along a ramp: see :func:`torchllms_b200.parts.rope.ramp_scaled`."""

    factor: float
    original: float
    fast: float
    slow: float

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "RampScaling":
        return cls(*(require_key(raw, key, float, where) for key in ("factor", "original", "fast", "slow")))

    def to_dict(self) -> Dict[str, Any]:
        return {"factor": self.factor, "fast": self.fast, "original": self.original, "slow": self.slow}


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: int
    rot_dims: int
    rot_base: float
    scaling: Optional[RampScaling] = None

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "AttentionConfig":
        rot = _object(raw, "rot", where)
        scaling = _object(rot, "scaling", f"{where}.rot") if rot.get("scaling") is not None else None
        return cls(heads=require_key(raw, "heads", int, where), kv_heads=require_key(raw, "kv_heads", int, where),
                   dim=require_key(raw, "dim", int, where), vdim=require_key(raw, "vdim", int, where),
                   scale=require_key(raw, "scale", float, where), conv=require_key(raw, "conv", int, where),
                   rot_dims=require_key(rot, "dims", int, f"{where}.rot"), rot_base=require_key(rot, "base", float, f"{where}.rot"),
                   scaling=None if scaling is None else RampScaling.from_dict(scaling, f"{where}.rot.scaling"))

    def to_dict(self) -> Dict[str, Any]:
        rot: Dict[str, Any] = {"base": self.rot_base, "dims": self.rot_dims}
        if self.scaling is not None:
            rot["scaling"] = self.scaling.to_dict()
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "rot": rot, "scale": self.scale,
                "vdim": self.vdim}

    def validate(self, at: str) -> None:
        _positive(self, ("heads", "kv_heads", "dim", "vdim", "conv"), at)
        if self.heads % self.kv_heads != 0:
            raise ConfigError(f"{at}: 'heads' ({self.heads}) must be a multiple of 'kv_heads' ({self.kv_heads})")
        if self.rot_dims < 0 or self.rot_dims % 2 or self.rot_dims > self.dim:
            raise ConfigError(f"{at}: 'rot.dims' must be even and at most 'dim' ({self.dim}), got {self.rot_dims}")
        if not self.rot_base > 0:
            raise ConfigError(f"{at}: 'rot.base' must be positive")
        s = self.scaling
        if s is not None and (min(s.factor, s.original, s.fast, s.slow) <= 0 or self.rot_base == 1):
            raise ConfigError(f"{at}: 'rot.scaling' needs positive numbers and a 'rot.base' other than one")


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "DeltaConfig":
        return cls(*(require_key(raw, key, int, where) for key in ("heads", "kv_heads", "dim", "vdim", "conv")))

    def to_dict(self) -> Dict[str, Any]:
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}

    def validate(self, at: str) -> None:
        _positive(self, ("heads", "kv_heads", "dim", "vdim", "conv"), at)
        if self.heads % self.kv_heads != 0:
            raise ConfigError(f"{at}: 'heads' ({self.heads}) must be a multiple of 'kv_heads' ({self.kv_heads})")


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: DeltaConfig
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "ParallelConfig":
        return cls(AttentionConfig.from_dict(_object(raw, "left", where), f"{where}.left"),
                   DeltaConfig.from_dict(_object(raw, "right", where), f"{where}.right"),
                   require_key(raw, "left_scale", float, where), require_key(raw, "right_scale", float, where))

    def to_dict(self) -> Dict[str, Any]:
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": self.right.to_dict(), "right_scale": self.right_scale}

    def validate(self, at: str) -> None:
        self.left.validate(f"{at}.left")
        self.right.validate(f"{at}.right")


@dataclass(frozen=True)
class MlpConfig:
    kind: str                       # "dense" or "moe"
    ff: int                         # dense: the hidden size; moe: one expert's
    experts: int = 0
    top: int = 0
    groups: int = 1
    keep_groups: int = 1

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "MlpConfig":
        kind = require_key(raw, "kind", str, where)
        if kind == "dense":
            return cls(kind, require_key(raw, "ff", int, where))
        if kind == "moe":
            router = _object(raw, "router", where)
            count = keep = 1
            if router.get("groups") is not None:
                groups = _object(router, "groups", f"{where}.router")
                count, keep = (require_key(groups, key, int, f"{where}.router.groups") for key in ("count", "keep"))
            return cls(kind, require_key(_object(raw, "expert", where), "ff", int, f"{where}.expert"),
                       experts=require_key(router, "experts", int, f"{where}.router"),
                       top=require_key(router, "top", int, f"{where}.router"), groups=count, keep_groups=keep)
        raise ConfigError(f"{where}: unknown feed-forward kind {kind!r}; known: dense, moe")

    def to_dict(self) -> Dict[str, Any]:
        if self.kind == "dense":
            return {"ff": self.ff, "kind": "dense"}
        return {"expert": {"ff": self.ff}, "kind": "moe",
                "router": {"experts": self.experts, "groups": {"count": self.groups, "keep": self.keep_groups}, "top": self.top}}

    def validate(self, at: str) -> None:
        if self.ff <= 0:
            raise ConfigError(f"{at}: the feed-forward's 'ff' must be positive")
        if self.kind == "moe":
            if not 0 < self.top <= self.experts:
                raise ConfigError(f"{at}: router 'top' must lie between 1 and 'experts' ({self.experts}), got {self.top}")
            if self.groups < 1 or self.experts % self.groups or not 0 < self.keep_groups <= self.groups \
                    or self.keep_groups * (self.experts // self.groups) < self.top:
                raise ConfigError(f"{at}: router 'groups' must cut {self.experts} experts into equal groups of which 'keep' hold the "
                                  f"{self.top} chosen; got count {self.groups}, keep {self.keep_groups}")


@dataclass(frozen=True)
class LayerConfig:
    mixer: ParallelConfig
    mlp: Optional[MlpConfig]
    weights_of: Optional[int] = None        # the layer whose tensors this one uses; None: its own

    def to_dict(self) -> Dict[str, Any]:
        out = {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(), "type": "parallel"}
        if self.weights_of is not None:
            out["weights_of"] = self.weights_of
        return out


@dataclass(frozen=True)
class BomotarConfig(ModelConfig):
    architecture: str
    vocab_size: int
    dim: int
    norm_eps: float
    residual_mult: float
    buckets: int
    mul_prev: int
    mul_cur: int
    layers: Tuple[LayerConfig, ...]
    max_seq_len: int = DEFAULT_MAX_POSITIONS

    @classmethod
    def from_json(cls, raw: Mapping[str, Any], where: str) -> "BomotarConfig":
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError(f"{where}: key 'layers' must be a list with one object per layer")
        parsed = []
        for i, layer in enumerate(layers):
            at = f"{where}: layers[{i}]"
            if not isinstance(layer, Mapping):
                raise ConfigError(f"{at} must be an object")
            kind = require_key(layer, "type", str, at)
            if kind != "parallel":
                raise ConfigError(f"{at}: unknown layer type {kind!r}; known: parallel")
            mlp = layer.get("mlp")
            parsed.append(LayerConfig(ParallelConfig.from_dict(_object(layer, "mixer", at), f"{at}.mixer"),
                                      None if mlp is None else MlpConfig.from_dict(mlp, f"{at}.mlp"),
                                      None if layer.get("weights_of") is None else require_key(layer, "weights_of", int, at)))
        bigram = _object(_object(raw, "embedding", where), "bigram", f"{where}: embedding")
        return cls(
            architecture=NAME,
            vocab_size=require_key(raw, "vocab", int, where),
            dim=require_key(raw, "width", int, where),
            norm_eps=require_key(_object(raw, "norm", where), "eps", float, f"{where}: norm"),
            residual_mult=require_key(raw, "residual_mult", float, where),
            **{key: require_key(bigram, key, int, f"{where}: embedding.bigram") for key in ("buckets", "mul_prev", "mul_cur")},
            layers=tuple(parsed),
        ).validate(where)

    def validate(self, where: str = "config") -> "BomotarConfig":
        _positive(self, ("vocab_size", "dim", "max_seq_len", "buckets"), where)
        for i, layer in enumerate(self.layers):
            at = f"{where}: layers[{i}]"
            layer.mixer.validate(f"{at}.mixer")
            if layer.mlp is not None:
                layer.mlp.validate(at)
            owner = self.layers[self.owner(i, at)]
            if (owner.mixer, owner.mlp) != (layer.mixer, layer.mlp):
                raise ConfigError(f"{at}: 'weights_of' names layer {layer.weights_of}, whose sizes are not this layer's")
        return self

    def owner(self, i: int, at: str = "config") -> int:
        """The layer whose tensors layer ``i`` uses (itself, without ``weights_of``)."""
        seen = set()
        while self.layers[i].weights_of is not None:
            seen.add(i)
            i = self.layers[i].weights_of
            if not 0 <= i < len(self.layers) or i in seen:
                raise ConfigError(f"{at}: 'weights_of' does not lead to a layer with tensors of its own")
        return i

    def owners(self) -> List[int]:
        """The layers that have tensors of their own, in order."""
        return [i for i, layer in enumerate(self.layers) if layer.weights_of is None]

    def to_hf(self) -> Dict[str, Any]:
        return {
            "architecture": NAME,
            "embedding": {"bigram": {"buckets": self.buckets, "mul_cur": self.mul_cur, "mul_prev": self.mul_prev}},
            "layers": [layer.to_dict() for layer in self.layers],
            "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult,
            "vocab": self.vocab_size,
            "width": self.dim,
        }


def parse_config(raw: Mapping[str, Any], source: str) -> BomotarConfig:
    return BomotarConfig.from_json(raw, source)


def build_spec(cfg: BomotarConfig) -> ModelSpec:
    norm = part("rmsnorm", dim=cfg.dim, eps=cfg.norm_eps)
    out_norm = part("rmsnorm", dim=cfg.dim, eps=cfg.norm_eps, weight_scale=cfg.residual_mult)
    layers, index = [], {}
    for i in cfg.owners():
        layer = cfg.layers[i]
        a, r = layer.mixer.left, layer.mixer.right
        left = part("rotary_gated_attention", dim=cfg.dim, n_heads=a.heads, n_kv_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.vdim,
                    scale=a.scale, conv_taps=a.conv, rot_dims=a.rot_dims, rot_base=a.rot_base, rot_pairing="half", gate="element",
                    out_scale=layer.mixer.left_scale, rot_ramp=None if a.scaling is None else a.scaling.to_dict())
        right = part("gated_delta", dim=cfg.dim, n_heads=r.heads, n_qk_heads=r.kv_heads, head_dim=r.dim, v_head_dim=r.vdim,
                     conv_taps=r.conv, q_scale=r.dim ** -0.5, norm_eps=cfg.norm_eps, unit_eps=UNIT_EPS, decay="channel",
                     low_rank_gate=True, gate_activation="sigmoid", out_scale=layer.mixer.right_scale)
        mixer = part("side_by_side_sum", dim=cfg.dim, left=left, right=right)
        mlp = layer.mlp
        if mlp is None:
            ffn = None
        elif mlp.kind == "dense":
            ffn = part("activated", dim=cfg.dim, hidden=mlp.ff, activation="gelu_tanh")
        else:
            ffn = part("routed_experts", dim=cfg.dim, n_experts=mlp.experts, top=mlp.top, hidden=mlp.ff, activation="silu", gated=True,
                       choice_correction=True, n_groups=mlp.groups, keep_groups=mlp.keep_groups, group_score_top=1)
        block = part("sandwich", mixer=mixer, feed_forward=ffn, mixer_norm=norm, mixer_out_norm=out_norm,
                     ffn_norm=None if ffn is None else norm, ffn_out_norm=None if ffn is None else out_norm, mixer_prefix="mix",
                     ffn_prefix="mlp", mixer_norm_prefix="norm1", mixer_out_norm_prefix="norm1b", ffn_norm_prefix="norm2",
                     ffn_out_norm_prefix="norm2b")
        index[i] = len(layers)
        layers.append(LayerSpec(name=f"l{i}", block=block))
    # every run has a cache and a state of its own, also the runs of one layer's weights
    runs = tuple(RunEntry(index[cfg.owner(i)]) for i in range(len(cfg.layers)))
    return ModelSpec(
        dim=cfg.dim, vocab_size=cfg.vocab_size, max_positions=cfg.max_seq_len,
        embedding_tensor="embed", layers=tuple(layers), run_order=runs,
        final_norm=norm, final_norm_prefix="final.norm", head_tensor="head",
        pair_table=PairTable(PAIR_TENSOR, cfg.buckets, cfg.mul_prev, cfg.mul_cur),
    )


# checkpoint name (inside a layer) -> the parts' own names
_LAYER_NAMES = {f"{n}": f"{n}.weight" for n in ("norm1", "norm1b", "norm2", "norm2b")}
for _n in ("q", "k", "v", "g", "o"):
    _LAYER_NAMES[f"mix.left.{_n}"] = f"mix.left.w{_n}.weight"
for _n in ("q", "k", "v", "b", "a1", "a2", "g1", "g2", "o"):
    _LAYER_NAMES[f"mix.right.{_n}"] = f"mix.right.w{_n}.weight"
for _side in ("left", "right"):
    for _n in ("q", "k", "v"):
        _LAYER_NAMES[f"mix.{_side}.{_n}.conv"] = f"mix.{_side}.w{_n}.conv"
_LAYER_NAMES.update({"mix.right.norm": "mix.right.norm.weight", "mlp.up": "mlp.up.weight", "mlp.down": "mlp.down.weight",
                     "mlp.router": "mlp.router.weight"})
_TOP_NAMES = {"final.norm": "final.norm.weight"}
_LAYER_RE = re.compile(r"^(l\d+)\.(.+)$")
_EXPERT_RE = re.compile(r"^mlp\.e(\d+)\.(gate|up|down)$")


def adapt_tensors(cfg: BomotarConfig, found: Dict[str, LazyTensor]) -> Dict[str, LazyTensor]:
    """The checkpoint's names to the parts' names; anything unknown keeps its name, so that the
    strict check reports it."""
    out: Dict[str, LazyTensor] = {}
    # stored for a feed-forward that the layer does not have: nothing reads them
    unread = {f"l{i}.{n}" for i, layer in enumerate(cfg.layers) if layer.mlp is None for n in ("norm2", "norm2b")}
    for name, t in found.items():
        if name in unread:
            continue
        new = _TOP_NAMES.get(name, name)
        m = _LAYER_RE.match(name)
        if m:
            inner = m.group(2)
            e = _EXPERT_RE.match(inner)
            if e:
                new = f"{m.group(1)}.mlp.experts.{int(e.group(1))}.{e.group(2)}.weight"
            elif inner in _LAYER_NAMES:
                new = f"{m.group(1)}.{_LAYER_NAMES[inner]}"
        if new in out:
            raise ValueError(f"checkpoint provides tensor {new!r} under two names")
        out[new] = t
    return out


def tensor_shapes(cfg: BomotarConfig) -> Iterator[Tuple[str, Tuple[int, ...], str]]:
    """``(checkpoint name, shape, kind of initial values)`` of every tensor, in the order random weights are drawn in.
    No configuration carries the inner sizes of the low-rank projections: random weights take a head's key size for
    the decay and its value size for the gate."""
    d = cfg.dim
    yield "embed", (cfg.vocab_size, d), "table"
    yield PAIR_TENSOR, (cfg.buckets + 1, d), "small"
    for i in cfg.owners():
        a, r, mlp, p = cfg.layers[i].mixer.left, cfg.layers[i].mixer.right, cfg.layers[i].mlp, f"l{i}"
        for n in ("1", "2") if mlp is not None else ("1",):
            yield f"{p}.norm{n}", (d,), "gain"
            yield f"{p}.norm{n}b", (d,), "gain"
        for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
            yield f"{p}.mix.left.{n}", (rows, d), "matrix"
            yield f"{p}.mix.left.{n}.conv", (rows, a.conv), "taps"
        yield f"{p}.mix.left.g", (a.heads * a.vdim, d), "matrix"
        yield f"{p}.mix.left.o", (d, a.heads * a.vdim), "matrix"
        for n, rows in (("q", r.kv_heads * r.dim), ("k", r.kv_heads * r.dim), ("v", r.heads * r.vdim)):
            yield f"{p}.mix.right.{n}", (rows, d), "matrix"
            yield f"{p}.mix.right.{n}.conv", (rows, r.conv), "taps"
        yield f"{p}.mix.right.b", (r.heads, d), "matrix"
        yield f"{p}.mix.right.A_log", (r.heads,), "small"
        yield f"{p}.mix.right.norm", (r.vdim,), "gain"
        yield f"{p}.mix.right.a1", (r.dim, d), "matrix"
        yield f"{p}.mix.right.a2", (r.heads * r.dim, r.dim), "matrix"
        yield f"{p}.mix.right.dt_bias", (r.heads * r.dim,), "decay_bias"
        yield f"{p}.mix.right.g1", (r.vdim, d), "matrix"
        yield f"{p}.mix.right.g2", (r.heads * r.vdim, r.vdim), "matrix"
        yield f"{p}.mix.right.o", (d, r.heads * r.vdim), "matrix"
        if mlp is not None and mlp.kind == "dense":
            yield f"{p}.mlp.up", (mlp.ff, d), "matrix"
            yield f"{p}.mlp.down", (d, mlp.ff), "matrix"
        elif mlp is not None:
            for e in range(mlp.experts):
                yield f"{p}.mlp.e{e}.gate", (mlp.ff, d), "matrix"
                yield f"{p}.mlp.e{e}.up", (mlp.ff, d), "matrix"
                yield f"{p}.mlp.e{e}.down", (d, mlp.ff), "matrix"
            yield f"{p}.mlp.router", (mlp.experts, d), "matrix"
            yield f"{p}.mlp.correction", (mlp.experts,), "correction"
    yield "final.norm", (d,), "gain"
    yield "head", (cfg.vocab_size, d), "matrix"


def random_tensors(cfg: BomotarConfig, seed: int, *, device="cpu", dtype: torch.dtype = torch.float32) -> Iterator[Tuple[str, torch.Tensor]]:
    """Seeded random weights under the checkpoint's names (one generator, one order, drawn in
    float32, then cast): matrices ``N(0, 1/fan_in)``, table rows of unit size, gains around one, small
    convolution taps, decays mostly close to one."""
    gen = torch.Generator(device=device)
    gen.manual_seed(int(seed))
    for name, shape, init in tensor_shapes(cfg):
        t = torch.randn(shape, generator=gen, device=device, dtype=torch.float32)
        if init == "matrix":
            t = t * shape[1] ** -0.5
        elif init in ("small", "taps"):
            t = t * 0.3
        elif init == "correction":
            t = t * 0.02
        elif init == "decay_bias":
            t = t - 3.0
        elif init == "gain":
            t = 1.0 + t * 0.1
        yield name, t.to(dtype)


BOMOTAR = register_architecture(Architecture(
    name=NAME,
    parse_config=parse_config,
    build_spec=build_spec,
    adapt_tensors=adapt_tensors,
    random_tensors=random_tensors,
    chat_template=None,
))
