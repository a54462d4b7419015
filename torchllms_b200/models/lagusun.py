"""Lagusun as an :class:`~torchllms_b200.config.registry.Architecture`.

A small decoder whose ``config.json`` lists its layers one by one; every layer names its mixer
(``attention`` or ``attention_2``) with that mixer's own sizes, and its feed-forward (``moe`` or none).
A span of layers (``loop``: ``start``, ``stop``, ``times``) runs several times in a row with the same
weights, every pass with a cache of its own.  What the design fixes and no file carries:

* the stream is the embedding table's row times ``embedding.scale``; the head is a matrix of its own;
* a layer is ``x += ls1 * mixer(norm1(x))``, ``x += ls2 * ff(norm2(x))`` with a stored vector for each sum;
  every norm cuts the row into ``norm.groups`` equal runs with a root mean square each and has a plain
  weight per coordinate;
* a pass of the looped span starts with ``x = loop.in [x; embedding output] + loop.step[pass]``;
* ``attention``: no biases, values are the keys as projected, an RMS norm over all of q and all of k
  ahead of the rotation (pairs ``i``, ``i + rot.dims / 2``), keys of the query's own chunk of
  ``mask.size`` positions, a softmax with one added to its denominator;
* ``attention_2``: biases on q, k and v, rotation with frequencies rescaled by band (``rot.scaling``),
  rotated heads of q and k and the heads of v divided by their root mean square, a capped score
  ``softcap * tanh(score / softcap)``, a sliding window of ``mask.size`` keys, and for every visible key
  the weight ``sigmoid(score + pb[head])`` without a sum over the keys;
* ``moe``: experts ``down(gelu(up x))`` (the exact gelu), sigmoid scores, a correction that steers the
  choice alone, weights ``score / (sum + 1e-20) * router.scale``, and a shared expert of the same form.

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
from ..parts.spec import LayerSpec, ModelSpec, RunEntry, part
from ..weights.loader import LazyTensor

NAME = "Lagusun"

# The design has no longest sequence (rotary positions); tables are made this long unless whoever
# builds the engine asks for more.
DEFAULT_MAX_POSITIONS = 32768

RENORM_EPS = 1e-20            # weights = score / (sum of the chosen scores + RENORM_EPS)
JOIN_TENSOR, STEP_TENSOR = "loop.in", "loop.step"


def _object(raw: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"{where}: key '{key}' must be an object")
    return value


@dataclass(frozen=True)
class BandScaling:
    """Rotary frequencies rescaled by band: see :func:`torchllms_b200.parts.rope.band_scaled`."""

    factor: float
    low: float
    high: float
    original: float

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "BandScaling":
        return cls(*(require_key(raw, key, float, where) for key in ("factor", "low", "high", "original")))

    def to_dict(self) -> Dict[str, Any]:
        return {"factor": self.factor, "high": self.high, "low": self.low, "original": self.original}


@dataclass(frozen=True)
class AttentionConfig:
    """Both kinds of attention; ``softcap`` and ``scaling`` belong to ``attention_2``."""

    kind: str                       # "attention" or "attention_2"
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    mask_size: int                  # attention: positions of a chunk; attention_2: keys of a window
    rot_dims: int
    rot_base: float
    scaling: Optional[BandScaling] = None
    softcap: float = 0.0

    @classmethod
    def from_dict(cls, kind: str, raw: Mapping[str, Any], where: str) -> "AttentionConfig":
        rot, mask = _object(raw, "rot", where), _object(raw, "mask", where)
        second = kind == "attention_2"
        scaling = _object(rot, "scaling", f"{where}.rot") if rot.get("scaling") is not None else None
        return cls(kind, heads=require_key(raw, "heads", int, where), kv_heads=require_key(raw, "kv_heads", int, where),
                   dim=require_key(raw, "dim", int, where), vdim=require_key(raw, "vdim", int, where),
                   scale=require_key(raw, "scale", float, where), mask_size=require_key(mask, "size", int, f"{where}.mask"),
                   rot_dims=require_key(rot, "dims", int, f"{where}.rot"), rot_base=require_key(rot, "base", float, f"{where}.rot"),
                   scaling=None if scaling is None else BandScaling.from_dict(scaling, f"{where}.rot.scaling"),
                   softcap=require_key(raw, "softcap", float, where) if second else 0.0)

    def to_dict(self) -> Dict[str, Any]:
        rot: Dict[str, Any] = {"base": self.rot_base, "dims": self.rot_dims}
        if self.scaling is not None:
            rot["scaling"] = self.scaling.to_dict()
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "mask": {"size": self.mask_size}, "rot": rot,
               "scale": self.scale, "vdim": self.vdim}
        if self.kind == "attention_2":
            out["softcap"] = self.softcap
        return out

    def validate(self, at: str) -> None:
        for key in ("heads", "kv_heads", "dim", "vdim"):
            if getattr(self, key) <= 0:
                raise ConfigError(f"{at}: mixer '{key}' must be positive, got {getattr(self, key)}")
        if self.heads % self.kv_heads != 0:
            raise ConfigError(f"{at}: 'heads' ({self.heads}) must be a multiple of 'kv_heads' ({self.kv_heads})")
        if self.mask_size < 1:
            raise ConfigError(f"{at}: 'mask.size' must be positive, got {self.mask_size}")
        if self.rot_dims < 0 or self.rot_dims % 2 or self.rot_dims > self.dim:
            raise ConfigError(f"{at}: 'rot.dims' must be even and at most 'dim' ({self.dim}), got {self.rot_dims}")
        if not self.rot_base > 0:
            raise ConfigError(f"{at}: 'rot.base' must be positive")
        s = self.scaling
        if s is not None and not (s.factor > 0 and s.low > 0 and s.high >= s.low and s.original > 0):
            raise ConfigError(f"{at}: 'rot.scaling' needs positive numbers with 'high' at least 'low'")
        if self.kind == "attention" and self.vdim != self.dim:
            raise ConfigError(f"{at}: values are the keys, so 'vdim' ({self.vdim}) must equal 'dim' ({self.dim})")
        if self.kind == "attention_2" and not self.softcap > 0:
            raise ConfigError(f"{at}: 'softcap' must be positive, got {self.softcap}")


@dataclass(frozen=True)
class MlpConfig:
    """A layer of experts."""

    ff: int                         # one expert's hidden size
    experts: int
    top: int
    router_scale: float
    shared_ff: int = 0              # 0: no shared expert

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "MlpConfig":
        kind = require_key(raw, "kind", str, where)
        if kind != "moe":
            raise ConfigError(f"{where}: unknown feed-forward kind {kind!r}; known: moe")
        router, expert = _object(raw, "router", where), _object(raw, "expert", where)
        shared = None if raw.get("shared") is None else _object(raw, "shared", where)
        return cls(require_key(expert, "ff", int, f"{where}.expert"), experts=require_key(router, "experts", int, f"{where}.router"),
                   top=require_key(router, "top", int, f"{where}.router"),
                   router_scale=require_key(router, "scale", float, f"{where}.router"),
                   shared_ff=0 if shared is None else require_key(shared, "ff", int, f"{where}.shared"))

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"expert": {"ff": self.ff}, "kind": "moe",
                               "router": {"experts": self.experts, "scale": self.router_scale, "top": self.top}}
        if self.shared_ff:
            out["shared"] = {"ff": self.shared_ff}
        return out

    def validate(self, at: str) -> None:
        if self.ff <= 0 or self.shared_ff < 0:
            raise ConfigError(f"{at}: an expert's 'ff' must be positive")
        if not 0 < self.top <= self.experts:
            raise ConfigError(f"{at}: router 'top' must lie between 1 and 'experts' ({self.experts}), got {self.top}")


@dataclass(frozen=True)
class LayerConfig:
    mixer: AttentionConfig
    mlp: Optional[MlpConfig]


_KINDS = ("attention", "attention_2")


@dataclass(frozen=True)
class LagusunConfig(ModelConfig):
    architecture: str
    vocab_size: int
    dim: int
    norm_eps: float
    norm_groups: int
    embedding_scale: float
    layers: Tuple[LayerConfig, ...]
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    max_seq_len: int = DEFAULT_MAX_POSITIONS

    @classmethod
    def from_json(cls, raw: Mapping[str, Any], where: str) -> "LagusunConfig":
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError(f"{where}: key 'layers' must be a list with one object per layer")
        parsed = []
        for i, layer in enumerate(layers):
            at = f"{where}: layers[{i}]"
            if not isinstance(layer, Mapping):
                raise ConfigError(f"{at} must be an object")
            kind = require_key(layer, "type", str, at)
            if kind not in _KINDS:
                raise ConfigError(f"{at}: unknown layer type {kind!r}; known: {', '.join(_KINDS)}")
            mixer = AttentionConfig.from_dict(kind, _object(layer, "mixer", at), f"{at}.mixer")
            mlp = layer.get("mlp")
            parsed.append(LayerConfig(mixer, None if mlp is None else MlpConfig.from_dict(mlp, f"{at}.mlp")))
        start = stop = 0
        times = 1
        if raw.get("loop") is not None:
            loop = _object(raw, "loop", where)
            start, stop, times = (require_key(loop, key, int, f"{where}: loop") for key in ("start", "stop", "times"))
            if not (0 <= start < stop <= len(parsed)) or times < 1:
                raise ConfigError(f"{where}: 'loop' must name layers start .. stop - 1 of the {len(parsed)} there are, run at least "
                                  f"once; got start {start}, stop {stop}, times {times}")
        norm = _object(raw, "norm", where)
        return cls(
            architecture=NAME,
            vocab_size=require_key(raw, "vocab", int, where),
            dim=require_key(raw, "width", int, where),
            norm_eps=require_key(norm, "eps", float, f"{where}: norm"),
            norm_groups=require_key(norm, "groups", int, f"{where}: norm"),
            embedding_scale=require_key(_object(raw, "embedding", where), "scale", float, f"{where}: embedding"),
            layers=tuple(parsed), loop_start=start, loop_stop=stop, loop_times=times,
        ).validate(where)

    @property
    def loops(self) -> bool:
        return self.loop_stop > self.loop_start

    def validate(self, where: str = "config") -> "LagusunConfig":
        for key in ("vocab_size", "dim", "norm_groups", "max_seq_len"):
            if getattr(self, key) <= 0:
                raise ConfigError(f"{where}: '{key}' must be positive, got {getattr(self, key)}")
        if self.dim % self.norm_groups != 0:
            raise ConfigError(f"{where}: 'norm.groups' ({self.norm_groups}) must divide 'width' ({self.dim})")
        for i, layer in enumerate(self.layers):
            at = f"{where}: layers[{i}]"
            layer.mixer.validate(at)
            if layer.mlp is not None:
                layer.mlp.validate(at)
        if self.loops or self.loop_times != 1:
            if not (0 <= self.loop_start < self.loop_stop <= len(self.layers)) or self.loop_times < 1:
                raise ConfigError(f"{where}: 'loop' must name layers that there are, run at least once")
        return self

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """``(layer, pass)`` of every layer run in order; ``pass`` is a number for the first layer
        of every pass of the looped span and ``None`` elsewhere."""
        n = len(self.layers)
        if not self.loops:
            return [(i, None) for i in range(n)]
        out: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(self.loop_start)]
        for t in range(self.loop_times):
            out += [(i, t if i == self.loop_start else None) for i in range(self.loop_start, self.loop_stop)]
        return out + [(i, None) for i in range(self.loop_stop, n)]

    def to_hf(self) -> Dict[str, Any]:
        out = {
            "architecture": NAME,
            "embedding": {"scale": self.embedding_scale},
            "layers": [{"mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict(), "type": l.mixer.kind}
                       for l in self.layers],
            "norm": {"eps": self.norm_eps, "groups": self.norm_groups},
            "vocab": self.vocab_size,
            "width": self.dim,
        }
        if self.loops:
            out["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        return out


def parse_config(raw: Mapping[str, Any], source: str) -> LagusunConfig:
    return LagusunConfig.from_json(raw, source)


def build_spec(cfg: LagusunConfig) -> ModelSpec:
    norm = part("rmsnorm", dim=cfg.dim, eps=cfg.norm_eps, groups=cfg.norm_groups)
    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        common = dict(dim=cfg.dim, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, v_head_dim=m.vdim, scale=m.scale,
                      rot_dims=m.rot_dims, rot_base=m.rot_base, rot_pairing="half", norm_eps=cfg.norm_eps,
                      rot_band=None if m.scaling is None else m.scaling.to_dict())
        if m.kind == "attention":
            mixer = part("rotary_gated_attention", chunk=m.mask_size, values_are_keys=True, qk_row_norm=True, sinks="zero", **common)
        else:
            mixer = part("rotary_gated_attention", window=m.mask_size, qkv_bias=True, qk_head_norm=True, v_head_norm=True,
                         softcap=m.softcap, weights="sigmoid", score_bias=True, **common)
        mlp = layer.mlp
        ffn = None if mlp is None else \
            part("routed_experts", dim=cfg.dim, n_experts=mlp.experts, top=mlp.top, hidden=mlp.ff, activation="gelu", score="sigmoid",
                 choice_correction=True, router_scale=mlp.router_scale, renormalize=True, renorm_eps=RENORM_EPS,
                 shared_hidden=mlp.shared_ff or None)
        block = part("prenorm", mixer=mixer, feed_forward=ffn, mixer_norm=norm, ffn_norm=None if ffn is None else norm,
                     mixer_prefix="mix", ffn_prefix="mlp", mixer_norm_prefix="norm1", ffn_norm_prefix="norm2",
                     mixer_scale="ls1", ffn_scale="ls2")
        layers.append(LayerSpec(name=f"l{i}", block=block))
    # every run has a cache of its own, also the runs of one layer in different passes
    runs = tuple(RunEntry(i) if t is None else RunEntry(i, join_embedding=JOIN_TENSOR, add_row=(STEP_TENSOR, t)) for i, t in cfg.runs())
    return ModelSpec(
        dim=cfg.dim, vocab_size=cfg.vocab_size, max_positions=cfg.max_seq_len,
        embedding_tensor="embed", layers=tuple(layers), run_order=runs,
        final_norm=norm, final_norm_prefix="final.norm", head_tensor="head",
        embedding_scale=cfg.embedding_scale,
        row_tensors=((STEP_TENSOR, cfg.loop_times),) if cfg.loops else (),
        join_tensors=(JOIN_TENSOR,) if cfg.loops else (),
    )


# checkpoint name (inside a layer) -> the parts' own names
_LAYER_NAMES = {
    "norm1": "norm1.weight", "norm2": "norm2.weight",
    "mix.q": "mix.wq.weight", "mix.q.b": "mix.wq.bias", "mix.k": "mix.wk.weight", "mix.k.b": "mix.wk.bias",
    "mix.v": "mix.wv.weight", "mix.v.b": "mix.wv.bias", "mix.o": "mix.wo.weight",
    "mix.q.norm": "mix.q_norm.weight", "mix.k.norm": "mix.k_norm.weight", "mix.pb": "mix.score_bias",
    "mlp.router": "mlp.router.weight", "mlp.shared.up": "mlp.shared.up.weight", "mlp.shared.down": "mlp.shared.down.weight",
}
_TOP_NAMES = {"final.norm": "final.norm.weight"}
_LAYER_RE = re.compile(r"^(l\d+)\.(.+)$")
_EXPERT_RE = re.compile(r"^mlp\.e(\d+)\.(up|down)$")


def adapt_tensors(cfg: LagusunConfig, found: Dict[str, LazyTensor]) -> Dict[str, LazyTensor]:
    """The checkpoint's names to the parts' names; anything unknown keeps its name, so that the
    strict check reports it."""
    out: Dict[str, LazyTensor] = {}
    # stored for a feed-forward that the layer does not have: nothing reads them
    unread = {f"l{i}.{n}" for i, layer in enumerate(cfg.layers) if layer.mlp is None for n in ("norm2", "ls2")}
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


def tensor_shapes(cfg: LagusunConfig) -> Iterator[Tuple[str, Tuple[int, ...], str]]:
    """``(checkpoint name, shape, init)`` of every tensor, in the order random weights are drawn in."""
    d = cfg.dim
    yield "embed", (cfg.vocab_size, d), "matrix"
    if cfg.loops:
        yield JOIN_TENSOR, (d, 2 * d), "matrix"
        yield STEP_TENSOR, (cfg.loop_times, d), "small"
    for i, layer in enumerate(cfg.layers):
        m, mlp, p = layer.mixer, layer.mlp, f"l{i}"
        for n in ("1", "2") if mlp is not None else ("1",):
            yield f"{p}.norm{n}", (d,), "gain"
            yield f"{p}.ls{n}", (d,), "gain"
        n_q, n_k, n_v = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
        if m.kind == "attention":
            for n, rows in (("q", n_q), ("k", n_k)):
                yield f"{p}.mix.{n}", (rows, d), "matrix"
                yield f"{p}.mix.{n}.norm", (rows,), "gain"
        else:
            for n, rows in (("q", n_q), ("k", n_k), ("v", n_v)):
                yield f"{p}.mix.{n}", (rows, d), "matrix"
                yield f"{p}.mix.{n}.b", (rows,), "small"
            yield f"{p}.mix.pb", (m.heads,), "score_bias"
        yield f"{p}.mix.o", (d, m.heads * m.vdim), "matrix"
        if mlp is not None:
            for e in range(mlp.experts):
                yield f"{p}.mlp.e{e}.up", (mlp.ff, d), "matrix"
                yield f"{p}.mlp.e{e}.down", (d, mlp.ff), "matrix"
            yield f"{p}.mlp.router", (mlp.experts, d), "matrix"
            yield f"{p}.mlp.correction", (mlp.experts,), "small"
            if mlp.shared_ff:
                yield f"{p}.mlp.shared.up", (mlp.shared_ff, d), "matrix"
                yield f"{p}.mlp.shared.down", (d, mlp.shared_ff), "matrix"
    yield "final.norm", (d,), "gain"
    yield "head", (cfg.vocab_size, d), "matrix"


def random_tensors(cfg: LagusunConfig, seed: int, *, device="cpu", dtype: torch.dtype = torch.float32) -> Iterator[Tuple[str, torch.Tensor]]:
    """Seeded random weights under the checkpoint's names (one generator, one order, drawn in
    float32, then cast): matrices ``N(0, 1/fan_in)``, gains and layer scales around one, a score bias that
    keeps the unnormalised weights of a long window from adding up."""
    gen = torch.Generator(device=device)
    gen.manual_seed(int(seed))
    for name, shape, init in tensor_shapes(cfg):
        t = torch.randn(shape, generator=gen, device=device, dtype=torch.float32)
        if init == "matrix":
            t = t * shape[1] ** -0.5
        elif init == "small":
            t = t * 0.1
        elif init == "gain":
            t = 1.0 + t * 0.1
        elif init == "score_bias":
            t = t * 0.5 - 4.0
        yield name, t.to(dtype)


LAGUSUN = register_architecture(Architecture(
    name=NAME,
    parse_config=parse_config,
    build_spec=build_spec,
    adapt_tensors=adapt_tensors,
    random_tensors=random_tensors,
    chat_template=None,
))
