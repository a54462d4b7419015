"""Small Bomotar configurations with random weights for the tests, and the two ways of running
them: the plain implementation (``plain_bomotar``) and the engine, either over the CUDA kernels
or, without a GPU, over their plain PyTorch twins (``torch_ops.TorchOps``), which still exercises
the package's parts, cache manager, step function and scheduler.

The configurations differ from each other in every size, so that nothing can lean on two numbers
being equal or on a number being one: grouped and ungrouped heads on both sides, key and value sizes
that differ, convolutions of one tap and of several (not the same on both sides), rotations over a part of
a head and over all of it, with and without a rescaling, inner sizes of the low-rank projections
that differ and are no multiples of eight, layers that share weights in any order, layers without a
feed-forward, one expert per token and several, experts with and without groups.
"""

from __future__ import annotations

import json
from pathlib import Path
from typing import Dict, List, Optional

import numpy as np
import torch

import plain_bomotar as plain
from nagolix_cases import BACKENDS, feed, make_replayer, stored_dtype, tokens_for  # noqa: F401  (generic helpers)


def ramp(factor=4.0, original=64, fast=8.0, slow=1.5):
    return {"factor": factor, "fast": fast, "original": original, "slow": slow}


def attention(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, rot_dims=8, base=1000.0, scaling=None, scale=None):
    rot = {"base": base, "dims": rot_dims}
    if scaling is not None:
        rot["scaling"] = scaling
    return {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "rot": rot, "scale": scale or dim ** -0.5, "vdim": vdim}


def delta(heads=4, kv_heads=2, dim=12, vdim=20, conv=2):
    return {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim}


def dense(ff=80):
    return {"ff": ff, "kind": "dense"}


def moe(experts=8, top=3, ff=24, groups=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"expert": {"ff": ff}, "kind": "moe", "router": router}


def layer(left=None, right=None, left_scale=0.8, right_scale=1.3, mlp=None, ranks=(5, 9)):
    """``ranks``: inner sizes of the low-rank projections (decay, gate), which the stored tensors carry."""
    return {"mixer": {"left": left or attention(), "left_scale": left_scale, "right": right or delta(), "right_scale": right_scale},
            "mlp": mlp, "type": "parallel", "_ranks": ranks}


def again(layers: list, j: int) -> dict:
    """A layer that uses layer ``j``'s weights."""
    return dict(layers[j], weights_of=j)


def config(layers, width=48, vocab=89, eps=1e-5, mult=0.6, buckets=101, mul_prev=17, mul_cur=5):
    return {"architecture": "Bomotar", "embedding": {"bigram": {"buckets": buckets, "mul_cur": mul_cur, "mul_prev": mul_prev}},
            "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


def clean(cfg: dict) -> dict:
    """The configuration as a file carries it (without the tests' own notes)."""
    out = dict(cfg)
    out["layers"] = [{k: v for k, v in l.items() if not k.startswith("_")} for l in cfg["layers"]]
    return out


_MIXED = [
    layer(attention(scaling=ramp()), delta(), mlp=moe(8, 3, 24, groups=(4, 2))),
    layer(attention(heads=3, kv_heads=1, dim=12, vdim=8, conv=4, rot_dims=12, base=300.0), delta(heads=3, kv_heads=3, dim=8, vdim=16, conv=3),
          left_scale=1.4, right_scale=0.5, mlp=dense(56), ranks=(8, 16)),
]
_AWKWARD = [
    # odd head sizes, one key/value head per head, convolutions of one tap and of five, odd inner sizes, a rotation of two
    # coordinates, one expert per token out of ungrouped ones
    layer(attention(heads=3, kv_heads=3, dim=10, vdim=7, conv=1, rot_dims=2, base=50.0, scaling=ramp(2.0, 30, 4.0, 1.0)),
          delta(heads=2, kv_heads=1, dim=6, vdim=11, conv=5), left_scale=1.0, right_scale=1.0, mlp=moe(5, 1, 18), ranks=(3, 1)),
    layer(attention(heads=1, kv_heads=1, dim=9, vdim=14, conv=2, rot_dims=6, base=9.0), delta(heads=3, kv_heads=1, dim=7, vdim=5, conv=1),
          mlp=None, ranks=(1, 2)),
]
_WIDE = [
    layer(attention(heads=4, kv_heads=1, dim=64, vdim=128, conv=4, rot_dims=64, base=250000.0, scaling=ramp(3.0, 100, 16.0, 1.0)),
          delta(heads=4, kv_heads=2, dim=64, vdim=64, conv=4), mlp=dense(384), ranks=(32, 64)),
    layer(attention(heads=4, kv_heads=2, dim=32, vdim=64, conv=2, rot_dims=16), delta(heads=2, kv_heads=1, dim=160, vdim=48, conv=3),
          mlp=moe(8, 2, 96, groups=(2, 1)), ranks=(24, 40)),
]

# name -> (config, page size)
CASES = {
    # every kind of feed-forward, layers that share weights (also a layer whose weights stand further down the list)
    "mixed": (config([_MIXED[0], _MIXED[1], again(_MIXED, 0), again(_MIXED, 1)], width=48, vocab=89), 8),
    "awkward": (config([dict(_AWKWARD[1], weights_of=2), _AWKWARD[0], _AWKWARD[1], dict(_AWKWARD[1], weights_of=0)], width=44, vocab=61,
                       eps=1e-4, mult=1.0, buckets=7, mul_prev=1, mul_cur=3), 4),
    # sizes the tensor-core kernels take, prompts longer than pages and than the kernels' chunks
    "wide": (config([_WIDE[0], _WIDE[1]], width=256, vocab=211, buckets=300, mul_prev=1009, mul_cur=263), 16),
}


def tensors_for(cfg: dict, seed: int, sharp: float = 1.0) -> Dict[str, torch.Tensor]:
    """Random float32 tensors under the checkpoint's names.  ``sharp`` scales the attention's query side."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * (gain / cols ** 0.5)

    def vec(n, centre=0.0, spread=0.1):
        return centre + spread * torch.randn(n, generator=g)

    out = {"embed": torch.randn(cfg["vocab"], d, generator=g),
           "bigram": 0.7 * torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, d, generator=g)}
    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        a, r, mlp, p = l["mixer"]["left"], l["mixer"]["right"], l["mlp"], f"l{i}."
        ra, rg = l["_ranks"]
        for n in ("1", "2") if mlp is not None else ("1",):
            out[p + "norm" + n], out[p + f"norm{n}b"] = vec(d, 1.0), vec(d, 0.8, 0.2)
        H, G, dk, dv, q = a["heads"], a["kv_heads"], a["dim"], a["vdim"], p + "mix.left."
        for name, rows, gain in (("q", H * dk, 2.0 * sharp), ("k", G * dk, 2.0), ("v", G * dv, 1.5)):
            out[q + name] = mat(rows, d, gain)
            out[q + name + ".conv"] = 0.5 * torch.randn(rows, a["conv"], generator=g)
        out[q + "g"], out[q + "o"] = mat(H * dv, d, 2.0), mat(d, H * dv)
        H, G, dk, dv, q = r["heads"], r["kv_heads"], r["dim"], r["vdim"], p + "mix.right."
        for name, rows in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
            out[q + name] = mat(rows, d, 2.0)
            out[q + name + ".conv"] = 0.5 * torch.randn(rows, r["conv"], generator=g)
        out[q + "b"], out[q + "A_log"], out[q + "dt_bias"] = mat(H, d, 2.0), vec(H, -1.0, 0.7), vec(H * dk, -1.0, 1.0)
        out[q + "a1"], out[q + "a2"], out[q + "g1"], out[q + "g2"] = mat(ra, d, 1.5), mat(H * dk, ra, 1.5), mat(rg, d, 1.5), mat(H * dv, rg, 1.5)
        out[q + "norm"], out[q + "o"] = vec(dv, 1.0), mat(d, H * dv)
        if mlp is not None and mlp["kind"] == "dense":
            out[p + "mlp.up"], out[p + "mlp.down"] = mat(mlp["ff"], d, 2.0), mat(d, mlp["ff"])
        elif mlp is not None:
            E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            for e in range(E):
                out[p + f"mlp.e{e}.gate"], out[p + f"mlp.e{e}.up"] = mat(ff, d, 2.0), mat(ff, d, 2.0)
                out[p + f"mlp.e{e}.down"] = mat(d, ff)
            out[p + "mlp.router"] = mat(E, d, 1.5)
            out[p + "mlp.correction"] = 0.3 * torch.randn(E, generator=g)       # choice scores of both signs, seldom close
    out["final.norm"], out["head"] = vec(d, 1.0), mat(cfg["vocab"], d)
    return out


def write_folder(tmp, name: str, cfg: dict, tensors: Dict[str, torch.Tensor], dtype=torch.float32) -> Path:
    from safetensors.torch import save_file
    folder = Path(tmp) / f"bomotar_{name}"
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(clean(cfg)))
    save_file({k: v.to(dtype).contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))
    return folder


def stored(tensors: Dict[str, torch.Tensor], dtype) -> Dict[str, torch.Tensor]:
    """What the file stores is what both sides compute with."""
    return tensors if dtype == torch.float32 else {k: v.to(dtype).float() for k, v in tensors.items()}


def case_folder(tmp, name: str, sharp: Optional[float] = None, dtype=torch.float32):
    """In float32 the attention is sharp; in bfloat16 it is not, or rounding alone would scatter the logits."""
    cfg, page = CASES[name]
    if sharp is None:
        sharp = 2.0 if dtype == torch.float32 else 1.0
    tensors = stored(tensors_for(cfg, seed=sum(map(ord, name)), sharp=sharp), dtype)
    return cfg, tensors, write_folder(tmp, name, cfg, tensors, dtype), page


def clear_tokens(cfg: dict, tensors, n: int, seed: int = 0, dtype: str = "bfloat16") -> List[int]:
    """Random tokens on which no router of the model has a close call: everywhere the last expert and the last group
    chosen stand above the first left out by a margin in choice score (0.03 for bfloat16, where the rows that the
    router reads carry the rounding of everything before them; 1e-4 for float32).  A choice that rounding flips
    would move that row's logits, and through cache and states later rows', by far more than rounding does.  The
    sequence is grown a few tokens at a time, a block being drawn again until its own positions are clear (the
    model is causal)."""
    if not any(l["mlp"] is not None and l["mlp"]["kind"] == "moe" for l in cfg["layers"]):
        return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], size=n).tolist()
    margin, block = (0.03, 2) if dtype == "bfloat16" else (1e-4, 20)
    rng = np.random.default_rng(1000 + seed)
    tokens: List[int] = []
    while len(tokens) < n:
        k = min(block, n - len(tokens))
        for _ in range(400):
            drawn = rng.integers(0, cfg["vocab"], size=k).tolist()
            margins: list = []
            plain.forward(cfg, tensors, tokens + drawn, margins_out=margins)
            if min((float(m[len(tokens):].min()) for m in margins), default=np.inf) >= margin:
                break
        else:
            raise AssertionError("no tokens with clear routing found: spread the correction further")
        tokens += drawn
    return tokens


class Expected:
    """The plain logits of a sequence and how far an engine may be from them.  In float32: 2e-4 of
    the largest logit on every logit (8e-4 at least: a wrong key, expert or state moves them by tenths).  In bfloat16
    the yardstick is what rounding itself does to this model: the plain implementation is run again with
    bfloat16 rounding of every projection and activation, to nearest and twice up or down at random, and a row of the
    engine's logits may differ from the exact ones (root mean square over the vocabulary) by three times what the worst
    of these differs, the
    typical row's figure standing in where a row's own is smaller; one row in twenty may pass
    that, by half at most."""

    def __init__(self, cfg, tensors, tokens, dtype: str):
        self.dtype = dtype
        self.logits = plain.forward(cfg, tensors, tokens).to(torch.float32).numpy()
        if dtype == "bfloat16":
            noise = 0.0
            for rounding in (torch.bfloat16, plain.either_way(1), plain.either_way(2)):
                rounded = plain.forward(cfg, tensors, tokens, rounding=rounding).to(torch.float32).numpy()
                noise = np.maximum(noise, np.sqrt(((rounded - self.logits) ** 2).mean(-1)))
            self.allowed = 3.0 * np.maximum(noise, np.median(noise))

    def check(self, got: np.ndarray, what: str = "") -> None:
        assert got.shape == self.logits.shape, f"{what}: {got.shape} logits for {self.logits.shape}"
        if self.dtype == "float32":
            err = np.abs(got - self.logits)
            limit = 2e-4 * max(4.0, float(np.abs(self.logits).max()))
            assert err.max() <= limit, f"{what}: logits differ by {err.max()} (allowed {limit}), row {int(err.max(-1).argmax())}"
        else:
            err = np.sqrt(((got - self.logits) ** 2).mean(-1))
            worst = int(np.argmax(err / self.allowed))
            assert err[worst] <= 1.5 * self.allowed[worst], \
                f"{what}: row {worst} differs by {err[worst]} (rms), rounding alone allows {self.allowed[worst]}"
            assert (err > self.allowed).mean() <= 0.05, f"{what}: {(err > self.allowed).sum()} of {len(err)} rows over their allowance"


def plain_logits(cfg, tensors, tokens, dtype: str) -> Expected:
    return Expected(cfg, tensors, tokens, dtype)
