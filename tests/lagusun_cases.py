"""Small Lagusun configurations with random weights for the tests, and the two ways of running
them: the plain implementation (``plain_lagusun``) and the engine, either over the CUDA kernels
or, without a GPU, over their plain PyTorch twins (``torch_ops.TorchOps``), which still exercises
the package's parts, cache manager, step function and scheduler.

The configurations differ from each other in every size, so that nothing can lean on two numbers
being equal or one: grouped and ungrouped heads, key and value sizes that differ, rotations over a
part of a head, over all of it and over none, frequencies in all three bands of the rescaling and
without it, windows and chunks of one position, smaller and larger than a page and than a prompt,
one norm group and several (of widths that are no multiple of four), one expert per token and
several, with and without a shared expert, layers without a feed-forward, loops over some layers,
over all of them, once, three times, and no loop.
"""

from __future__ import annotations

import json
from pathlib import Path
from typing import Dict, List, Optional

import numpy as np
import torch

import plain_lagusun as plain
from nagolix_cases import BACKENDS, feed, make_replayer, stored_dtype, tokens_for  # noqa: F401  (generic helpers)

BAND = {"factor": 4.0, "high": 3.0, "low": 1.0, "original": 40}      # wavelengths below 13, up to 40 and beyond


def chunked(heads=4, kv_heads=2, dim=16, rot_dims=8, base=10000.0, size=12, scale=None, mlp=None):
    return {"mixer": {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": size}, "rot": {"base": base, "dims": rot_dims},
                      "scale": scale or dim ** -0.5, "vdim": dim}, "mlp": mlp, "type": "attention"}


def windowed(heads=3, kv_heads=1, dim=12, vdim=20, rot_dims=8, base=500.0, scaling=BAND, size=7, softcap=4.0, scale=None, mlp=None):
    rot = {"base": base, "dims": rot_dims}
    if scaling:
        rot["scaling"] = scaling
    return {"mixer": {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": size}, "rot": rot, "scale": scale or dim ** -0.5,
                      "softcap": softcap, "vdim": vdim}, "mlp": mlp, "type": "attention_2"}


def moe(experts=6, top=2, ff=24, scale=1.3, shared=20):
    out = {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "scale": scale, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(layers, width=48, vocab=89, eps=1e-5, groups=3, scale=3.0, loop=None):
    out = {"architecture": "Lagusun", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps, "groups": groups},
           "vocab": vocab, "width": width}
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


# name -> (config, page size)
CASES = {
    # both mixers with and without experts, sizes all different; the last layers but one run three times
    "mixed": (config([
        windowed(mlp=moe(6, 2, 24)),
        chunked(mlp=None),
        windowed(heads=4, kv_heads=2, dim=8, vdim=12, rot_dims=4, scaling=None, size=19, softcap=30.0, mlp=None),
        chunked(heads=2, kv_heads=1, dim=24, rot_dims=24, size=33, base=50.0, mlp=None),
        windowed(heads=2, kv_heads=2, dim=20, vdim=8, rot_dims=16, size=5, mlp=moe(5, 3, 16, scale=0.8, shared=None)),
    ], width=48, vocab=89, loop=(1, 4, 3)), 8),
    # awkward sizes: a width that is no multiple of 8 in groups that are none of 4, one key/value head per head, no rotation,
    # an odd half of the rotated part, a window and a chunk of one position, one expert per token, every layer in a
    # loop that runs once, an embedding scale of one
    "awkward": (config([
        chunked(heads=3, kv_heads=3, dim=10, rot_dims=6, base=50.0, size=5, mlp=moe(7, 1, 20)),
        windowed(heads=2, kv_heads=2, dim=6, vdim=14, rot_dims=6, size=3, softcap=1.5, mlp=None),
        windowed(heads=1, kv_heads=1, dim=9, vdim=5, rot_dims=0, size=1, mlp=None),
        chunked(heads=5, kv_heads=1, dim=7, rot_dims=2, size=1, mlp=moe(3, 3, 12, scale=2.1, shared=6)),
    ], width=44, vocab=61, eps=1e-4, groups=2, scale=1.0, loop=(0, 4, 1)), 4),
    # sizes the tensor-core kernels take, prompts longer than pages and than the kernels' tiles; no loop
    "wide": (config([
        windowed(heads=4, kv_heads=2, dim=64, vdim=128, rot_dims=32, base=9000.0, size=70, softcap=20.0, mlp=moe(8, 2, 96, shared=64)),
        chunked(heads=6, kv_heads=2, dim=128, rot_dims=64, base=1000.0, size=90, mlp=None),
        windowed(heads=8, kv_heads=1, dim=40, vdim=32, rot_dims=16, scaling=None, size=200, mlp=None),
    ], width=192, vocab=211, groups=4, scale=12.0), 16),
}


def tensors_for(cfg: dict, seed: int, sharp: float = 1.0) -> Dict[str, torch.Tensor]:
    """Random float32 tensors under the checkpoint's names.  ``sharp`` scales the query sides where a norm does not
    take the scale away again, so that attention is peaked and a single wrong key moves the logits."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * (gain / cols ** 0.5)

    def vec(n, centre=0.0, spread=0.1):
        return centre + spread * torch.randn(n, generator=g)

    out = {"embed": torch.randn(cfg["vocab"], d, generator=g) * 0.3, "final.norm": vec(d, 1.0), "head": mat(cfg["vocab"], d)}
    loop = cfg.get("loop")
    if loop:
        out["loop.in"] = mat(d, 2 * d, 1.5)
        out["loop.step"] = 0.5 * torch.randn(loop["times"], d, generator=g)
    for i, layer in enumerate(cfg["layers"]):
        m, mlp, p = layer["mixer"], layer["mlp"], f"l{i}."
        for n in ("1", "2") if mlp is not None else ("1",):
            out[p + "norm" + n], out[p + "ls" + n] = vec(d, 1.0), vec(d, 0.7, 0.3)
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out[p + "mix.q"], out[p + "mix.k"], out[p + "mix.o"] = mat(H * dk, d, 1.5), mat(G * dk, d, 1.5), mat(d, H * dv)
        if layer["type"] == "attention":
            out[p + "mix.q.norm"], out[p + "mix.k.norm"] = vec(H * dk, 1.0 * sharp), vec(G * dk, 1.0)
        else:
            out[p + "mix.v"] = mat(G * dv, d)
            for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
                out[p + f"mix.{n}.b"] = vec(rows, 0.0, 0.3)
            out[p + "mix.pb"] = vec(H, -1.5, 0.7)
        if mlp is not None:
            r, ff = mlp["router"], mlp["expert"]["ff"]
            for e in range(r["experts"]):
                out[p + f"mlp.e{e}.up"], out[p + f"mlp.e{e}.down"] = mat(ff, d, 2.0), mat(d, ff)
            out[p + "mlp.router"] = mat(r["experts"], d, 1.5)      # logits of order one: scores that do not crowd at 0 and 1
            out[p + "mlp.correction"] = vec(r["experts"], 0.0, 0.2)
            if mlp.get("shared"):
                sf = mlp["shared"]["ff"]
                out[p + "mlp.shared.up"], out[p + "mlp.shared.down"] = mat(sf, d, 2.0), mat(d, sf)
    return out


def write_folder(tmp, name: str, cfg: dict, tensors: Dict[str, torch.Tensor], dtype=torch.float32) -> Path:
    from safetensors.torch import save_file
    folder = Path(tmp) / f"lagusun_{name}"
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.to(dtype).contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))
    return folder


def stored(tensors: Dict[str, torch.Tensor], dtype) -> Dict[str, torch.Tensor]:
    """What the file stores is what both sides compute with."""
    return tensors if dtype == torch.float32 else {k: v.to(dtype).float() for k, v in tensors.items()}


def case_folder(tmp, name: str, sharp: Optional[float] = None, dtype=torch.float32):
    """In float32 the weights are sharp (peaked attention); in bfloat16 they are not, or rounding alone would
    scatter the logits."""
    cfg, page = CASES[name]
    if sharp is None:
        sharp = 3.0 if dtype == torch.float32 else 1.0
    tensors = stored(tensors_for(cfg, seed=sum(map(ord, name)), sharp=sharp), dtype)
    return cfg, tensors, write_folder(tmp, name, cfg, tensors, dtype), page


def clear_tokens(cfg: dict, tensors, n: int, seed: int = 0, dtype: str = "bfloat16") -> List[int]:
    """Random tokens on which no router of the model has a close call: everywhere the last expert chosen stands above
    the first one left out by a margin in score (0.04 for bfloat16, where the rows that the router reads carry the
    rounding of everything before them; 1e-4 for float32).  A choice that rounding flips would move that row's
    logits, and through the cache later rows', by far more than rounding does.  The sequence is grown a few tokens at
    a time, a block being drawn again until its own positions are clear (the model is causal)."""
    if not any(l["mlp"] is not None for l in cfg["layers"]):
        return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], size=n).tolist()
    margin, block = (0.04, 2) if dtype == "bfloat16" else (1e-4, 20)
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
            raise AssertionError("no tokens with clear routing found: make the router sharper")
        tokens += drawn
    return tokens


class Expected:
    """The plain logits of a sequence and how far an engine may be from them.  In float32: 2.5e-4 of
    the largest logit on every logit (1e-3 at least: a wrong key, expert or pass moves them by tenths).  In bfloat16
    the yardstick is what rounding itself does to this model: the plain implementation is run a second time with
    bfloat16 rounding of every projection and activation, and a row of the engine's logits may differ from the exact
    ones (root mean square over the vocabulary) by three times what that emulation differs, the
    typical row's figure standing in where a row's own is smaller; one row in twenty may pass
    that, by half at most."""

    def __init__(self, cfg, tensors, tokens, dtype: str):
        self.dtype = dtype
        self.logits = plain.forward(cfg, tensors, tokens).to(torch.float32).numpy()
        if dtype == "bfloat16":
            rounded = plain.forward(cfg, tensors, tokens, rounding=torch.bfloat16).to(torch.float32).numpy()
            noise = np.sqrt(((rounded - self.logits) ** 2).mean(-1))
            self.allowed = 3.0 * np.maximum(noise, np.median(noise))

    def check(self, got: np.ndarray, what: str = "") -> None:
        assert got.shape == self.logits.shape, f"{what}: {got.shape} logits for {self.logits.shape}"
        if self.dtype == "float32":
            err = np.abs(got - self.logits)
            limit = 2.5e-4 * max(4.0, float(np.abs(self.logits).max()))
            assert err.max() <= limit, f"{what}: logits differ by {err.max()} (allowed {limit}), row {int(err.max(-1).argmax())}"
        else:
            err = np.sqrt(((got - self.logits) ** 2).mean(-1))
            worst = int(np.argmax(err / self.allowed))
            assert err[worst] <= 1.5 * self.allowed[worst], \
                f"{what}: row {worst} differs by {err[worst]} (rms), rounding alone allows {self.allowed[worst]}"
            assert (err > self.allowed).mean() <= 0.05, f"{what}: {(err > self.allowed).sum()} of {len(err)} rows over their allowance"


def plain_logits(cfg, tensors, tokens, dtype: str) -> Expected:
    return Expected(cfg, tensors, tokens, dtype)
