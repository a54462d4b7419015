"""Lagusun written out from its equations: whole sequences, float64, one function per mechanism.

Slow and plain on purpose: explicit ``[n, n]`` score matrices, Python loops over heads and experts.
It reads the design's ``config.json`` dictionary itself and takes the checkpoint's tensors by their
stored names; nothing of the package is imported, so the engine and this file can only agree by
computing the same design.

``rounding=torch.bfloat16`` rounds the results of the matrix products and of the activations that
the design allows in 16 bits, which shows how far 16-bit storage alone moves the logits.
"""

from __future__ import annotations

import math
from typing import List, Mapping, Optional

import torch

F64 = torch.float64


def _r(x: torch.Tensor, rounding) -> torch.Tensor:
    return x if rounding is None else x.to(rounding).to(F64)


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """``x / sqrt(mean(x^2) + eps)`` over the last axis."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def grouped_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """Every one of ``groups`` equal runs of neighbouring coordinates has a root mean square of its own."""
    n = x.shape[-1] // groups
    parts = [unit_rms(x[..., g * n:(g + 1) * n], eps) for g in range(groups)]
    return torch.cat(parts, dim=-1) * w


def frequencies(dims: int, base: float, scaling: Optional[Mapping]) -> List[float]:
    """Angle per position of every rotated pair; ``scaling`` stretches the long wavelengths."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            length = 2.0 * math.pi / f
            lo, hi, orig, factor = scaling["low"], scaling["high"], scaling["original"], scaling["factor"]
            if length > orig / lo:
                f = f / factor
            elif length >= orig / hi:
                s = (orig / length - lo) / (hi - lo)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate(x: torch.Tensor, rot: Mapping) -> torch.Tensor:
    """``x [n, heads, d]``: coordinate ``i`` of a head turns with coordinate ``i + dims/2``, for the first
    ``dims`` of them, row ``p`` by ``p`` times the pair's frequency."""
    half = rot["dims"] // 2
    if half == 0:
        return x
    freq = torch.tensor(frequencies(rot["dims"], rot["base"], rot.get("scaling")), dtype=F64)
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * freq[None, :]
    cos, sin = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half:]], dim=-1)


def same_chunk(n: int, size: int) -> torch.Tensor:
    """``[n, n]``: row ``i`` sees column ``j`` of its own chunk, up to itself."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & (i // size == j // size)


def near_past(n: int, size: int) -> torch.Tensor:
    """``[n, n]``: row ``i`` sees itself and the ``size - 1`` columns before it."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & (i - j < size)


def softmax_with_zero_sink(s: torch.Tensor, seen: torch.Tensor) -> torch.Tensor:
    """Softmax over the seen columns with ``exp(0)`` added to the denominator."""
    s = s.masked_fill(~seen, float("-inf"))
    m = s.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-m))


def sigmoid_weights(s: torch.Tensor, seen: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """Every seen column's weight by itself."""
    return torch.sigmoid(s + bias).masked_fill(~seen, 0.0)


def chunked_attention(h, W: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float, rounding) -> torch.Tensor:
    n = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = _r(h @ W[p + ".q"].T, rounding)
    k = _r(h @ W[p + ".k"].T, rounding)
    v = k.view(n, G, d)
    q = (unit_rms(q, eps) * W[p + ".q.norm"]).view(n, H, d)
    k = (unit_rms(k, eps) * W[p + ".k.norm"]).view(n, G, d)
    q, k = _r(rotate(q, m["rot"]), rounding), _r(rotate(k, m["rot"]), rounding)
    seen = same_chunk(n, m["mask"]["size"])
    heads = []
    for a in range(H):
        g = a // (H // G)
        w = softmax_with_zero_sink(q[:, a] @ k[:, g].T * m["scale"], seen)
        heads.append(w @ v[:, g])
    return _r(_r(torch.cat(heads, dim=-1), rounding) @ W[p + ".o"].T, rounding)


def window_attention(h, W: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float, rounding) -> torch.Tensor:
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = _r(h @ W[p + ".q"].T + W[p + ".q.b"], rounding).view(n, H, d)
    k = _r(h @ W[p + ".k"].T + W[p + ".k.b"], rounding).view(n, G, d)
    v = _r(h @ W[p + ".v"].T + W[p + ".v.b"], rounding).view(n, G, dv)
    q = _r(unit_rms(rotate(q, m["rot"]), eps), rounding)
    k = _r(unit_rms(rotate(k, m["rot"]), eps), rounding)
    v = _r(unit_rms(v, eps), rounding)
    seen = near_past(n, m["mask"]["size"])
    cap = m["softcap"]
    heads = []
    for a in range(H):
        g = a // (H // G)
        s = q[:, a] @ k[:, g].T * m["scale"]
        s = cap * torch.tanh(s / cap)
        heads.append(sigmoid_weights(s, seen, W[p + ".pb"][a]) @ v[:, g])
    return _r(_r(torch.cat(heads, dim=-1), rounding) @ W[p + ".o"].T, rounding)


def erf_gelu(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def expert(h, W, p: str, rounding) -> torch.Tensor:
    u = _r(erf_gelu(_r(h @ W[p + ".up"].T, rounding)), rounding)
    return _r(u @ W[p + ".down"].T, rounding)


def route(z: torch.Tensor, correction: torch.Tensor, router: Mapping, margins_out: Optional[list] = None):
    """``z [n, E]`` logits -> ``(chosen [n, top], weights [n, top])``.  ``margins_out`` receives, per token, how far
    the last expert chosen stood above the first one left out."""
    s = torch.sigmoid(z)
    ordered = (s + correction).sort(-1, descending=True)
    top = router["top"]
    if margins_out is not None and top < router["experts"]:
        margins_out.append(ordered.values[:, top - 1] - ordered.values[:, top])
    chosen = ordered.indices[:, :top]
    w = s.gather(1, chosen)
    return chosen, w / (w.sum(-1, keepdim=True) + 1e-20) * router["scale"]


def experts_ffn(h, W, p: str, mlp: Mapping, rounding, margins_out: Optional[list] = None) -> torch.Tensor:
    z = _r(h, rounding) @ W[p + ".router"].T
    chosen, w = route(z, W[p + ".correction"], mlp["router"], margins_out)
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, slot = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += w[rows, slot][:, None] * expert(h[rows], W, f"{p}.e{e}", rounding)
    if mlp.get("shared"):
        out = out + expert(h, W, p + ".shared", rounding)
    return _r(out, rounding)


def run_order(config: Mapping) -> List[tuple]:
    """``(layer, pass number or None)`` of every layer run; a number stands on the first layer of every pass."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def enter_pass(x: torch.Tensor, x0: torch.Tensor, W, t: int, rounding) -> torch.Tensor:
    """What a pass over the looped layers starts from: a product of the stream beside the embedding output, and
    the pass's own row."""
    both = torch.cat([_r(x, rounding), _r(x0, rounding)], dim=-1)
    return both @ W["loop.in"].T + W["loop.step"][t]


def forward(config: Mapping, W: Mapping[str, torch.Tensor], tokens, rounding=None, layers_out: Optional[list] = None,
            margins_out: Optional[list] = None) -> torch.Tensor:
    """Logits ``[n, vocab]`` (float64) of one whole sequence.  ``layers_out`` receives the stream after every layer
    run, ``margins_out`` the routers' margins (see :func:`route`)."""
    W = {k: v.to(F64) for k, v in W.items()}
    eps, groups = config["norm"]["eps"], config["norm"]["groups"]
    x0 = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    x = x0
    for i, t in run_order(config):
        if t is not None:
            x = enter_pass(x, x0, W, t, rounding)
        layer, p = config["layers"][i], f"l{i}"
        mixer = chunked_attention if layer["type"] == "attention" else window_attention
        h = _r(grouped_norm(x, W[p + ".norm1"], groups, eps), rounding)
        x = x + mixer(h, W, p + ".mix", layer["mixer"], eps, rounding) * W[p + ".ls1"]
        if layer.get("mlp"):
            h = _r(grouped_norm(x, W[p + ".norm2"], groups, eps), rounding)
            x = x + experts_ffn(h, W, p + ".mlp", layer["mlp"], rounding, margins_out) * W[p + ".ls2"]
        if layers_out is not None:
            layers_out.append(x.clone())
    return _r(grouped_norm(x, W["final.norm"], groups, eps), rounding) @ W["head"].T
