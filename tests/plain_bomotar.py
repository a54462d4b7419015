"""Bomotar written out from its equations: whole sequences, float64, one function per mechanism.

Slow and plain on purpose: explicit ``[n, n]`` score matrices, token-by-token recurrences, Python
loops over heads and experts.  It reads the design's ``config.json`` dictionary itself and takes
the checkpoint's tensors by their stored names; nothing of the package is imported, so the engine
and this file can only agree by computing the same design.

``rounding=torch.bfloat16`` rounds the results of the matrix products, of the short convolutions and
of the activations, which the design allows in 16 bits: it shows how far 16-bit storage alone moves
the logits.  A function in its place rounds as it likes (:func:`either_way`).
"""

from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


def _r(x: torch.Tensor, rounding) -> torch.Tensor:
    if rounding is None:
        return x
    return rounding(x) if callable(rounding) else x.to(rounding).to(F64)


def either_way(seed: int):
    """A rounding to bfloat16's grid that goes up or down with the probabilities of the distances: another sample of what
    16-bit storage may do than rounding to nearest is."""
    g = torch.Generator().manual_seed(seed)

    def rounded(x: torch.Tensor) -> torch.Tensor:
        step = torch.exp2(torch.floor(torch.log2(x.abs().clamp(min=1e-30))) - 7)
        return torch.floor(x / step + torch.rand(x.shape, generator=g, dtype=F64)) * step
    return rounded


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + UNIT_EPS)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def bigram_rows(tokens: torch.Tensor, bigram: Mapping) -> torch.Tensor:
    """The row of the pair table that each place takes: the last one where there is no token before."""
    n = bigram["buckets"]
    rows = [n]
    for before, now in zip(tokens.tolist(), tokens.tolist()[1:]):
        rows.append((before * bigram["mul_prev"] + now * bigram["mul_cur"]) % n)
    return torch.tensor(rows[:len(tokens)])


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``y[t, c] = sum_j w[c, j] * u[t - taps + 1 + j, c]`` with zeros before the start."""
    n, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < n:
            y[back:] += u[:n - back] * w[:, j]
    return y


def frequencies(rot: Mapping) -> List[float]:
    """Angular frequencies of the rotated pairs; with ``scaling``, long wavelengths are stretched by a
    factor, short ones kept, and a ramp over the pair's number lies between."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not s:
        return f

    def pair_of(turns):          # which (fractional) coordinate turns so often within the original length
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(pair_of(s["fast"])), 0), min(math.ceil(pair_of(s["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * ramp + fi * (1.0 - ramp))
    return out


def rotate_half(x: torch.Tensor, rot: Mapping) -> torch.Tensor:
    """``x [n, heads, d]``: the first ``dims`` coordinates of every head turned by the position's angles."""
    n, dims, s = x.shape[0], rot["dims"], rot.get("scaling")
    half = dims // 2
    a = torch.arange(n, dtype=F64)[:, None] * torch.tensor(frequencies(rot), dtype=F64)[None, :]
    grow = 0.1 * math.log(s["factor"]) + 1.0 if s else 1.0
    c, d = grow * torch.cos(a)[:, None, :], grow * torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * d, v * c + u * d, x[..., dims:]], dim=-1)


def conv_attention(h, W: Mapping[str, torch.Tensor], p: str, cfg: Mapping, rounding) -> torch.Tensor:
    n = h.shape[0]
    H, G, d, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]

    def branch(name):
        return _r(causal_conv(_r(h @ W[f"{p}.{name}"].T, rounding), W[f"{p}.{name}.conv"]), rounding)

    q = _r(rotate_half(branch("q").view(n, H, d), cfg["rot"]), rounding)
    k = _r(rotate_half(branch("k").view(n, G, d), cfg["rot"]), rounding)
    v = branch("v").view(n, G, dv)
    later = torch.ones(n, n, dtype=torch.bool).triu(1)
    out = torch.zeros(n, H, dv, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T * cfg["scale"]).masked_fill(later, float("-inf"))
        out[:, a] = torch.softmax(s, dim=-1) @ v[:, g]
    gate = torch.sigmoid(_r(h @ W[p + ".g"].T, rounding))
    return _r(_r(out.reshape(n, H * dv) * gate, rounding) @ W[p + ".o"].T, rounding)


def channel_delta(q, k, v, beta, decay):
    """``q, k [n, G, d]``, ``v [n, H, dv]``, ``beta [n, H]``, ``decay [n, H, d]``: a matrix per head whose rows
    decay each at its own rate, then is corrected under the current key and read by the current query."""
    n, H, dv = v.shape
    G, d = k.shape[1:]
    of = [a // (H // G) for a in range(H)]           # the head of q and k that goes with head a
    S = torch.zeros(H, d, dv, dtype=F64)
    out = torch.zeros(n, H, dv, dtype=F64)
    for t in range(n):
        S = decay[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t, of]))
        S = S + k[t, of][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t, of])
    return out


def decay_of(h, W, p: str, cfg: Mapping, rounding) -> torch.Tensor:
    n, H, d = h.shape[0], cfg["heads"], cfg["dim"]
    z = _r(_r(h @ W[p + ".a1"].T, rounding) @ W[p + ".a2"].T, rounding) + W[p + ".dt_bias"]
    rate = torch.exp(W[p + ".A_log"])[:, None]
    return torch.exp(-rate * torch.nn.functional.softplus(z).view(n, H, d))


def delta_mixer(h, W, p: str, cfg: Mapping, eps: float, rounding) -> torch.Tensor:
    n = h.shape[0]
    H, G, d, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]

    def branch(name):
        y = _r(h @ W[f"{p}.{name}"].T, rounding)
        return _r(silu(_r(causal_conv(y, W[f"{p}.{name}.conv"]), rounding)), rounding)

    q = unit(branch("q").view(n, G, d)) * d ** -0.5
    k = unit(branch("k").view(n, G, d))
    beta = torch.sigmoid(_r(h @ W[p + ".b"].T, rounding))
    o = channel_delta(q, k, branch("v").view(n, H, dv), beta, decay_of(h, W, p, cfg, rounding))
    gate = torch.sigmoid(_r(_r(h @ W[p + ".g1"].T, rounding) @ W[p + ".g2"].T, rounding))
    o = (rms(o, eps) * W[p + ".norm"]).reshape(n, H * dv) * gate
    return _r(_r(o, rounding) @ W[p + ".o"].T, rounding)


def parallel_mixer(h, W, p: str, cfg: Mapping, eps: float, rounding) -> torch.Tensor:
    left = conv_attention(h, W, p + ".left", cfg["left"], rounding)
    right = delta_mixer(h, W, p + ".right", cfg["right"], eps, rounding)
    return cfg["left_scale"] * left + cfg["right_scale"] * right


def dense_ff(h, W, p: str, rounding) -> torch.Tensor:
    u = _r(gelu_tanh(_r(h @ W[p + ".up"].T, rounding)), rounding)
    return _r(u @ W[p + ".down"].T, rounding)


def route(z: torch.Tensor, correction: torch.Tensor, router: Mapping, margins_out: Optional[list] = None):
    """``z [n, E]`` logits -> ``(chosen [n, top], weights [n, top])``.  ``margins_out`` receives, per token, how
    close the choice was: of the experts, and of the groups."""
    n, E = z.shape
    s = torch.softmax(z, dim=-1)
    choice = s + correction
    groups = router.get("groups")
    margin = torch.full((n,), float("inf"), dtype=F64)
    if groups:
        per = E // groups["count"]
        best = choice.view(n, groups["count"], per).max(-1).values.sort(-1, descending=True)
        keep = groups["keep"]
        if keep < groups["count"]:
            margin = best.values[:, keep - 1] - best.values[:, keep]
        allowed = torch.zeros(n, groups["count"], dtype=torch.bool).scatter_(1, best.indices[:, :keep], True)
        choice = choice.masked_fill(~allowed.repeat_interleave(per, dim=1), float("-inf"))
    ordered, top = choice.sort(-1, descending=True), router["top"]
    if top < E:
        margin = torch.minimum(margin, ordered.values[:, top - 1] - ordered.values[:, top])
    if margins_out is not None:
        margins_out.append(margin)
    chosen = ordered.indices[:, :top]
    return chosen, s.gather(1, chosen)


def experts_ff(h, W, p: str, mlp: Mapping, rounding, margins_out: Optional[list] = None) -> torch.Tensor:
    chosen, w = route(h @ W[p + ".router"].T, W[p + ".correction"], mlp["router"], margins_out)
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            x = h[rows]
            u = _r(silu(_r(x @ W[f"{p}.e{e}.gate"].T, rounding)) * _r(x @ W[f"{p}.e{e}.up"].T, rounding), rounding)
            out[rows] += w[rows, place][:, None] * _r(u @ W[f"{p}.e{e}.down"].T, rounding)
    return _r(out, rounding)


def owner_of(config: Mapping, i: int) -> int:
    """The layer whose tensors layer ``i`` uses."""
    while config["layers"][i].get("weights_of") is not None:
        i = config["layers"][i]["weights_of"]
    return i


def forward(config: Mapping, tensors: Mapping[str, torch.Tensor], tokens, rounding=None, layers_out: Optional[list] = None,
            margins_out: Optional[list] = None) -> torch.Tensor:
    """Logits ``[n, vocab]`` (float64) of one whole sequence.  ``layers_out`` receives the stream after every
    layer, ``margins_out`` the routers' margins (see :func:`route`)."""
    W: Dict[str, torch.Tensor] = {k: v.to(F64) for k, v in tensors.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = W["embed"][tokens] + W["bigram"][bigram_rows(tokens, config["embedding"]["bigram"])]
    for i, layer in enumerate(config["layers"]):
        p, mlp = f"l{owner_of(config, i)}", layer.get("mlp")
        h = _r(rms(x, eps) * W[p + ".norm1"], rounding)
        x = x + m * (rms(parallel_mixer(h, W, p + ".mix", layer["mixer"], eps, rounding), eps) * W[p + ".norm1b"])
        if mlp is not None:
            h = _r(rms(x, eps) * W[p + ".norm2"], rounding)
            y = dense_ff(h, W, p + ".mlp", rounding) if mlp["kind"] == "dense" else \
                experts_ff(h, W, p + ".mlp", mlp, rounding, margins_out)
            x = x + m * (rms(y, eps) * W[p + ".norm2b"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return _r(rms(x, eps) * W["final.norm"], rounding) @ W["head"].T
