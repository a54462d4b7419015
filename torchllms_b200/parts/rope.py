"""Rotary position encoding with the llama3 frequency rescaling.

Reference: ``RotaryPositionalEmbeddings`` (torchllms/models/networks.py:204-352).
``rope_init`` (:252-282) builds ``theta_i = base^(-2i/hd)`` and, for
``rope_type == "llama3"``, rescales low frequencies by ``1/factor`` and blends
the middle band (:259-277); ``build_rope_cache`` (:284-297) tabulates
``cos(p * theta_i), sin(p * theta_i)`` in float32 for every position; ``forward``
(:321-352) rotates adjacent lanes ``(x[2i], x[2i+1])`` in float32.  Keys are
stored after rotation, values as they are (:551-553).

The table is built once on the host in float32, exactly as the reference does
it, and gathered by the kernel; the rotation itself runs in float32 in the
kernel that also writes K and V into their pages.
"""

from __future__ import annotations

import math
from typing import Any, Mapping, Optional

import torch

from .base import BuildEnv, PositionEncoding, register_position_encoding


def rotary_frequencies(head_dim: int, theta: float, scaling: Optional[Mapping[str, Any]] = None) -> torch.Tensor:
    """``[head_dim / 2]`` float32 angular frequencies (torchllms/models/networks.py:253-279)."""
    exponent = torch.arange(0, head_dim, 2)[: head_dim // 2].float() / head_dim
    freq = 1.0 / (theta ** exponent)
    scaling = dict(scaling or {})
    rope_type = scaling.get("rope_type", "default")
    if rope_type == "llama3":
        factor = scaling["factor"]
        low = scaling["low_freq_factor"]
        high = scaling["high_freq_factor"]
        original = scaling["original_max_position_embeddings"]
        wavelen = 2 * math.pi / freq
        scaled = torch.where(wavelen > original / low, freq / factor, freq)
        smooth = (original / wavelen - low) / (high - low)
        blended = (1 - smooth) * scaled / factor + smooth * scaled
        medium = ~(wavelen < original / high) & ~(wavelen > original / low)
        freq = torch.where(medium, blended, scaled)
    elif rope_type == "linear":
        freq = freq / float(scaling["factor"])         # every frequency divided by one factor
    elif rope_type != "default":
        raise ValueError(f"unknown rope_type {rope_type!r}")
    return freq


def rotary_table(freq: torch.Tensor, max_positions: int) -> torch.Tensor:
    """``[max_positions, head_dim / 2, 2]`` float32 (cos, sin) (torchllms/models/networks.py:284-297)."""
    positions = torch.arange(max_positions, dtype=freq.dtype)
    angles = torch.einsum("i,j->ij", positions, freq).float()
    return torch.stack([torch.cos(angles), torch.sin(angles)], dim=-1).contiguous()


_precise_tables: dict = {}


def band_scaled(freq: torch.Tensor, factor: float, low: float, high: float, original: float) -> torch.Tensor:
    """Frequencies rescaled by band (the llama3 rule) in ``freq``'s own precision: with wavelength
    ``l = 2 pi / f``, ``f`` stays where ``l < original / high``, becomes ``f / factor`` where ``l > original / low``,
    and between the two is blended by ``s = (original / l - low) / (high - low)``."""
    wavelen = 2.0 * math.pi / freq
    s = (original / wavelen - low) / (high - low) if high != low else torch.ones_like(freq)
    blended = (1.0 - s) * freq / factor + s * freq
    return torch.where(wavelen < original / high, freq, torch.where(wavelen > original / low, freq / factor, blended))


def ramp_scaled(freq: torch.Tensor, theta: float, factor: float, original: float, fast: float, slow: float):
    """Frequencies rescaled along a ramp (YaRN) in ``freq``'s own precision, and what cos and sin are multiplied by.
    ``freq[i] = theta^(-2i/dims)``.  The coordinate that turns ``n`` times within ``original`` positions is
    ``c(n) = dims ln(original / (2 pi n)) / (2 ln theta)``; pairs up to ``floor(c(fast))`` keep their frequency, pairs from
    ``ceil(c(slow))`` on are divided by ``factor``, and in between the two are blended linearly in the pair's number.  Cos
    and sin grow by ``0.1 ln(factor) + 1``."""
    dims = 2 * freq.numel()
    at = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
    lo, hi = max(math.floor(at(fast)), 0), min(math.ceil(at(slow)), dims - 1)
    i = torch.arange(freq.numel(), dtype=freq.dtype)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return freq / factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def precise_rotary_table(dims: int, theta: float, factor: float, max_positions: int, device="cpu",
                         band: Optional[Mapping[str, float]] = None, ramp: Optional[Mapping[str, float]] = None) -> torch.Tensor:
    """``[max_positions, dims / 2, 2]`` float32 (cos, sin) of the angles ``p * theta^(-2i/dims) / factor``,
    the angles taken in 64-bit so that the table is exact to float32 rounding at any position.
    ``band`` (``factor``, ``low``, ``high``, ``original``) rescales the frequencies by :func:`band_scaled`; ``ramp``
    (``factor``, ``original``, ``fast``, ``slow``) rescales frequencies and entries by :func:`ramp_scaled`.
    Layers with the same numbers on the same device share one table."""
    bands = None if band is None else tuple(float(band[k]) for k in ("factor", "low", "high", "original"))
    ramps = None if ramp is None else tuple(float(ramp[k]) for k in ("factor", "original", "fast", "slow"))
    key = (int(dims), float(theta), float(factor), int(max_positions), str(device), bands, ramps)
    table = _precise_tables.get(key)
    if table is None:
        i = torch.arange(dims // 2, dtype=torch.float64)
        freq = float(theta) ** (-2.0 * i / dims) / float(factor)
        if bands is not None:
            freq = band_scaled(freq, *bands)
        grow = 1.0
        if ramps is not None:
            freq, grow = ramp_scaled(freq, float(theta), *ramps)
        angles = torch.arange(max_positions, dtype=torch.float64)[:, None] * freq[None, :]
        table = (grow * torch.stack([torch.cos(angles), torch.sin(angles)], dim=-1)).to(torch.float32).contiguous().to(device)
        if len(_precise_tables) >= 8:
            _precise_tables.clear()
        _precise_tables[key] = table
    return table


@register_position_encoding("rope")
class RotaryEncoding(PositionEncoding):
    """``pairing`` is ``"interleaved"`` (lanes 2i, 2i+1: the reference's and Meta's
    convention) or ``"half"`` (lanes i, i + hd/2: Hugging Face's)."""

    graph_safe = True
    takes_row_scaled = True      # the kernel scales every row before it rotates and stores it

    def __init__(self, env: BuildEnv, *, head_dim: int, theta: float,
                 scaling: Optional[Mapping[str, Any]] = None, pairing: str = "interleaved"):
        if pairing not in ("interleaved", "half"):
            raise ValueError(f"rope pairing must be 'interleaved' or 'half', got {pairing!r}")
        self.env = env
        self.head_dim = int(head_dim)
        self.pairing = pairing
        self.freq = rotary_frequencies(self.head_dim, float(theta), scaling)
        self.table = rotary_table(self.freq, env.max_positions).to(env.device)

    def weight_bytes(self) -> int:
        return 0  # the table is gathered by rows, not streamed

    def encode_and_store(self, qkv, ctx, cache, n_heads: int, n_kv_heads: int, head_dim: int):
        return self.env.ops.rope_kv_write(
            qkv, ctx.positions, self.table,
            n_heads=n_heads, n_kv_heads=n_kv_heads, head_dim=head_dim,
            interleaved=(self.pairing == "interleaved"),
            k_pages=cache.k_pages if cache.writes else None,
            v_pages=cache.v_pages if cache.writes else None,
            slot_mapping=cache.slot_mapping, page_size=cache.page_size, out_dtype=self.env.dtype)
