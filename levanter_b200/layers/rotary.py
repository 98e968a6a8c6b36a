"""Rotary position embeddings: default (with linear ``factor``), Llama-3 smoothing, and YaRN.

Frequencies are computed exactly as the reference does (src/levanter/layers/rotary.py:30-46 default,
:97-136 llama3, :186-229 yarn incl. the mscale temperature on cos/sin) with the Hugging Face half-split
``rotate_half`` convention (:17-22).  The cos/sin table is built once per (config, head_dim, length) on
the host side of the model and applied either by the fused CUDA kernel (``ops.rope``) or by PyTorch ops.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from ..config import ChoiceRegistry


def rotate_half(x: torch.Tensor) -> torch.Tensor:
    h = x.shape[-1] // 2
    return torch.cat((-x[..., h:], x[..., :h]), dim=-1)


class RotaryEmbeddings:
    """Callable that rotates ``q`` (``[..., pos, heads..., head_dim]`` with positions given explicitly).

    The first ``rotary_dim = 2 * len(inv_freq)`` dimensions of a head turn, the rest pass.  Dimension ``i`` is paired with ``i +
    rotary_dim / 2``, or, ``interleaved``, ``2i`` with ``2i + 1``."""

    def __init__(self, head_dim: int, inv_freq: torch.Tensor, position_scale: float = 1.0, temperature: float = 1.0, interleaved: bool = False):
        self.head_dim = head_dim
        self.inv_freq = inv_freq.float()  # [rotary_dim // 2]
        self.position_scale = position_scale
        self.temperature = temperature
        self.interleaved = interleaved
        self._cache: dict = {}

    @property
    def rotary_dim(self) -> int:
        return 2 * self.inv_freq.shape[0]

    @property
    def is_plain(self) -> bool:
        """Whole heads in the half-split layout: what the tables of :meth:`cos_sin` and :meth:`table` describe."""
        return self.rotary_dim == self.head_dim and not self.interleaved

    def frequencies_on(self, device) -> torch.Tensor:
        """``inv_freq`` on a device, kept: its address goes into captured graphs."""
        key = ("inv_freq", str(device))
        if key not in self._cache:
            self._cache[key] = self.inv_freq.to(device).contiguous()
        return self._cache[key]

    def cos_sin(self, position_ids: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
        """cos, sin of shape ``position_ids.shape + [rotary_dim]`` in fp32 (half-split layout)."""
        inv = self.inv_freq.to(position_ids.device)
        freqs = (position_ids.float() * self.position_scale).unsqueeze(-1) * inv
        emb = torch.cat((freqs, freqs), dim=-1)
        return torch.cos(emb) * self.temperature, torch.sin(emb) * self.temperature

    def table(self, seq_len: int, device) -> Tuple[torch.Tensor, torch.Tensor]:
        """Cached ``[seq_len, head_dim]`` fp32 cos/sin tables for positions ``0..seq_len-1``."""
        key = (seq_len, str(device))
        if key not in self._cache:
            pos = torch.arange(seq_len, device=device)
            cos, sin = self.cos_sin(pos)
            self._cache[key] = (cos.contiguous(), sin.contiguous())
        return self._cache[key]

    def __call__(self, q: torch.Tensor, position_ids: torch.Tensor) -> torch.Tensor:
        """``q``: ``[batch?, pos, heads, head_dim]``; ``position_ids``: ``[pos]`` or ``[batch, pos]``."""
        cos, sin = self.cos_sin(position_ids)
        cos = cos.unsqueeze(-2)
        sin = sin.unsqueeze(-2)
        r = self.rotary_dim
        x = q[..., :r].float()
        if self.interleaved:
            half = r // 2
            cos, sin = cos[..., :half], sin[..., :half]
            u, v = x[..., 0::2], x[..., 1::2]
            out = torch.stack((u * cos - v * sin, v * cos + u * sin), dim=-1).flatten(-2)
        else:
            out = x * cos + rotate_half(x) * sin
        out = out.to(q.dtype)
        return out if r == q.shape[-1] else torch.cat((out, q[..., r:]), dim=-1)


def _base_inv_freq(theta: float, head_dim: int) -> torch.Tensor:
    return 1.0 / (theta ** (torch.arange(0, head_dim, 2, dtype=torch.float32) / head_dim))


@dataclass(frozen=True)
class RotaryEmbeddingsConfig(ChoiceRegistry):
    @classmethod
    def default_choice_name(cls) -> Optional[str]:
        return "default"

    def build(self, head_dim: int) -> RotaryEmbeddings:
        raise NotImplementedError

    @staticmethod
    def from_hf_config(rope_theta: float, config: Optional[dict]) -> "RotaryEmbeddingsConfig":
        if config is None:
            return DefaultRotaryEmbeddingsConfig(theta=rope_theta)
        tpe = config.get("rope_type", config.get("type", "default"))
        if tpe in ("default", "linear"):
            return DefaultRotaryEmbeddingsConfig(theta=rope_theta, factor=float(config.get("factor", 1.0)))
        if tpe == "llama3":
            return Llama3RotaryEmbeddingsConfig.make_from_hf_config(rope_theta, config)
        if tpe == "yarn":
            return YarnRotaryEmbeddingsConfig.make_from_hf_config(rope_theta, config)
        raise ValueError(f"unknown rope scaling type {tpe}")

    def to_hf_config(self) -> Tuple[float, Optional[dict]]:
        raise NotImplementedError


@RotaryEmbeddingsConfig.register_subclass("default")
@dataclass(frozen=True)
class DefaultRotaryEmbeddingsConfig(RotaryEmbeddingsConfig):
    theta: float = 10000
    factor: float = 1.0
    rotary_dim: Optional[int] = None  # the first dimensions of a head that turn; None: all
    interleaved: bool = False         # dimension 2i is paired with 2i + 1, not i with i + rotary_dim / 2

    def build(self, head_dim: int) -> RotaryEmbeddings:
        r = self.rotary_dim if self.rotary_dim is not None else head_dim
        if r % 2 != 0 or not 0 < r <= head_dim:
            raise ValueError(f"cannot rotate {r} of {head_dim} dimensions")
        return RotaryEmbeddings(head_dim, _base_inv_freq(self.theta, r) / self.factor, interleaved=self.interleaved)

    def to_hf_config(self):
        if self.rotary_dim is not None or self.interleaved:
            raise ValueError("a partial or interleaved rotation has no Hugging Face rope config")
        if self.factor == 1.0:
            return self.theta, None
        return self.theta, {"rope_type": "linear", "factor": self.factor}


RotaryEmbeddingsConfig.register_subclass("linear")(DefaultRotaryEmbeddingsConfig)
DefaultRotaryEmbeddingsConfig._choice_name = "default"


@RotaryEmbeddingsConfig.register_subclass("llama3")
@dataclass(frozen=True)
class Llama3RotaryEmbeddingsConfig(RotaryEmbeddingsConfig):
    theta: float = 500000
    factor: float = 8.0
    low_freq_factor: float = 1.0
    high_freq_factor: float = 4.0
    original_max_position_embeddings: int = 8192

    def build(self, head_dim: int) -> RotaryEmbeddings:
        inv_freq = _base_inv_freq(self.theta, head_dim)
        old = self.original_max_position_embeddings
        low_wavelen = old / self.low_freq_factor
        high_wavelen = old / self.high_freq_factor
        wavelen = 2 * math.pi / inv_freq
        inv_llama = torch.where(wavelen > low_wavelen, inv_freq / self.factor, inv_freq)
        smooth = (old / wavelen - self.low_freq_factor) / (self.high_freq_factor - self.low_freq_factor)
        smoothed = (1 - smooth) * inv_llama / self.factor + smooth * inv_llama
        medium = (~(wavelen < high_wavelen)) & (~(wavelen > low_wavelen))
        inv_llama = torch.where(medium, smoothed, inv_llama)
        return RotaryEmbeddings(head_dim, inv_llama)

    @classmethod
    def make_from_hf_config(cls, rope_theta: float, config: dict):
        return cls(theta=rope_theta, factor=float(config.get("factor", 8.0)),
                   low_freq_factor=float(config.get("low_freq_factor", 1.0)),
                   high_freq_factor=float(config.get("high_freq_factor", 4.0)),
                   original_max_position_embeddings=int(config.get("original_max_position_embeddings", 8192)))

    def to_hf_config(self):
        return self.theta, {"rope_type": "llama3", "factor": self.factor, "low_freq_factor": self.low_freq_factor,
                            "high_freq_factor": self.high_freq_factor,
                            "original_max_position_embeddings": self.original_max_position_embeddings}


@RotaryEmbeddingsConfig.register_subclass("yarn")
@dataclass(frozen=True)
class YarnRotaryEmbeddingsConfig(RotaryEmbeddingsConfig):
    theta: float = 10000
    factor: float = 1.0
    beta_fast: float = 32.0
    beta_slow: float = 1.0
    original_max_position_embeddings: int = 2048
    mscale: float = 1.0

    def build(self, head_dim: int) -> RotaryEmbeddings:
        half = head_dim // 2
        inv_freq = _base_inv_freq(self.theta, head_dim)

        def find_dim(n_rot: float) -> float:
            return (half * math.log(self.original_max_position_embeddings / (n_rot * 2 * math.pi))) / (2 * math.log(self.theta))

        low = int(math.floor(find_dim(self.beta_fast)))
        high = int(math.ceil(find_dim(self.beta_slow)))
        low, high = max(low, 0), min(high, half - 1)
        ramp = torch.clamp((torch.arange(half, dtype=torch.float32) - low) / max(high - low, 1), 0.0, 1.0)
        inv = (inv_freq / self.factor) * ramp + inv_freq * (1 - ramp)
        temperature = 1.0 if self.factor < 1.0 else math.sqrt(0.1 * self.mscale * math.log(self.factor) + 1.0)
        return RotaryEmbeddings(head_dim, inv, position_scale=1.0 / self.factor, temperature=temperature)

    @classmethod
    def make_from_hf_config(cls, rope_theta: float, config: dict):
        return cls(theta=rope_theta, factor=float(config.get("factor", 1.0)), beta_fast=float(config.get("beta_fast", 32.0)),
                   beta_slow=float(config.get("beta_slow", 1.0)),
                   original_max_position_embeddings=int(config.get("original_max_position_embeddings", 2048)),
                   mscale=float(config.get("mscale", 1.0)))

    def to_hf_config(self):
        return self.theta, {"type": "yarn", "factor": self.factor, "beta_fast": self.beta_fast, "beta_slow": self.beta_slow,
                            "original_max_position_embeddings": self.original_max_position_embeddings, "mscale": self.mscale}


@RotaryEmbeddingsConfig.register_subclass("yarn_partial")
@dataclass(frozen=True)
class PartialYarnRotaryEmbeddingsConfig(RotaryEmbeddingsConfig):
    """YaRN over the first ``rotary_dim`` dimensions of a head: a frequency that turns ``beta_fast`` times or more within the original
    context stays, one that turns ``beta_slow`` times or less is divided by ``factor``, with a ramp over the pairs in between; cos and
    sin are multiplied by ``0.1 ln(factor) + 1``.  (:class:`YarnRotaryEmbeddingsConfig` keeps another published variant's ramp,
    position scale and temperature.)"""

    theta: float = 10000
    factor: float = 1.0
    beta_fast: float = 32.0
    beta_slow: float = 1.0
    original_max_position_embeddings: int = 2048
    rotary_dim: Optional[int] = None  # the first dimensions of a head that turn; None: all

    def build(self, head_dim: int) -> RotaryEmbeddings:
        r = self.rotary_dim if self.rotary_dim is not None else head_dim
        if r % 2 != 0 or not 0 < r <= head_dim:
            raise ValueError(f"cannot rotate {r} of {head_dim} dimensions")

        def pair_of(turns: float) -> float:  # (fractional) pair that turns that often within the original context
            return r * math.log(self.original_max_position_embeddings / (2 * math.pi * turns)) / (2 * math.log(self.theta))

        low = max(math.floor(pair_of(self.beta_fast)), 0)
        high = min(math.ceil(pair_of(self.beta_slow)), r - 1)
        i = torch.arange(r // 2, dtype=torch.float64)
        ramp = ((i - low) / max(high - low, 0.001)).clamp(0.0, 1.0)
        freq = float(self.theta) ** (-2.0 * i / r)
        return RotaryEmbeddings(head_dim, freq / self.factor * ramp + freq * (1.0 - ramp), temperature=0.1 * math.log(self.factor) + 1.0)

    def to_hf_config(self):
        raise ValueError("a partial rotation has no Hugging Face rope config")


def rope_config_from_hf(get, default_theta: float = 10000.0) -> RotaryEmbeddingsConfig:
    """RoPE config from an HF config accessor ``get(key, default)``: understands both the legacy ``rope_theta`` +
    ``rope_scaling`` keys and the merged ``rope_parameters`` dict of newer ``transformers`` releases."""
    params = get("rope_parameters", None)
    theta = get("rope_theta", None)
    scaling = get("rope_scaling", None)
    if isinstance(params, dict):
        if "rope_theta" not in params and any(isinstance(v, dict) for v in params.values()):
            # per-layer-type parameters (e.g. full_attention / sliding_attention): take the global one
            params = params.get("full_attention") or next(v for v in params.values() if isinstance(v, dict))
        theta = params.get("rope_theta", theta)
        if params.get("rope_type", params.get("type", "default")) != "default":
            scaling = {k: v for k, v in params.items() if k != "rope_theta"}
    if theta is None:
        theta = default_theta
    return RotaryEmbeddingsConfig.from_hf_config(float(theta), scaling)


def rope_to_hf_dict(rope: RotaryEmbeddingsConfig) -> dict:
    """Keys to merge into an HF config for ``rope``: legacy (``rope_theta``, ``rope_scaling``) and ``rope_parameters``."""
    theta, scaling = rope.to_hf_config()
    params = {"rope_theta": theta, "rope_type": "default"}
    if scaling:
        params.update(scaling)
        params["rope_type"] = scaling.get("rope_type", scaling.get("type", "default"))
        params.pop("type", None)
    return {"rope_theta": theta, "rope_scaling": scaling, "rope_parameters": params}


def rope_from_entry(rot: Optional[dict]) -> Optional[RotaryEmbeddingsConfig]:
    """The rotation that a layer's ``{base, dims, scaling: {factor, original, fast, slow}}`` entry describes (None: no rotation)."""
    if rot is None:
        return None
    s = rot.get("scaling")
    if s is None:
        return DefaultRotaryEmbeddingsConfig(theta=float(rot["base"]), rotary_dim=rot["dims"])
    return PartialYarnRotaryEmbeddingsConfig(theta=float(rot["base"]), rotary_dim=rot["dims"], factor=float(s["factor"]), beta_fast=float(s["fast"]),
                                             beta_slow=float(s["slow"]), original_max_position_embeddings=s["original"])


def rope_to_entry(rope: RotaryEmbeddingsConfig, head_dim: int) -> dict:
    """The inverse of :func:`rope_from_entry` for heads of ``head_dim``."""
    rot = dict(base=rope.theta, dims=head_dim if rope.rotary_dim is None else rope.rotary_dim)
    if isinstance(rope, PartialYarnRotaryEmbeddingsConfig):
        rot["scaling"] = dict(factor=rope.factor, original=rope.original_max_position_embeddings, fast=rope.beta_fast, slow=rope.beta_slow)
    elif not isinstance(rope, DefaultRotaryEmbeddingsConfig) or rope.interleaved or rope.factor != 1.0:
        raise ValueError(f"a layer entry cannot describe {rope}")
    return rot
