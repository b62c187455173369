"""``CudaLayeredModel`` — decoders whose configuration lists their layers one by one, each with its own token
mixer, feed-forward and sizes (``OrionLayeredDesc`` in include/orion_cuda.h) — and the readers of Metapel's and Zulozen's
``config.json``."""
from __future__ import annotations

import ctypes as C
import json
import os
from dataclasses import dataclass, field
from typing import List, Optional

import numpy as np

from . import _ffi
from .backend import CudaBackend
from .errors import ModelError, check
from .model import CudaModel
from .types import DType


MIXERS = {"mingru": _ffi.MIXER_MIN_GRU, "latent_attention": _ffi.MIXER_LATENT_ATTENTION, "attention": _ffi.MIXER_ATTENTION}
ACTIVATIONS = {"gelu_tanh": _ffi.ACT_GELU_TANH, "relu2": _ffi.ACT_RELU2}
BLOCKS = {"parallel": _ffi.BLOCK_PARALLEL, "sandwich": _ffi.BLOCK_SANDWICH}


@dataclass(frozen=True)
class LayerSpec:
    """One layer: its mixer ("mingru", "latent_attention" or "attention"), the mixer's sizes, its feed-forward (0 = none)."""
    mixer: str
    ffn_dim: int = 0
    # mingru
    width: int = 0
    # both kinds of attention; window 0 = every earlier token is seen
    heads: int = 0
    dim: int = 0
    rot_dim: int = 0  # latent_attention
    value_dim: int = 0
    kv_rank: int = 0  # latent_attention
    window: int = 0
    rope_dims: int = 0
    rope_base: float = 0.0
    scale: float = 0.0
    # attention; chunk 0 = no chunks
    kv_heads: int = 0
    chunk: int = 0
    qk_norm: bool = False
    sinks: bool = False
    head_gate: bool = False
    # dense feed-forward
    activation: str = "gelu_tanh"
    ffn_bias: bool = False
    # mixture of experts of width ffn_dim (experts 0 = dense); shared_dim 0 = no shared expert
    experts: int = 0
    experts_per_token: int = 0
    shared_dim: int = 0

    def _c(self) -> "_ffi.OrionLayerDesc":
        return _ffi.OrionLayerDesc(
            MIXERS[self.mixer], self.ffn_dim, self.width, self.heads, self.dim, self.rot_dim, self.value_dim, self.kv_rank,
            self.window, self.rope_dims, self.rope_base, self.scale, self.kv_heads, self.chunk, int(self.qk_norm),
            int(self.sinks), int(self.head_gate), ACTIVATIONS[self.activation], int(self.ffn_bias), self.experts,
            self.experts_per_token, self.shared_dim)

    def cache_values_per_token(self) -> int:
        if self.mixer == "latent_attention":
            return self.kv_rank + self.rot_dim
        return self.kv_heads * (self.dim + self.value_dim) if self.mixer == "attention" else 0


@dataclass
class LayeredMetadata:
    architecture: str
    name: str
    hidden_size: int
    vocab_size: int
    layers: List[LayerSpec]
    norm_eps: float
    conv_taps: int = 0  # parallel blocks
    dtype: DType = DType.BF16
    eos_token_ids: List[int] = field(default_factory=list)
    block: str = "parallel"
    untied_lm_head: bool = False
    residual_mult: float = 1.0  # sandwich blocks

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def cache_values_per_token(self) -> int:
        """Values the paged cache holds per token, over all layers."""
        return sum(s.cache_values_per_token() for s in self.layers)

    @classmethod
    def from_config(cls, config: dict, name: str = "model") -> "LayeredMetadata":
        """The ``config.json`` of any design in ``READERS``."""
        try:
            if config["architecture"] not in READERS:
                raise ModelError(f"unsupported architecture {config['architecture']}")
            return READERS[config["architecture"]](config, name)
        except (KeyError, TypeError, ValueError) as e:
            raise ModelError(f"config.json is malformed: {type(e).__name__}: {e}") from e

    @classmethod
    def load(cls, directory: str) -> "LayeredMetadata":
        path = os.path.join(directory, "config.json")
        try:
            with open(path) as f:
                config = json.load(f)
        except OSError as e:
            raise ModelError(f"{path}: {e}") from e
        except ValueError as e:
            raise ModelError(f"config.json is malformed: {e}") from e
        return cls.from_config(config, os.path.basename(os.path.normpath(directory)) or "model")


def _read_metapel(config: dict, name: str) -> LayeredMetadata:
    specs = [_metapel_layer(i, entry) for i, entry in enumerate(config["layers"])]
    return LayeredMetadata(architecture=config["architecture"], name=name, hidden_size=int(config["width"]),
                           vocab_size=int(config["vocab"]), layers=specs, norm_eps=float(config["norm"]["eps"]),
                           conv_taps=int(config["canon"]["taps"]))


def _metapel_layer(i: int, entry: dict) -> LayerSpec:
    kind, m, mlp = entry["type"], entry["mixer"], entry["mlp"]
    ffn = 0
    if mlp is not None:
        if mlp["kind"] != "dense":
            raise ModelError(f"unsupported feed-forward {mlp['kind']!r} in layer {i}")
        ffn = int(mlp["ff"])
    if kind == "mingru":
        return LayerSpec("mingru", ffn, width=int(m["width"]))
    if kind == "latent_attention":
        return LayerSpec("latent_attention", ffn, heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]),
                         value_dim=int(m["vdim"]), kv_rank=int(m["kv_rank"]), window=_mask_size(m),
                         rope_dims=int(m["rot"]["dims"]), rope_base=float(m["rot"]["base"]), scale=float(m["scale"]))
    raise ModelError(f"unsupported mixer {kind!r} in layer {i}")


def _read_zulozen(config: dict, name: str) -> LayeredMetadata:
    specs = [_zulozen_layer(i, entry) for i, entry in enumerate(config["layers"])]
    return LayeredMetadata(architecture=config["architecture"], name=name, hidden_size=int(config["width"]),
                           vocab_size=int(config["vocab"]), layers=specs, norm_eps=float(config["norm"]["eps"]),
                           block="sandwich", untied_lm_head=True, residual_mult=float(config["residual_mult"]))


def _zulozen_layer(i: int, entry: dict) -> LayerSpec:
    kind, m, mlp = entry["type"], entry["mixer"], entry["mlp"]
    if kind != "attention":
        raise ModelError(f"unsupported mixer {kind!r} in layer {i}")
    ffn = {}
    if mlp is not None and mlp["kind"] == "dense":
        ffn = dict(ffn_dim=int(mlp["ff"]), activation="relu2", ffn_bias=True)
    elif mlp is not None and mlp["kind"] == "moe":
        shared = mlp.get("shared")
        ffn = dict(ffn_dim=int(mlp["expert"]["ff"]), experts=int(mlp["router"]["experts"]),
                   experts_per_token=int(mlp["router"]["top"]), shared_dim=int(shared["ff"]) if shared else 0)
    elif mlp is not None:
        raise ModelError(f"unsupported feed-forward {mlp['kind']!r} in layer {i}")
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    return LayerSpec("attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), value_dim=int(m["vdim"]),
                     chunk=_mask_size(m), rope_dims=int(rot["dims"]), rope_base=float(rot["base"]), scale=float(m["scale"]),
                     qk_norm=True, sinks=True, head_gate=True, **ffn)


def _mask_size(mixer: dict) -> int:
    return int(mixer["mask"]["size"]) if mixer.get("mask") else 0


#: config.json "architecture" -> reader
READERS = {"Metapel": _read_metapel, "Zulozen": _read_zulozen}


class CudaLayeredModel(CudaModel):
    """A GPU-executing layer-list model. Weights arrive through ``load_tensor`` / ``load_state`` /
    ``load_checkpoint``. If ``num_state_slots()`` is not 0, batches name a state slot per sequence
    (``ForwardBatch.state_slots``, handed out by a ``KvCacheManager`` made with ``num_state_slots``)."""

    def __init__(self, meta: LayeredMetadata, num_blocks: int, block_size: int, backend: CudaBackend, *,
                 compute_dtype: DType = DType.BF16, max_batch_tokens: int = 8192, max_batch_sequences: int = 256,
                 num_state_slots: Optional[int] = None, max_positions: Optional[int] = None):
        self._meta, self._backend, self._h = meta, backend, C.c_void_p()
        self.compute_dtype, self.num_blocks, self.block_size = compute_dtype, num_blocks, block_size
        layers = (_ffi.OrionLayerDesc * max(1, meta.num_layers))(*[s._c() for s in meta.layers])
        d = _ffi.OrionLayeredDesc(
            meta.hidden_size, meta.vocab_size, meta.num_layers, layers, meta.norm_eps, meta.conv_taps,
            max_positions or num_blocks * block_size,  # no sequence is longer than the whole cache
            num_blocks, block_size, num_state_slots or max_batch_sequences, int(compute_dtype), max_batch_tokens,
            max_batch_sequences, BLOCKS[meta.block], int(meta.untied_lm_head), meta.residual_mult)
        check(_ffi.lib().orion_cuda_model_create_layered(backend._h, C.byref(d), C.byref(self._h)))

    @classmethod
    def new(cls, meta: LayeredMetadata, weights, num_blocks: int, block_size: int, backend: CudaBackend,
            **kw) -> "CudaLayeredModel":
        m = cls(meta, num_blocks, block_size, backend, **kw)
        m.load_state(weights)
        return m

    @classmethod
    def from_directory(cls, directory: str, num_blocks: int, block_size: int, backend: CudaBackend,
                       **kw) -> "CudaLayeredModel":
        m = cls(LayeredMetadata.load(directory), num_blocks, block_size, backend, **kw)
        m.load_checkpoint(directory)
        return m

    def read_kv(self) -> List[np.ndarray]:
        """The caches of the attention layers in f32, one after the other: latents as ``[block][slot][kv_rank + rot_dim]``, keys
        and values as two arrays ``[block][kv head][slot][dim]``."""
        shapes = []
        for s in self._meta.layers:
            if s.mixer == "latent_attention":
                shapes.append((self.num_blocks, self.block_size, s.kv_rank + s.rot_dim))
            elif s.mixer == "attention":
                shapes += [(self.num_blocks, s.kv_heads, self.block_size, n) for n in (s.dim, s.value_dim)]
        sizes = [int(np.prod(s)) for s in shapes]
        out = np.zeros(max(1, sum(sizes)), np.float32)
        check(_ffi.lib().orion_cuda_model_read_kv(self._h, out.ctypes.data_as(C.POINTER(C.c_float)), out.size))
        ends = np.cumsum(sizes)
        return [out[e - n:e].reshape(s) for e, n, s in zip(ends, sizes, shapes)]
