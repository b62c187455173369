"""``CudaLayeredModel`` — decoders whose configuration lists their layers one by one, each with its own token
mixer, feed-forward and sizes (``OrionLayeredDesc`` in include/orion_cuda.h) — and the readers of Metapel's, Zulozen's,
Belizen's and Vusenex's ``config.json``."""
from __future__ import annotations

import ctypes as C
import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import numpy as np

from . import _ffi
from .backend import CudaBackend
from .errors import ModelError, check
from .model import CudaModel, safetensors_shapes
from .types import DType


MIXERS = {"mingru": _ffi.MIXER_MIN_GRU, "latent_attention": _ffi.MIXER_LATENT_ATTENTION, "attention": _ffi.MIXER_ATTENTION,
          "gla": _ffi.MIXER_GLA}
ACTIVATIONS = {"gelu_tanh": _ffi.ACT_GELU_TANH, "relu2": _ffi.ACT_RELU2, "geglu_tanh": _ffi.ACT_GEGLU_TANH}
BLOCKS = {"parallel": _ffi.BLOCK_PARALLEL, "sandwich": _ffi.BLOCK_SANDWICH, "prenorm": _ffi.BLOCK_PRENORM,
          "gated_postnorm": _ffi.BLOCK_GATED_POSTNORM}
QK_NORMS = {False: _ffi.QK_NORM_NONE, True: _ffi.QK_NORM_ALL_HEADS, "per_head": _ffi.QK_NORM_PER_HEAD}
SINKS = {False: _ffi.SINK_NONE, True: _ffi.SINK_LEARNED, "zero": _ffi.SINK_ZERO}
ROUTERS = {"sigmoid_input": _ffi.ROUTER_SIGMOID_INPUT, "softmax": _ffi.ROUTER_SOFTMAX, "softmax_renorm": _ffi.ROUTER_SOFTMAX_RENORM}
EXPERT_FORMS = {"swiglu": _ffi.EXPERT_SWIGLU, "clamped": _ffi.EXPERT_CLAMPED, "gelu": _ffi.EXPERT_GELU}


@dataclass(frozen=True)
class Yarn:
    """Frequencies stretched by ``factor`` where they turn few times within ``original`` positions (``slow`` turns: wholly,
    ``fast`` turns: not at all)."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Loop:
    """Layers ``start`` to ``stop - 1`` run ``times`` times in a row; each pass keeps a cache and state of its own."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class Bigram:
    """A table of embeddings of pairs of tokens: row (previous * ``mul_prev`` + token * ``mul_cur``) mod ``buckets``, and a further row
    for a sequence's first token."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class QueryTemperature:
    """Queries are multiplied by 1 + ``coef`` ln(floor((position + 1) / ``every``) + 1)."""
    coef: float
    every: float


@dataclass(frozen=True)
class LayerSpec:
    """One layer: its mixer ("mingru", "latent_attention", "attention" or "gla"), the mixer's sizes, its feed-forward (0 = none)."""
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
    qk_norm: object = False  # False, True (over all heads at once) or "per_head"
    sinks: object = False  # False, True (a learned logit per head) or "zero"
    head_gate: bool = False
    # dense feed-forward
    activation: str = "gelu_tanh"
    ffn_bias: bool = False
    # mixture of experts of width ffn_dim (experts 0 = dense); shared_dim 0 = no shared expert
    experts: int = 0
    experts_per_token: int = 0
    shared_dim: int = 0
    # attention: first positions seen besides the window, pairs of dimensions half the rotated size apart, biases of q, k and v, a
    # gate per value, soft cap of the scores (0 = none)
    keep_first: int = 0
    rope_halves: bool = False
    qkv_bias: bool = False
    value_gate: bool = False
    softcap: float = 0.0
    yarn: Optional[Yarn] = None
    # gla (heads, dim and value_dim as above)
    decay_tau: float = 0.0
    decay_rank: int = 0
    # router and experts
    router: str = "sigmoid_input"
    router_identity: int = 0
    expert_form: str = "swiglu"
    expert_limit: float = 0.0
    shared_limit: float = 0.0
    router_groups: int = 0  # 0 = experts form no groups
    router_keep: int = 0
    # attention: the values are the keys before their norm; a learned logarithm of the distance is taken off the scores
    keys_as_values: bool = False
    distance_bias: bool = False
    q_temp: Optional[QueryTemperature] = None
    ungated: bool = False  # latent_attention: no gate on the output

    def _c(self) -> "_ffi.OrionLayerDesc":
        return _ffi.OrionLayerDesc(
            MIXERS[self.mixer], self.ffn_dim, self.width, self.heads, self.dim, self.rot_dim, self.value_dim, self.kv_rank,
            self.window, self.rope_dims, self.rope_base, self.scale, self.kv_heads, self.chunk, QK_NORMS[self.qk_norm],
            SINKS[self.sinks], int(self.head_gate), ACTIVATIONS[self.activation], int(self.ffn_bias), self.experts,
            self.experts_per_token, self.shared_dim, self.keep_first, int(self.rope_halves), int(self.qkv_bias),
            int(self.value_gate), self.softcap, *((y.factor, y.original, y.fast, y.slow) if (y := self.yarn) else (0.0,) * 4),
            self.decay_tau, self.decay_rank, ROUTERS[self.router], self.router_identity, EXPERT_FORMS[self.expert_form],
            self.expert_limit, self.shared_limit, self.router_groups, self.router_keep, int(self.keys_as_values),
            int(self.distance_bias), *((t.coef, t.every) if (t := self.q_temp) else (0.0, 0.0)), int(self.ungated))

    def cache_values_per_token(self) -> int:
        if self.mixer == "latent_attention":
            return self.kv_rank + self.rot_dim
        if self.keys_as_values:
            return self.kv_heads * self.dim  # besides an f32 factor per head
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
    residual_mult: float = 1.0  # sandwich and prenorm blocks
    embed_scale: float = 1.0
    logit_softcap: float = 0.0
    loop: Optional[Loop] = None
    scalar_norms: bool = False  # the gain of a norm of the stream's width is one number
    max_positions: int = 0  # rows of a table of learned positions; 0 = no such table
    bigram: Optional[Bigram] = None

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def layer_runs(self) -> List[LayerSpec]:
        """The layers in the order in which they run; a looped layer comes once per pass."""
        if self.loop is None:
            return list(self.layers)
        a, b = self.loop.start, self.loop.stop
        return self.layers[:a] + self.layers[a:b] * self.loop.times + self.layers[b:]

    def cache_values_per_token(self) -> int:
        """Values the paged cache holds per token, over all layer runs."""
        return sum(s.cache_values_per_token() for s in self.layer_runs())

    @classmethod
    def from_config(cls, config: dict, name: str = "model",
                    shapes: Optional[Dict[str, Tuple[int, ...]]] = None) -> "LayeredMetadata":
        """The ``config.json`` of any design in ``READERS``. ``shapes``: the checkpoint's tensors, for the sizes that no
        configuration gives."""
        try:
            if config["architecture"] not in READERS:
                raise ModelError(f"unsupported architecture {config['architecture']}")
            return READERS[config["architecture"]](config, name, shapes or {})
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
        return cls.from_config(config, os.path.basename(os.path.normpath(directory)) or "model", safetensors_shapes(directory))


def _read_metapel(config: dict, name: str, shapes: dict) -> LayeredMetadata:
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


def _read_zulozen(config: dict, name: str, shapes: dict) -> LayeredMetadata:
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


def _read_belizen(config: dict, name: str, shapes: dict) -> LayeredMetadata:
    specs = [_belizen_layer(i, entry, shapes) for i, entry in enumerate(config["layers"])]
    loop = config.get("loop")
    if loop is not None:
        loop = Loop(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not 0 <= loop.start < loop.stop <= len(specs) or loop.times < 1:
            raise ModelError(f"layers {loop.start} to {loop.stop} of {len(specs)} cannot be looped {loop.times} times")
    return LayeredMetadata(architecture=config["architecture"], name=name, hidden_size=int(config["width"]),
                           vocab_size=int(config["vocab"]), layers=specs, norm_eps=float(config["norm"]["eps"]),
                           block="prenorm", residual_mult=float(config["residual_mult"]),
                           embed_scale=float(config["embedding"]["scale"]), logit_softcap=float(config.get("logit_softcap") or 0.0),
                           loop=loop)


def _belizen_layer(i: int, entry: dict, shapes: dict) -> LayerSpec:
    kind, m, mlp = entry["type"], entry["mixer"], entry["mlp"]
    ffn = {}
    if mlp is not None and mlp["kind"] == "dense":
        ffn = dict(ffn_dim=int(mlp["ff"]), activation="geglu_tanh")
    elif mlp is not None and mlp["kind"] == "moe":
        router, shared = mlp["router"], mlp.get("shared")
        ffn = dict(ffn_dim=int(mlp["expert"]["ff"]), experts=int(router["experts"]), experts_per_token=int(router["top"]),
                   router="softmax", router_identity=int(router.get("identity") or 0), expert_form="clamped",
                   expert_limit=float(mlp["expert"]["limit"]), shared_dim=int(shared["ff"]) if shared else 0,
                   shared_limit=float(shared["limit"]) if shared else 0.0)
    elif mlp is not None:
        raise ModelError(f"unsupported feed-forward {mlp['kind']!r} in layer {i}")
    if kind == "gla":
        if f"l{i}.mix.a1" not in shapes:
            raise ModelError(f"missing tensor `l{i}.mix.a1`: its rows are the rank of the decays of layer {i}")
        return LayerSpec("gla", heads=int(m["heads"]), dim=int(m["dim"]), value_dim=int(m["vdim"]), decay_tau=float(m["tau"]),
                         decay_rank=int(shapes[f"l{i}.mix.a1"][0]), **ffn)
    if kind != "attention":
        raise ModelError(f"unsupported mixer {kind!r} in layer {i}")
    rot, mask = m.get("rot") or {"dims": 0, "base": 1.0}, m.get("mask") or {}
    yarn = rot.get("scaling")
    if yarn is not None:
        yarn = Yarn(float(yarn["factor"]), float(yarn["original"]), float(yarn["fast"]), float(yarn["slow"]))
    return LayerSpec("attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), value_dim=int(m["vdim"]),
                     window=_mask_size(m), keep_first=int(mask.get("keep_first") or 0), rope_dims=int(rot["dims"]),
                     rope_base=float(rot["base"]), yarn=yarn, rope_halves=True, scale=float(m["scale"]),
                     softcap=float(m.get("softcap") or 0.0), qk_norm="per_head", qkv_bias=True, value_gate=True, **ffn)


def _read_vusenex(config: dict, name: str, shapes: dict) -> LayeredMetadata:
    specs = [_vusenex_layer(i, entry) for i, entry in enumerate(config["layers"])]
    pairs = config["embedding"]["bigram"]
    return LayeredMetadata(architecture=config["architecture"], name=name, hidden_size=int(config["width"]),
                           vocab_size=int(config["vocab"]), layers=specs, norm_eps=float(config["norm"]["eps"]),
                           block="gated_postnorm", untied_lm_head=True, scalar_norms=True, max_positions=int(config["max_positions"]),
                           bigram=Bigram(int(pairs["buckets"]), int(pairs["mul_prev"]), int(pairs["mul_cur"])))


def _vusenex_layer(i: int, entry: dict) -> LayerSpec:
    kind, m, mlp = entry["type"], entry["mixer"], entry["mlp"]
    ffn = {}
    if mlp is not None and mlp["kind"] != "moe":
        raise ModelError(f"unsupported feed-forward {mlp['kind']!r} in layer {i}")
    if mlp is not None:
        router, shared, groups = mlp["router"], mlp.get("shared"), mlp["router"].get("groups") or {"count": 0, "keep": 0}
        ffn = dict(ffn_dim=int(mlp["expert"]["ff"]), experts=int(router["experts"]), experts_per_token=int(router["top"]),
                   router="softmax_renorm", router_groups=int(groups["count"]), router_keep=int(groups["keep"]), expert_form="gelu",
                   shared_dim=int(shared["ff"]) if shared else 0)
    if kind == "latent_attention":
        return LayerSpec("latent_attention", heads=int(m["heads"]), dim=int(m["dim"]), value_dim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                         scale=float(m["scale"]), ungated=True, **ffn)
    if kind != "attention":
        raise ModelError(f"unsupported mixer {kind!r} in layer {i}")
    if int(m["vdim"]) != int(m["dim"]):
        raise ModelError(f"layer {i}: values of {m['vdim']} dimensions cannot be keys of {m['dim']}")
    temp = m.get("q_temp")
    return LayerSpec("attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), value_dim=int(m["vdim"]),
                     scale=float(m["scale"]), qk_norm=True, qkv_bias=True, sinks="zero", keys_as_values=True, distance_bias=True,
                     q_temp=QueryTemperature(float(temp["coef"]), float(temp["every"])) if temp else None, **ffn)


def _mask_size(mixer: dict) -> int:
    return int(mixer["mask"]["size"]) if mixer.get("mask") else 0


#: config.json "architecture" -> reader
READERS = {"Metapel": _read_metapel, "Zulozen": _read_zulozen, "Belizen": _read_belizen, "Vusenex": _read_vusenex}


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
            min(max_positions or num_blocks * block_size,  # no sequence is longer than the whole cache
                meta.max_positions or 1 << 31),
            num_blocks, block_size, num_state_slots or max_batch_sequences, int(compute_dtype), max_batch_tokens,
            max_batch_sequences, BLOCKS[meta.block], int(meta.untied_lm_head), meta.residual_mult, meta.embed_scale,
            meta.logit_softcap, *((meta.loop.start, meta.loop.stop, meta.loop.times) if meta.loop else (0, 0, 0)),
            int(meta.scalar_norms), meta.max_positions, *((b.buckets, b.mul_prev, b.mul_cur) if (b := meta.bigram) else (0, 0, 0)))
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
        """The caches of the attention layers in f32, one after the other in the order in which they run: latents as ``[block][slot][kv_rank + rot_dim]``, keys
        and values as two arrays ``[block][kv head][slot][dim]``; where the values are the keys, one such array and the keys' factors
        ``[block][kv head][slot][1]``."""
        shapes = []
        for s in self._meta.layer_runs():
            if s.mixer == "latent_attention":
                shapes.append((self.num_blocks, self.block_size, s.kv_rank + s.rot_dim))
            elif s.mixer == "attention":
                shapes += [(self.num_blocks, s.kv_heads, self.block_size, n) for n in (s.dim, 1 if s.keys_as_values else s.value_dim)]
        sizes = [int(np.prod(s)) for s in shapes]
        out = np.zeros(max(1, sum(sizes)), np.float32)
        check(_ffi.lib().orion_cuda_model_read_kv(self._h, out.ctypes.data_as(C.POINTER(C.c_float)), out.size))
        ends = np.cumsum(sizes)
        return [out[e - n:e].reshape(s) for e, n, s in zip(ends, sizes, shapes)]
