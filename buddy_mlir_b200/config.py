"""Model configurations: uniform attention models (ModelConfig) and models given as a list of
described layers (LayeredConfig).

ModelConfig: the shapes of the decode path (the configs buddy-mlir's specs bake into
its generated ModelSession: tools/buddy-codegen/gen_session.py:156-180,
models/deepseek_r1/specs/*.json)."""
import ctypes as C
import math
from dataclasses import dataclass, replace
from typing import Optional, Tuple, Union

from . import _lib
from ._lib import LayerConfigC, ModelConfigC, StackConfigC


@dataclass(frozen=True)
class ModelConfig:
    name: str
    hidden: int
    n_layers: int
    q_heads: int
    kv_heads: int
    head_dim: int
    ffn: int
    vocab: int
    max_len: int
    eps: float = 1e-6
    rope_theta: float = 1e4
    qkv_bias: bool = True   # Qwen2
    qk_norm: bool = False   # Qwen3

    def to_c(self, tp_rank=0, tp_size=1):
        return ModelConfigC(self.hidden, self.n_layers, self.q_heads, self.kv_heads,
                            self.head_dim, self.ffn, self.vocab, self.max_len,
                            self.eps, self.rope_theta, int(self.qkv_bias),
                            int(self.qk_norm), tp_rank, tp_size)

    def create(self, lib, handle, tp_rank=0, tp_size=1):
        """b200_model_create into `handle`."""
        return lib.b200_model_create(C.byref(self.to_c(tp_rank, tp_size)), C.byref(handle))

    def with_(self, **kw):
        return replace(self, **kw)

    @property
    def q_dim(self):
        return self.q_heads * self.head_dim

    @property
    def kv_dim(self):
        return self.kv_heads * self.head_dim


@dataclass(frozen=True)
class LatentMixer:
    """Attention over a cached low-rank latent: per token one row of kv_rank + rot_dim values that
    all heads share; dim unrotated and rot_dim rotated query / key dimensions per head."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    window: int = 0                  # 0: every position before
    kv_from: Optional[int] = None    # attend to an earlier layer's cache


@dataclass(frozen=True)
class HeadsMixer:
    """Attention over keys and values cached per key/value head, with rotary positions on the first
    rot_dim dimensions of a head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_dim: int
    rot_base: float
    scale: float
    rot_halves: bool = False         # pairs (i, i + rot_dim/2); else (2i, 2i + 1)
    bias: bool = False               # on the query, key and value projections
    qk_norm: bool = False            # RMSNorm over the whole query and the whole key projection
    sink: float = -math.inf          # score of one more softmax entry that has no value
    out_gate: bool = False           # heads times sigmoid(W_g h)
    window: int = 0                  # 0: every position before


@dataclass(frozen=True)
class MemoryMixer:
    """Matrix memory: a gated recurrent [dim][vdim] state per head, with soft-capped exponential
    gates, a normaliser and a running maximum."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float
    q_scale: float
    floor: float                     # added to the normaliser


@dataclass(frozen=True)
class SideBySide:
    """Two mixers on the same input; the sum of their outputs, each times its factor."""
    left: HeadsMixer
    right: MemoryMixer
    left_scale: float = 1.0
    right_scale: float = 1.0


@dataclass(frozen=True)
class GatedFF:
    """down(g * sigmoid(gate_slope * g) * (u + up_offset)), g <= limit, |u| <= limit.  With
    experts > 0 a router picks `top` of that many such units per token, weighted by the softmax
    over the picked logits."""
    ff: int
    limit: float
    gate_slope: float
    up_offset: float
    experts: int = 0
    top: int = 0


@dataclass(frozen=True)
class PlainFF:
    """down(act(up h)), act one of _lib.ACT_*."""
    ff: int
    act: int


def _heads_fields(m, scale=1.0):
    return dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, rot_dim=m.rot_dim, rot_base=m.rot_base,
                scale=m.scale, rot_halves=int(m.rot_halves), qkv_bias=int(m.bias), qk_norm=int(m.qk_norm),
                out_gate=int(m.out_gate), sink=m.sink, window=m.window, mix_scale=scale)


def _memory_fields(m, scale=1.0):
    return dict(mem_heads=m.heads, mem_dim=m.dim, mem_vdim=m.vdim, mem_cap=m.gate_cap, mem_q_scale=m.q_scale,
                mem_floor=m.floor, mem_mix_scale=scale)


@dataclass(frozen=True)
class LayerSpec:
    """A mixer and a feed-forward.  Latent mixers run as a parallel block, x += mixer(h) + ff(h) with
    h = RMSNorm(x); the others as a sandwich, x += norm1b(mixer(norm1(x))), x += norm2b(ff(norm2(x)))."""
    mixer: Union[LatentMixer, HeadsMixer, MemoryMixer, SideBySide]
    ff: Union[GatedFF, PlainFF, None]

    def to_c(self):
        m, f = self.mixer, self.ff
        c = dict(kv_from=-1, mix_scale=1.0, mem_mix_scale=1.0, sink=-math.inf)
        if isinstance(m, LatentMixer):
            c.update(mixer=_lib.MIX_LATENT, block=_lib.BLOCK_PARALLEL, heads=m.heads, dim=m.dim, rot_dim=m.rot_dim,
                     vdim=m.vdim, kv_rank=m.kv_rank, window=m.window, kv_from=-1 if m.kv_from is None else m.kv_from,
                     scale=m.scale, rot_base=m.rot_base)
        else:
            c.update(block=_lib.BLOCK_SANDWICH)
            if isinstance(m, HeadsMixer):
                c.update(_heads_fields(m), mixer=_lib.MIX_HEADS)
            elif isinstance(m, MemoryMixer):
                c.update(_memory_fields(m), mixer=_lib.MIX_MEMORY)
            else:
                c.update(_heads_fields(m.left, m.left_scale), **_memory_fields(m.right, m.right_scale),
                         mixer=_lib.MIX_HEADS_MEMORY)
        if f is None:
            c.update(ff_kind=_lib.FF_NONE)
        elif isinstance(f, PlainFF):
            c.update(ff_kind=_lib.FF_PLAIN, ff=f.ff, ff_act=f.act)
        else:
            c.update(ff_kind=_lib.FF_EXPERTS if f.experts else _lib.FF_GATED, ff=f.ff, experts=f.experts, top=f.top,
                     limit=f.limit, gate_slope=f.gate_slope, up_offset=f.up_offset)
        return LayerConfigC(**c)


@dataclass(frozen=True)
class LayeredConfig:
    """A model of described layers, with the transposed embedding table as the output head."""
    name: str
    hidden: int
    vocab: int
    eps: float
    layers: Tuple[LayerSpec, ...]
    max_len: int = 4096              # positions of a single-sequence session's cache
    dtype: str = "bfloat16"          # or "float32"
    embed_scale: float = 1.0         # factor on the embedding rows (not on the head)
    loop: Tuple[int, int, int] = (0, 0, 1)   # layers start .. stop-1 run `times` times, with a cache per pass;
                                     # the embedding output is added before every pass but the first
    side_dim: int = 0                # per-token layer input of that size (sandwich layers), 0: none

    @property
    def n_layers(self):
        return len(self.layers)

    def create(self, lib, handle, tp_rank=0, tp_size=1):
        """b200_model_create_layered into `handle`."""
        c = ModelConfigC(hidden=self.hidden, n_layers=self.n_layers, vocab=self.vocab, max_len=self.max_len,
                         eps=self.eps, tp_rank=tp_rank, tp_size=tp_size)
        stack = StackConfigC(self.embed_scale, *self.loop, self.side_dim)
        arr = (LayerConfigC * self.n_layers)(*[l.to_c() for l in self.layers])
        dtype = {"bfloat16": _lib.BF16, "float32": _lib.F32}[self.dtype]
        return lib.b200_model_create_layered(C.byref(c), C.byref(stack), arr, dtype, C.byref(handle))

    def with_(self, **kw):
        return replace(self, **kw)


# DeepSeek-R1-Distill-Qwen-1.5B (Qwen2 architecture), max_token_len 1024 as in
# models/deepseek_r1/specs/f32.json.
DEEPSEEK_R1_1P5B = ModelConfig("deepseek_r1_1p5b", 1536, 28, 12, 2, 128, 8960,
                               151936, 1024)
# Qwen3-8B architecture (QK-RMSNorm, no qkv bias), context 4096.
QWEN3_8B = ModelConfig("qwen3_8b", 4096, 36, 32, 8, 128, 12288, 151936, 4096,
                       rope_theta=1e6, qkv_bias=False, qk_norm=True)
# Small shapes for tests (same structure, seconds on a CPU).
TINY_QWEN2 = ModelConfig("tiny_qwen2", 256, 2, 4, 2, 64, 512, 1024, 128)
TINY_QWEN3 = ModelConfig("tiny_qwen3", 256, 2, 8, 2, 128, 512, 1024, 128,
                         qkv_bias=False, qk_norm=True)
# Small shapes that still reach both row modes of the persistent decode kernel
# (K = 512 and 1536 warp-per-row; K = 2112 shared rows with a ragged last block).
TINY_MEGA = ModelConfig("tiny_mega", 512, 2, 12, 2, 128, 2112, 2048, 256)
