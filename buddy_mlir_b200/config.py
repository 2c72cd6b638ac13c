"""Model configurations: uniform attention models (ModelConfig) and models given as a list of
described layers (LayeredConfig).

ModelConfig: the shapes of the decode path (the configs buddy-mlir's specs bake into
its generated ModelSession: tools/buddy-codegen/gen_session.py:156-180,
models/deepseek_r1/specs/*.json)."""
import ctypes as C
from dataclasses import dataclass, replace
from typing import Optional, Tuple

from . import _lib
from ._lib import LayerConfigC, ModelConfigC


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
class LayerSpec:
    mixer: LatentMixer
    ff: Optional[GatedFF]

    def to_c(self):
        m, f = self.mixer, self.ff
        kind = _lib.FF_NONE if f is None else (_lib.FF_EXPERTS if f.experts else _lib.FF_GATED)
        return LayerConfigC(_lib.MIX_LATENT, m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.window,
                            -1 if m.kv_from is None else m.kv_from, m.scale, m.rot_base, kind,
                            f.ff if f else 0, f.experts if f else 0, f.top if f else 0,
                            f.limit if f else 0.0, f.gate_slope if f else 0.0, f.up_offset if f else 0.0)


@dataclass(frozen=True)
class LayeredConfig:
    """A model of described layers: parallel blocks x += mixer(h) + ff(h), h = RMSNorm(x), and the
    transposed embedding table as the output head."""
    name: str
    hidden: int
    vocab: int
    eps: float
    layers: Tuple[LayerSpec, ...]
    max_len: int = 4096              # positions of a single-sequence session's cache
    dtype: str = "bfloat16"          # or "float32"

    @property
    def n_layers(self):
        return len(self.layers)

    def create(self, lib, handle, tp_rank=0, tp_size=1):
        """b200_model_create_layered into `handle`."""
        c = ModelConfigC(hidden=self.hidden, n_layers=self.n_layers, vocab=self.vocab, max_len=self.max_len,
                         eps=self.eps, tp_rank=tp_rank, tp_size=tp_size)
        arr = (LayerConfigC * self.n_layers)(*[l.to_c() for l in self.layers])
        dtype = {"bfloat16": _lib.BF16, "float32": _lib.F32}[self.dtype]
        return lib.b200_model_create_layered(C.byref(c), arr, dtype, C.byref(handle))

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
