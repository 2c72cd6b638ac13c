"""The Butolorn architecture: config.json -> LayeredConfig.

Two kinds of layers, in sandwich blocks: attention with biased projections, and a sink attention
side by side with a matrix memory.  What the architecture fixes (which branch each kind has, the
activation, the sink's score, the memory's query factor and floor) is here; every size and
constant comes from the configuration.
"""
from . import _lib
from .config import HeadsMixer, LayeredConfig, LayerSpec, MemoryMixer, PlainFF, SideBySide

SINK_SCORE = 0.0
MEMORY_FLOOR = 1e-6


def _heads(c, **branches):
    return HeadsMixer(heads=c["heads"], kv_heads=c["kv_heads"], dim=c["dim"], vdim=c["vdim"], rot_dim=c["rot"]["dims"],
                      rot_base=c["rot"]["base"], scale=c["scale"], **branches)


def _mixer(kind, c):
    if kind == "attention":
        return _heads(c, rot_halves=True, bias=True)
    if kind == "parallel":
        r = c["right"]
        return SideBySide(_heads(c["left"], qk_norm=True, sink=SINK_SCORE, out_gate=True),
                          MemoryMixer(heads=r["heads"], dim=r["dim"], vdim=r["vdim"], gate_cap=r["gate_cap"],
                                      q_scale=r["dim"] ** -0.5, floor=MEMORY_FLOOR),
                          c["left_scale"], c["right_scale"])
    raise ValueError(f"unknown mixer {kind!r}")


def _feed_forward(c):
    if c is None:
        return None
    if c["kind"] == "dense":
        return PlainFF(c["ff"], _lib.ACT_RELU2)
    raise ValueError(f"unknown feed-forward kind {c['kind']!r}")


def parse(c, dtype="bfloat16", max_len=4096):
    layers = tuple(LayerSpec(_mixer(e["type"], e["mixer"]), _feed_forward(e["mlp"])) for e in c["layers"])
    loop, side = c.get("loop"), c.get("token_side")
    return LayeredConfig("butolorn", c["width"], c["vocab"], c["norm"]["eps"], layers, max_len=max_len, dtype=dtype,
                         embed_scale=c["embedding"]["scale"],
                         loop=(loop["start"], loop["stop"], loop["times"]) if loop else (0, 0, 1),
                         side_dim=side["dim"] if side else 0)
