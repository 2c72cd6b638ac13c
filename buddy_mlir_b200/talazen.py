"""The Talazen architecture: config.json -> LayeredConfig.

Constants the architecture fixes (the gate's slope and the offset of the up branch) are here;
everything else comes from the configuration.
"""
from .config import GatedFF, LatentMixer, LayeredConfig, LayerSpec

GATE_SLOPE = 1.702
UP_OFFSET = 1.0


def _mixer(c):
    rot = c["rot"]
    if rot["dims"] != c["rot_dim"]:
        raise ValueError(f"rotary dims {rot['dims']} do not cover the rotated part of {c['rot_dim']}")
    mask = c.get("mask")
    return LatentMixer(heads=c["heads"], dim=c["dim"], rot_dim=c["rot_dim"], vdim=c["vdim"],
                       kv_rank=c["kv_rank"], scale=c["scale"], rot_base=rot["base"],
                       window=mask["size"] if mask else 0, kv_from=c.get("kv_from"))


def _feed_forward(c):
    if c is None:
        return None
    if c["kind"] == "dense":
        return GatedFF(c["ff"], c["limit"], GATE_SLOPE, UP_OFFSET)
    if c["kind"] == "moe":
        e, r = c["expert"], c["router"]
        return GatedFF(e["ff"], e["limit"], GATE_SLOPE, UP_OFFSET, r["experts"], r["top"])
    raise ValueError(f"unknown feed-forward kind {c['kind']!r}")


def parse(c, dtype="bfloat16", max_len=4096):
    layers = []
    for entry in c["layers"]:
        if entry["type"] != "latent_attention":
            raise ValueError(f"unknown mixer {entry['type']!r}")
        layers.append(LayerSpec(_mixer(entry["mixer"]), _feed_forward(entry["mlp"])))
    return LayeredConfig("talazen", c["width"], c["vocab"], c["norm"]["eps"], tuple(layers),
                         max_len=max_len, dtype=dtype)
