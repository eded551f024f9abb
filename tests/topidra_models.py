"""Small Topidra configurations and random weights for the tests."""
import numpy as np

from nn_b200.blocks import bf16_bits
from nn_b200.topidra import TopidraConfig


def attention(heads=6, kv_heads=2, dim=20, vdim=28, scale=0.3, size=13, ff=72):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def lightning(heads=3, dim=20, vdim=36, decay=None, ff=None):
    decay = list(np.linspace(0.5, 0.995, heads)) if decay is None else decay
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, vocab=103, width=60, eps=3e-5, loop=None):
    c = {"architecture": "Topidra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    # odd sizes, a loop in the middle, feed-forwards on either kind of layer and on none
    "mixed": config([lightning(ff=40), attention(), lightning(), attention(heads=4, kv_heads=4, dim=24, vdim=16, size=30, ff=None), lightning(heads=2, vdim=52)],
                    loop=(1, 3, 2)),
    # heads, windows, loops and feed-forwards of 1; decays of 0 and 1
    "ones": config([attention(heads=1, kv_heads=1, dim=8, vdim=16, size=1, ff=1), lightning(heads=2, dim=1, vdim=1, decay=[0.0, 1.0]),
                    attention(heads=2, kv_heads=1, dim=16, vdim=8, size=2, ff=16)], vocab=64, width=32, loop=(0, 3, 1)),
    # larger heads, windows across several tiles, the loop over everything; queries that count down
    "wide": config([attention(heads=8, kv_heads=1, dim=96, vdim=128, scale=0.08, size=70, ff=136), lightning(heads=2, dim=128, vdim=72, ff=64),
                    attention(heads=3, kv_heads=3, dim=128, vdim=64, scale=-0.1, size=200, ff=None)], vocab=200, width=96, loop=(0, 3, 2)),
    # no loop at all; heads beyond what the prompt kernels take
    "large_heads": config([lightning(heads=1, dim=144, vdim=200), attention(heads=4, kv_heads=2, dim=136, vdim=152, scale=0.05, size=40),
                           attention(heads=2, kv_heads=2, dim=264, vdim=24, scale=0.04, size=21)], vocab=90, width=64),
}


def weights_for(cfg: dict, seed: int) -> dict:
    """name -> bf16 bits; every matrix scaled so that activations stay of order one."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in TopidraConfig.from_dict(cfg).tensor_shapes().items():
        x = rng.standard_normal(shape)
        if "norm" in name:
            x = 1.0 + 0.2 * x
        elif name.endswith("sink"):
            x = 1.5 * x
        elif name == "embed":
            x = 0.5 * x
        else:
            x = 1.3 * x / np.sqrt(shape[-1])
        out[name] = bf16_bits(x.astype(np.float32))
    return out
