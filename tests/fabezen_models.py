"""Small Fabezen configurations and random weights for the tests."""
import numpy as np

from nn_b200.blocks import bf16_bits, f32
from nn_b200.fabezen import FabezenConfig


def delta(heads=3, kv_heads=1, dim=20, vdim=28, conv=3, ff=72, **extra):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}, **extra}


def channel(heads=4, kv_heads=2, dim=24, vdim=40, conv=2, ff=56, **extra):
    return {**delta(heads, kv_heads, dim, vdim, conv, ff, **extra), "type": "channel_delta"}


def latent(heads=3, dim=20, rot_dim=12, vdim=36, q_rank=28, kv_rank=44, size=11, base=5000.0, scale=0.17, ff=64, **extra):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "mask": {"size": size}, "rot": {"base": base, "dims": rot_dim}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}, **extra}


def config(layers, vocab=101, width=60, scale=3.0, eps=3e-5, mult=0.7, bigram=True):
    c = {"architecture": "Fabezen", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult,
         "embedding": {"scale": scale}}
    if bigram:
        c["embedding"]["bigram"] = {"buckets": 37, "mul_prev": 11, "mul_cur": 5}
    return c


CONFIGS = {
    # every mechanism, odd sizes, shared weights, a layer without feed-forward
    "mixed": config([delta(), channel(), latent(), delta(weights_of=0), channel(ff=None), latent(weights_of=2)]),
    # heads, key heads, taps and windows of 1; sizes that are powers of two
    "ones": config([channel(heads=1, kv_heads=1, dim=16, vdim=16, conv=1), latent(heads=1, dim=16, rot_dim=2, vdim=16, q_rank=8, kv_rank=16, size=1),
                    delta(heads=2, kv_heads=2, dim=8, vdim=64, conv=5)], vocab=64, width=32, mult=1.0, scale=1.0, bigram=False),
    # larger heads, windows across several tiles, all heads sharing one key head
    "wide": config([latent(heads=9, dim=48, rot_dim=16, vdim=80, q_rank=96, kv_rank=136, size=70), delta(heads=4, kv_heads=1, dim=96, vdim=128, conv=4),
                    channel(heads=2, kv_heads=2, dim=128, vdim=72, conv=3)], vocab=200, width=96),
}


def weights_for(cfg: dict, seed: int, low_rank: int = 12) -> dict:
    """name -> bf16 bits; every matrix scaled so that activations stay of order one, decays between fast and slow."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in FabezenConfig.from_dict(cfg).tensor_shapes().items():
        shape = tuple(low_rank if s is None else s for s in shape)
        x = rng.standard_normal(shape)
        if name.endswith("norm") or "norm" in name.rsplit(".", 1)[-1]:
            x = 1.0 + 0.2 * x
        elif name.endswith("A_log"):
            x = rng.uniform(-3.0, 1.0, shape)
        elif name.endswith("dt_bias"):
            x = rng.uniform(-3.0, 0.5, shape)
        elif name in ("embed", "bigram"):
            x = 0.5 * x
        elif name.endswith("conv"):
            x = x / np.sqrt(shape[-1])
        else:
            x = 1.3 * x / np.sqrt(shape[-1])
        out[name] = bf16_bits(x.astype(np.float32))
    return out


def wide64(w: dict) -> dict:
    """The same weights for the oracle."""
    return {k: f32(v).astype(np.float64) for k, v in w.items()}
