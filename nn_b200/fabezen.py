"""Fabezen: a decoder whose layers mix a gated delta rule (one decay per head, or one per head and key channel) with latent
attention over a sliding window, in any order, with a bigram embedding and a tied output.

The model is a list of blocks (nn_b200.blocks) over a 32-bit residual stream:
    x <- x + m * mixer(rms(x));  x <- x + m * ff(rms(x))
and the row kernel that adds a block's output also normalises for the next block.  Layers may share weights; what
a sequence carries is kept per layer.  The rest of the decoder is nn_b200.block_decoder.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .block_decoder import BlockDecoder
from .blocks import DeltaMixer, DenseGlu, LatentAttentionMixer, Source, Step, Workspace, f32, pad8, rms_rows

MIXERS = ("delta", "channel_delta", "latent_attention")


@dataclass
class LayerConfig:
    type: str
    mixer: dict
    mlp: dict | None
    weights_of: int | None = None


@dataclass
class FabezenConfig:
    vocab: int
    width: int
    layers: list = field(default_factory=list)
    eps: float = 1e-5
    residual_mult: float = 1.0
    embedding_scale: float = 1.0
    bigram: dict | None = None          # buckets, mul_prev, mul_cur

    @staticmethod
    def from_dict(j: dict) -> "FabezenConfig":
        layers = []
        for i, e in enumerate(j["layers"]):
            if e["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown type {e['type']!r}")
            if e.get("mlp") is not None and e["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {e['mlp'].get('kind')!r}")
            layers.append(LayerConfig(e["type"], dict(e["mixer"]), e.get("mlp"), e.get("weights_of")))
        for i, layer in enumerate(layers):
            if layer.weights_of is not None and not 0 <= layer.weights_of < len(layers):
                raise ValueError(f"layer {i}: weights_of {layer.weights_of}")
        emb = j.get("embedding") or {}
        return FabezenConfig(vocab=int(j["vocab"]), width=int(j["width"]), layers=layers, eps=float(j["norm"]["eps"]),
                             residual_mult=float(j.get("residual_mult", 1.0)), embedding_scale=float(emb.get("scale", 1.0)), bigram=emb.get("bigram"))

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ValueError("weights_of goes round in a circle")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    def tensor_shapes(self) -> dict:
        """name -> shape of every tensor of a weight file that the configuration fixes (low ranks are the file's own)."""
        D = self.width
        out = {"embed": (self.vocab, D), "final.norm": (D,)}
        if self.bigram is not None:
            out["bigram"] = (self.bigram["buckets"] + 1, D)
        for i, layer in enumerate(self.layers):
            if layer.weights_of is not None:
                continue
            p, m = f"l{i}.", layer.mixer
            out[p + "norm1"] = (D,)
            if layer.type == "latent_attention":
                H = m["heads"]
                t = {"dq": (m["q_rank"], D), "dq.norm": (m["q_rank"],), "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                     "dkv": (m["kv_rank"] + m["rot_dim"], D), "dkv.norm": (m["kv_rank"],), "uk": (H * m["dim"], m["kv_rank"]),
                     "uv": (H * m["vdim"], m["kv_rank"]), "o": (D, H * m["vdim"])}
            else:
                H, qk, v = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
                t = {"q": (qk, D), "k": (qk, D), "v": (v, D), "q.conv": (qk, m["conv"]), "k.conv": (qk, m["conv"]), "v.conv": (v, m["conv"]), "b": (H, D),
                     "A_log": (H,), "norm": (m["vdim"],), "o": (D, v)}
                if layer.type == "delta":
                    t.update({"a": (H, D), "dt_bias": (H,), "g": (v, D)})
                else:
                    t.update({"a1": (None, D), "a2": (H * m["dim"], None), "dt_bias": (H * m["dim"],), "g1": (None, D), "g2": (v, None)})
            out.update({p + "mix." + k: s for k, s in t.items()})
            if layer.mlp is not None:
                ff = layer.mlp["ff"]
                out.update({p + "norm2": (D,), p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
        return out


class _LayerWeights:
    """The blocks made from one layer's tensors."""

    def __init__(self, ws: Workspace, cfg: FabezenConfig, i: int, w):
        layer, p, m, dev = cfg.layers[i], f"l{i}.", cfg.layers[i].mixer, ws.dev
        t = lambda name: w[p + "mix." + name]
        self.norm1 = dev.from_numpy(f32(w[p + "norm1"]))
        if layer.type == "latent_attention":
            names = {"dq": "dq", "dq_norm": "dq.norm", "uq": "uq", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "o": "o"}
            self.mixer = LatentAttentionMixer(ws, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], float(m["scale"]),
                                              int(m["mask"]["size"]), m["rot"]["base"], int(m["rot"]["dims"]), cfg.eps,
                                              {k: t(n) for k, n in names.items()})
        else:
            names = {"q": "q", "k": "k", "v": "v", "b": "b", "o": "o", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "A_log": "A_log",
                     "dt_bias": "dt_bias", "norm": "norm"}
            names.update({n: n for n in (("a", "g") if layer.type == "delta" else ("a1", "a2", "g1", "g2"))})
            self.mixer = DeltaMixer(ws, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], cfg.eps, {k: t(n) for k, n in names.items()})
        self.norm2 = self.ff = None
        if layer.mlp is not None:
            self.norm2 = dev.from_numpy(f32(w[p + "norm2"]))
            self.ff = DenseGlu(ws, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"])

    def close(self) -> None:
        self.mixer.close()
        if self.ff is not None:
            self.ff.close()


class Fabezen(BlockDecoder):
    """weights in the shapes of FabezenConfig.tensor_shapes; the rest as BlockDecoder has it."""

    HEAD = "embed"           # also the embedding table

    def _build(self, weights) -> None:
        cfg, owned = self.cfg, {}
        self.layers = []
        for i in range(len(cfg.layers)):
            j = cfg.owner(i)
            if j not in owned:
                owned[j] = _LayerWeights(self.ws, cfg, j, weights)
                self._blocks.append(owned[j])
            self.layers.append((owned[j], owned[j].mixer.reserve(self.states, self.max_prefill)))
        self.bigram = self._table(weights["bigram"]) if cfg.bigram is not None else None

    def _layers(self, step: Step) -> None:
        """Embedding and every layer for the ids of the pass; leaves the residual stream in ``x``."""
        cfg, dev, ws = self.cfg, self.dev, self.ws
        D, x, h, m = cfg.width, ws["x"], ws["h"], cfg.residual_mult
        self._embed(step, self.head.w_ptr, self.head.k_ld, x, cfg.embedding_scale, self.bigram, cfg.bigram)
        source: Source | None = None
        for lw, cache in self.layers:
            rms_rows(step, dev, x, source, m, x if source else 0, lw.norm1, cfg.eps, D, h, self.dtype, pad8(D))
            source = lw.mixer.forward(h, cache, step)
            if lw.ff is not None:
                rms_rows(step, dev, x, source, m, x, lw.norm2, cfg.eps, D, h, self.dtype, pad8(D))
                source = lw.ff.forward(h, step)
        rms_rows(step, dev, x, source, m, x, None, cfg.eps, D, 0, self.dtype, 0)
