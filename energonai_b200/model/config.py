"""config.json of a layer-listed decoder -> LatentDecoderConfig.

    {"architecture": ..., "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "vdim", "kv_rank", "mask": {"size"}, "scale", "kv_from"?},
                 "mlp": {"kind": "moe", "router": {"experts", "top"}, "expert": {"ff", "limit"}} | null}, ...]}

Every size and constant of a model is read from there; a key that is missing or a kind that no
module implements is an error at load time, not a silently different model."""
from dataclasses import dataclass
from typing import List, Optional

GATE_ALPHA = 1.702          # slope of the sigmoid in the gated unit, fixed by the design


@dataclass
class LatentMixerConfig:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    window: int              # 0: no window
    scale: float
    kv_from: Optional[int] = None


@dataclass
class MoEConfig:
    experts: int
    top: int
    ff: int
    limit: float
    alpha: float = GATE_ALPHA


@dataclass
class LayerConfig:
    mixer: LatentMixerConfig
    mlp: Optional[MoEConfig] = None


@dataclass
class LatentDecoderConfig:
    vocab: int
    width: int
    eps: float
    layers: List[LayerConfig]

    def __post_init__(self):
        for i, lc in enumerate(self.layers):
            src = lc.mixer.kv_from
            if src is None:
                continue
            if not 0 <= src < i:
                raise ValueError(f"layer {i}: kv_from must name an earlier layer (got {src})")
            other = self.layers[src].mixer
            if other.kv_from is not None:
                raise ValueError(f"layer {i}: layer {src} has no latents of its own")
            if other.kv_rank != lc.mixer.kv_rank:
                raise ValueError(f"layer {i}: kv_rank {lc.mixer.kv_rank} differs from that of layer {src} ({other.kv_rank})")

    @classmethod
    def from_dict(cls, d):
        layers = []
        for i, ly in enumerate(d["layers"]):
            if ly["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown type {ly['type']!r}")
            m = ly["mixer"]
            mask = m.get("mask")
            window = int(mask["size"]) if mask is not None else 0
            if mask is not None and window < 1:
                raise ValueError(f"layer {i}: a window of {window} tokens")
            src = m.get("kv_from")
            mixer = LatentMixerConfig(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                                      window=window, scale=float(m["scale"]), kv_from=None if src is None else int(src))
            mlp, f = None, ly.get("mlp")
            if f is not None:
                if f.get("kind", "moe") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
                mlp = MoEConfig(experts=int(f["router"]["experts"]), top=int(f["router"]["top"]), ff=int(f["expert"]["ff"]),
                                limit=float(f["expert"]["limit"]))
            layers.append(LayerConfig(mixer, mlp))
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]), layers=layers)
