"""config.json of a layer-listed decoder -> LatentDecoderConfig or SandwichDecoderConfig.

    {"architecture": ..., "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "vdim", "kv_rank", "mask": {"size"}, "scale", "kv_from"?},
                 "mlp": {"kind": "moe", "router": {"experts", "top"}, "expert": {"ff", "limit"}} | null}, ...]}

Every size and constant of a model is read from there; a key that is missing or a kind that no
module implements is an error at load time, not a silently different model."""
from dataclasses import dataclass
from typing import List, Optional, Union

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


# ---- decoders of matrix-memory and grouped-attention layers ------------------------------------------
#
#     {"architecture": ..., "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
#      "layers": [{"type": "mlstm", "mixer": {"heads", "dim", "vdim", "gate_cap"}, "mlp": ...},
#                 {"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "q_temp": {"coef", "every"}?, "v_mix"?},
#                  "mlp": {"kind": "dense", "ff"} | null}, ...]}

@dataclass
class MemoryMixerConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass
class GroupedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    temp_coef: float = 0.0
    temp_every: int = 0              # 0: no query temperature
    v_mix: bool = False
    v_from: Optional[int] = None     # the layer whose values are mixed in (None: none, or this is that layer)


@dataclass
class DenseConfig:
    ff: int


@dataclass
class SandwichLayerConfig:
    mixer: Union[MemoryMixerConfig, GroupedAttentionConfig]
    mlp: Optional[DenseConfig] = None


def _known(where, d, keys):
    """A key that no module here implements may only be there to say that its mechanism is off."""
    for k, v in d.items():
        if k not in keys and v:
            raise ValueError(f"{where}: {k!r} is not implemented")


@dataclass
class SandwichDecoderConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: List[SandwichLayerConfig]

    @classmethod
    def from_dict(cls, d):
        layers, v_first = [], None
        for i, ly in enumerate(d["layers"]):
            m, where = ly["mixer"], f"layer {i}"
            _known(where, ly, ("type", "mixer", "mlp"))
            if ly["type"] == "mlstm":
                _known(where, m, ("heads", "dim", "vdim", "gate_cap"))
                mixer = MemoryMixerConfig(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), gate_cap=float(m["gate_cap"]))
                if mixer.gate_cap <= 0:
                    raise ValueError(f"{where}: gate_cap {mixer.gate_cap}")
            elif ly["type"] == "attention":
                _known(where, m, ("heads", "kv_heads", "dim", "vdim", "scale", "q_temp", "v_mix"))
                t = m.get("q_temp")
                mixer = GroupedAttentionConfig(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                               scale=float(m["scale"]), temp_coef=float(t["coef"]) if t else 0.0,
                                               temp_every=int(t["every"]) if t else 0, v_mix=bool(m.get("v_mix", False)))
                if mixer.kv_heads < 1 or mixer.heads % mixer.kv_heads:
                    raise ValueError(f"{where}: {mixer.heads} heads do not share {mixer.kv_heads} key / value heads")
                if t and mixer.temp_every < 1:
                    raise ValueError(f"{where}: a query temperature every {mixer.temp_every} positions")
                if mixer.v_mix and v_first is None:
                    v_first = i
                elif mixer.v_mix:
                    mixer.v_from, other = v_first, layers[v_first].mixer
                    if (other.kv_heads, other.vdim) != (mixer.kv_heads, mixer.vdim):
                        raise ValueError(f"{where}: its values cannot be mixed with those of layer {v_first}, which have another size")
            else:
                raise ValueError(f"{where}: unknown type {ly['type']!r}")
            mlp, f = None, ly.get("mlp")
            if f is not None:
                if f.get("kind", "dense") != "dense":
                    raise ValueError(f"{where}: unknown feed-forward kind {f['kind']!r}")
                _known(where, f, ("kind", "ff"))
                mlp = DenseConfig(ff=int(f["ff"]))
            layers.append(SandwichLayerConfig(mixer, mlp))
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]), embed_scale=float(d["embedding"]["scale"]),
                   layers=layers)
