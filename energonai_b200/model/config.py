"""config.json of a layer-listed decoder -> LatentDecoderConfig, SandwichDecoderConfig, HybridDecoderConfig or
ParallelDecoderConfig.

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


# ---- decoders of state-space layers and of attention beside gated linear attention -----------------------
#
#     {"architecture": ..., "vocab": V, "width": W, "norm": {"eps": e}, "residual_mult": m, "logit_scale": s,
#      "embedding": {"bigram": {"buckets", "mul_prev", "mul_cur"}?},
#      "layers": [{"type": "mamba2", "mixer": {"heads", "vdim", "state", "groups", "conv", "norm_groups"}, "mlp": ...},
#                 {"type": "parallel", "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}?,
#                                                         "rot": {"dims", "base", "scaling": {"factor"}?}?},
#                                                "right": {"heads", "dim", "vdim", "tau"}},
#                  "mlp": {"kind": "dense", "ff"} |
#                         {"kind": "moe", "router": {"experts", "top", "identity"?, "groups": {"count", "keep"}?},
#                          "expert": {"ff"}, "shared": {"ff"}?} | null}, ...]}

@dataclass
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                # taps of the convolution, the current token's included
    norm_groups: int


@dataclass
class ChunkAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    chunk: int = 0           # 0: none
    rot_dims: int = 0        # 0: no rotation
    rot_base: float = 1.0
    rot_factor: float = 1.0  # every frequency is divided by it

    @property
    def vdim(self):
        return self.dim      # the values are the keys


@dataclass
class GatedLinearConfig:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: Optional[int] = None      # of the decay's projection; the checkpoint's shapes give it (with_shapes)


@dataclass
class ParallelConfig:
    left: ChunkAttentionConfig
    right: GatedLinearConfig


@dataclass
class RoutedConfig:
    experts: int
    top: int
    ff: int
    identity: int = 0        # further choices, which return the input itself
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0       # 0: no shared expert


@dataclass
class HybridLayerConfig:
    mixer: Union[StateSpaceConfig, ParallelConfig]
    mlp: Optional[Union[DenseConfig, RoutedConfig]] = None


@dataclass
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int


def _need(ok, where, what):
    if not ok:
        raise ValueError(f"{where}: {what}")


def _sizes(where, d, *names):
    out = [int(d[n]) for n in names]
    _need(all(v > 0 for v in out), where, f"{', '.join(names)} must be positive (got {out})")
    return out


@dataclass
class HybridDecoderConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    logit_scale: float
    layers: List[HybridLayerConfig]
    bigram: Optional[BigramConfig] = None

    @staticmethod
    def _mixer(where, kind, m):
        if kind == "mamba2":
            _known(where, m, ("heads", "vdim", "state", "groups", "conv", "norm_groups"))
            c = StateSpaceConfig(*_sizes(where, m, "heads", "vdim", "state", "groups", "conv", "norm_groups"))
            _need(c.heads % c.groups == 0, where, f"{c.heads} heads do not share {c.groups} groups")
            _need(c.heads * c.vdim % c.norm_groups == 0, where, f"{c.heads * c.vdim} columns have no {c.norm_groups} equal parts")
            return c
        if kind != "parallel":
            raise ValueError(f"{where}: unknown type {kind!r}")
        _known(where, m, ("left", "right"))
        a, r = m["left"], m["right"]
        _known(where, a, ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"))
        heads, kv_heads, dim, vdim = _sizes(where, a, "heads", "kv_heads", "dim", "vdim")
        _need(heads % kv_heads == 0, where, f"{heads} heads do not share {kv_heads} key / value heads")
        _need(vdim == dim, where, f"the values are the keys: vdim {vdim} is not dim {dim}")
        left = ChunkAttentionConfig(heads, kv_heads, dim, float(a["scale"]))
        if a.get("mask"):
            _known(where, a["mask"], ("size",))
            left.chunk, = _sizes(where, a["mask"], "size")
        if a.get("rot"):
            rot = a["rot"]
            _known(where, rot, ("dims", "base", "scaling"))
            left.rot_dims, left.rot_base = int(rot["dims"]), float(rot["base"])
            _need(0 <= left.rot_dims <= dim and left.rot_dims % 2 == 0 and left.rot_base > 0, where, f"{left.rot_dims} rotated dimensions of {dim}")
            if rot.get("scaling"):
                _known(where, rot["scaling"], ("factor",))
                left.rot_factor = float(rot["scaling"]["factor"])
                _need(left.rot_factor > 0, where, f"a rotation slowed down by {left.rot_factor}")
        _known(where, r, ("heads", "dim", "vdim", "tau", "rank"))
        right = GatedLinearConfig(*_sizes(where, r, "heads", "dim", "vdim"), tau=float(r["tau"]), rank=int(r["rank"]) if r.get("rank") else None)
        _need(right.tau > 0, where, f"tau {right.tau}")
        return ParallelConfig(left, right)

    @staticmethod
    def _mlp(where, f):
        if f is None:
            return None
        if f["kind"] == "dense":
            _known(where, f, ("kind", "ff"))
            return DenseConfig(*_sizes(where, f, "ff"))
        if f["kind"] != "moe":
            raise ValueError(f"{where}: unknown feed-forward kind {f['kind']!r}")
        _known(where, f, ("kind", "router", "expert", "shared"))
        r = f["router"]
        _known(where, r, ("experts", "top", "identity", "groups"))
        _known(where, f["expert"], ("ff",))
        c = RoutedConfig(*_sizes(where, r, "experts", "top"), *_sizes(where, f["expert"], "ff"), identity=int(r.get("identity") or 0))
        if r.get("groups"):
            _known(where, r["groups"], ("count", "keep"))
            c.groups, c.keep = _sizes(where, r["groups"], "count", "keep")
        if f.get("shared"):
            _known(where, f["shared"], ("ff",))
            c.shared_ff, = _sizes(where, f["shared"], "ff")
        choices = c.experts + c.identity
        _need(c.identity >= 0 and choices % c.groups == 0 and c.keep <= c.groups, where, f"{choices} choices in {c.groups} groups of which {c.keep} are kept")
        _need(c.top <= choices // c.groups * c.keep, where, f"top {c.top} of {choices // c.groups * c.keep} open choices")
        return c

    @classmethod
    def from_dict(cls, d):
        layers = []
        for i, ly in enumerate(d["layers"]):
            where = f"layer {i}"
            _known(where, ly, ("type", "mixer", "mlp"))
            layers.append(HybridLayerConfig(cls._mixer(where, ly["type"], ly["mixer"]), cls._mlp(where, ly.get("mlp"))))
        _known("model", d, ("architecture", "vocab", "width", "norm", "residual_mult", "logit_scale", "embedding", "layers"))
        _known("norm", d["norm"], ("eps",))
        emb = d.get("embedding") or {}
        _known("embedding", emb, ("bigram",))
        bigram = None
        if emb.get("bigram"):
            _known("bigram", emb["bigram"], ("buckets", "mul_prev", "mul_cur"))
            b = emb["bigram"]
            bigram = BigramConfig(*_sizes("bigram", b, "buckets"), int(b["mul_prev"]), int(b["mul_cur"]))
            _need(0 <= bigram.mul_prev < 1 << 31 and 0 <= bigram.mul_cur < 1 << 31, "bigram", "its factors are not negative")
        return cls(*_sizes("model", d, "vocab", "width"), eps=float(d["norm"]["eps"]), residual_mult=float(d["residual_mult"]),
                   logit_scale=float(d["logit_scale"]), layers=layers, bigram=bigram)

    def with_shapes(self, shapes):
        """Takes the sizes that only a checkpoint gives, {tensor name: shape}: the rank of each decay projection."""
        for i, lc in enumerate(self.layers):
            if isinstance(lc.mixer, ParallelConfig) and f"l{i}.mix.right.a1" in shapes:
                rank = int(shapes[f"l{i}.mix.right.a1"][0])
                _need(lc.mixer.right.rank in (None, rank), f"layer {i}", f"the decay's projection has rank {rank}, the configuration asks for {lc.mixer.right.rank}")
                lc.mixer.right.rank = rank
        return self


# ---- decoders whose mixer and feed-forward read the stream side by side ----------------------------------
#
#     {"architecture": ..., "vocab": V, "width": W, "norm": {"eps": e}, "canon": {"taps": t},
#      "layers": [{"type": "latent_attention",
#                  "mixer": {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "kv_from"?,
#                            "rot": {"dims", "base", "scaling": {"factor", "original", "fast", "slow"}?}}, "mlp": ...},
#                 {"type": "mamba1", "mixer": {"inner", "state", "dt_rank", "conv"}, "mlp": ...},
#                 {"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap"?,
#                                                 "mask": {"size", "keep_first"?}?}, "mlp": {"kind": "dense", "ff"} | null}, ...]}

@dataclass
class RotaryLatentConfig:
    heads: int
    dim: int                 # of a query or key head, without the rotated part
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_scaling: Optional[tuple] = None      # (factor, original, fast, slow)
    kv_from: Optional[int] = None


@dataclass
class SelectiveScanConfig:
    inner: int
    state: int
    dt_rank: int
    conv: int                # taps of the convolution, the current token's included


@dataclass
class CappedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float = 0.0     # 0: none
    window: int = 0          # 0: none
    keep_first: int = 0      # positions that stay visible behind the window


@dataclass
class ParallelLayerConfig:
    mixer: Union[RotaryLatentConfig, SelectiveScanConfig, CappedAttentionConfig]
    mlp: Optional[DenseConfig] = None


@dataclass
class ParallelDecoderConfig:
    vocab: int
    width: int
    eps: float
    taps: int                # of the convolution in front of every sublayer
    layers: List[ParallelLayerConfig]

    @staticmethod
    def _mixer(where, kind, m):
        if kind == "mamba1":
            _known(where, m, ("inner", "state", "dt_rank", "conv"))
            c = SelectiveScanConfig(*_sizes(where, m, "inner", "state", "dt_rank", "conv"))
            _need(c.state <= 256, where, f"{c.state} states per channel (at most 256)")
            return c
        if kind == "attention":
            _known(where, m, ("heads", "kv_heads", "dim", "vdim", "scale", "softcap", "mask"))
            c = CappedAttentionConfig(*_sizes(where, m, "heads", "kv_heads", "dim", "vdim"), scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0))
            _need(c.heads % c.kv_heads == 0, where, f"{c.heads} heads do not share {c.kv_heads} key / value heads")
            _need(c.softcap >= 0, where, f"scores capped at {c.softcap}")
            if m.get("mask"):
                _known(where, m["mask"], ("size", "keep_first"))
                c.window, = _sizes(where, m["mask"], "size")
                c.keep_first = int(m["mask"].get("keep_first") or 0)
                _need(c.keep_first >= 0, where, f"a window that keeps {c.keep_first} positions")
            return c
        _need(kind == "latent_attention", where, f"unknown type {kind!r}")
        _known(where, m, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot", "kv_from"))
        rot, src = m["rot"], m.get("kv_from")
        _known(where, rot, ("dims", "base", "scaling"))
        c = RotaryLatentConfig(*_sizes(where, m, "heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"), scale=float(m["scale"]),
                               rot_base=float(rot["base"]), kv_from=None if src is None else int(src))
        _need(int(rot["dims"]) == c.rot_dim and c.rot_dim % 2 == 0 and c.rot_base > 0, where, f"{rot['dims']} of {c.rot_dim} dimensions rotated")
        if rot.get("scaling"):
            s = rot["scaling"]
            _known(where, s, ("factor", "original", "fast", "slow"))
            c.rot_scaling = tuple(float(s[k]) for k in ("factor", "original", "fast", "slow"))
            _need(all(v > 0 for v in c.rot_scaling) and c.rot_base != 1, where, f"rotation scaled by {c.rot_scaling}")
        return c

    @classmethod
    def from_dict(cls, d):
        _known("model", d, ("architecture", "vocab", "width", "norm", "canon", "layers"))
        _known("norm", d["norm"], ("eps",))
        _known("canon", d["canon"], ("taps",))
        layers = []
        for i, ly in enumerate(d["layers"]):
            where = f"layer {i}"
            _known(where, ly, ("type", "mixer", "mlp"))
            mlp, f = None, ly.get("mlp")
            if f is not None:
                _need(f.get("kind", "dense") == "dense", where, f"unknown feed-forward kind {f.get('kind')!r}")
                _known(where, f, ("kind", "ff"))
                mlp = DenseConfig(*_sizes(where, f, "ff"))
            c = cls._mixer(where, ly["type"], ly["mixer"])
            src = getattr(c, "kv_from", None)
            if src is not None:
                _need(0 <= src < i and isinstance(layers[src].mixer, RotaryLatentConfig), where, f"kv_from must name an earlier latent layer (got {src})")
                other = layers[src].mixer
                _need(other.kv_from is None, where, f"layer {src} has no latents of its own")
                same = lambda m: (m.kv_rank, m.rot_dim, m.rot_base, m.rot_scaling)
                _need(same(other) == same(c), where, f"its latents and rotation differ from those of layer {src}")
            layers.append(ParallelLayerConfig(c, mlp))
        taps, = _sizes("canon", d["canon"], "taps")
        _need(taps <= 16, "canon", f"a convolution of {taps} taps (at most 16)")
        return cls(*_sizes("model", d, "vocab", "width"), eps=float(d["norm"]["eps"]), taps=taps, layers=layers)
