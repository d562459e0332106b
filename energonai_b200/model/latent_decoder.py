"""The latent-attention / mixture-of-experts decoder: layers whose sublayers read the residual stream
itself and whose OUTPUT is normalised before it is added (x += norm(sublayer(x))).

Beside the fp32 stream travels its rounding to the operand dtype, which is what the products read."""
import torch
from torch import nn

from ..nn import RMSNorm1D
from ..norm import rms_residual
from .latent_attention import LatentAttention
from .layered_decoder import LayeredDecoder
from .moe import MixtureOfExperts
from .sequence_state import RingCache


class OutputNormBlock(nn.Module):
    """x += norm1(mixer(x)); x += norm2(mlp(x)) (mlp may be None)."""

    def __init__(self, mixer, mlp, width, padded, eps, dtype, device=None):
        super().__init__()
        norm = lambda: RMSNorm1D(padded, eps=eps, count=width, offset=1.0, dtype=dtype, device=device)
        self.mixer, self.norm1 = mixer, norm()
        self.mlp, self.norm2 = mlp, norm() if mlp is not None else None

    @staticmethod
    def _add(y, norm, x, xt, **kw):
        # in fp32 the stream is its own operand copy
        return rms_residual(y, norm.weight, norm.eps, x, xt=None if xt is x else xt, offset=norm.offset, count=norm.count, **kw)

    def _mlp(self, x, xt, first, rows_per_batch, routed):
        y, mix = self.mlp(xt, first=first, rows_per_batch=rows_per_batch, routed=routed)
        self._add(y, self.norm2, x, xt, mix=mix)

    def prompt(self, x, xt, ctx):
        self._add(self.mixer.prompt(xt, ctx), self.norm1, x, xt)
        if self.mlp is not None:
            self._mlp(x, xt, ctx.first, ctx.seq, None)

    def step(self, x, xt, ctx):
        router = self.mlp.router_for_step(ctx.batch) if self.mlp is not None else None
        routed = self._add(self.mixer.step(xt, ctx), self.norm1, x, xt, router=router)
        if self.mlp is not None:
            self._mlp(x, xt, None, 1, routed)


class LatentDecoder(LayeredDecoder):
    norm_offset = 1.0

    def build_layers(self, config, **kw):
        W, Wp = self.width, self.hidden_size
        for i, lc in enumerate(config.layers):
            m = lc.mixer
            mixer = LatentAttention(i, Wp, m.heads, m.dim, m.vdim, m.kv_rank, m.window, m.scale, config.eps, kv_from=m.kv_from, **kw)
            mlp = None
            if lc.mlp is not None:
                mlp = MixtureOfExperts(Wp, lc.mlp.experts, lc.mlp.top, lc.mlp.ff, lc.mlp.limit, lc.mlp.alpha, **kw)
            self.layers.append(OutputNormBlock(mixer, mlp, W, Wp, config.eps, **kw))
        for blk in self.layers:
            src = blk.mixer.kv_from
            if src is not None and self.layers[src].mixer.rank != blk.mixer.rank:
                raise ValueError(f"layer {blk.mixer.layer} reads the latents of layer {src}, which have another width")

    def caches(self):
        """One ring per layer that has latents of its own, as long as the longest window among its
        readers."""
        windows = {}
        for blk in self.layers:
            windows.setdefault(blk.mixer.source, []).append(blk.mixer.window)
        return {i: RingCache(self.layers[i].mixer.rank, 0 if min(w) <= 0 else max(w)) for i, w in windows.items()}

    def run(self, rows, ctx, on_layer=None):
        # fp32 residual stream and operand copy (in fp32 one and the same)
        x, xt = (rows.clone(),) * 2 if self.dtype == torch.float32 else (rows.float(), rows)
        for i, blk in enumerate(self.layers):
            (blk.prompt if ctx.is_prompt else blk.step)(x, xt, ctx)
            if on_layer is not None:
                on_layer(i, x)
        return x, None
