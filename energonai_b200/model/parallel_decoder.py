"""The decoder whose layers add mixer and feed-forward side by side,

    x += mixer(conv1(norm1(x))) + mlp(conv2(norm2(x))),

conv(h) = h + a causal convolution of h over a few tokens, per channel: latent attention, selective state space or capped
attention as mixer, dense feed-forwards.  Everything between two layers is one launch (stream_conv: residual sum,
both norms and both convolutions), and both sublayers end in one product: their inner columns lie side by side in
one row, and so do the columns of their output weights."""
import torch
from torch import nn

from ..gemm import project
from ..nn import init_weight
from ..norm import CONV_TAPS, stream_add, stream_conv
from .capped_attention import CappedAttention
from .config import CappedAttentionConfig, RotaryLatentConfig, SelectiveScanConfig
from .latent_attention import RotaryLatentAttention
from .layered_decoder import LayeredDecoder
from .mlp import GEGLUFeedForward
from .selective_scan import SelectiveScan
from .sequence_state import RingCache

MIXERS = {CappedAttentionConfig: CappedAttention, RotaryLatentConfig: RotaryLatentAttention, SelectiveScanConfig: SelectiveScan}


class ParallelBlock(nn.Module):
    def __init__(self, mixer, mlp, width, taps, dtype, device=None):
        super().__init__()
        table = lambda: nn.Parameter(torch.zeros(taps, width, dtype=torch.float32, device=device), requires_grad=False)
        self.mixer, self.mlp = mixer, mlp
        self.taps1, self.taps2 = table(), table() if mlp is not None else None             # norm weight times tap; the last row is the current token's
        for t in (self.taps1, self.taps2):
            if t is not None:
                t[-1].fill_(1.0)
        self.out_proj = init_weight(width, mixer.columns + (mlp.ff_padded if mlp is not None else 0), dtype=dtype, device=device)    # mixer | mlp
        self.bias = init_weight(width, std=0.0, dtype=dtype, device=device) if mixer.output_bias else None

    def forward(self, h1, h2, ctx):
        """What the layer adds to the stream."""
        n = self.mixer.columns
        inner = torch.empty((h1.shape[0], self.out_proj.shape[1]), dtype=h1.dtype, device=h1.device)
        self.mixer(h1, ctx, inner[:, :n])
        if self.mlp is not None:
            self.mlp.inner(h2, inner[:, n:])
        return project(inner, self.out_proj, bias=self.bias)


class ParallelDecoder(LayeredDecoder):
    def build_layers(self, config, **kw):
        W = self.hidden_size
        self.taps = min(n for n in CONV_TAPS if n >= config.taps)                          # (shorter tables are padded in front)
        for i, lc in enumerate(config.layers):
            mixer = MIXERS[type(lc.mixer)](i, W, lc.mixer, config.eps, **kw)
            mlp = GEGLUFeedForward(W, lc.mlp.ff, down=False, **kw) if lc.mlp is not None else None
            self.layers.append(ParallelBlock(mixer, mlp, W, self.taps, **kw))
        for blk in self.layers:
            src = getattr(blk.mixer, "kv_from", None)
            if src is not None and self.layers[src].mixer.rank != blk.mixer.rank:
                raise ValueError(f"layer {blk.mixer.layer} reads the rows of layer {src}, which have another width")

    def caches(self):
        out = {}
        for i, blk in enumerate(self.layers):
            out.update(blk.mixer.caches())
            out[i, "rows"] = RingCache(self.hidden_size, window=self.taps)                 # the normed rows both convolutions read
        return out

    def run(self, rows, ctx, on_layer=None):
        eps, count = self.config.eps, self.width
        x = y = None
        for i, blk in enumerate(self.layers):
            x, h1, h2 = stream_conv(x, blk.taps1, ctx.state.caches[i, "rows"].buf, eps, ctx.batch, count, src=rows if i == 0 else None, y=y,
                                    k2=blk.taps2, first=ctx.first, pos_device=ctx.pos)
            if on_layer is not None and i > 0:
                on_layer(i - 1, x)
            y = blk(h1, h2, ctx)
        # the final norm of a step (of a prompt only some rows go on to the head)
        h = stream_add(x, eps, count, y=y, w_next=None if ctx.is_prompt else self.norm.weight)
        if on_layer is not None:
            on_layer(len(self.layers) - 1, x)
        return x, h
