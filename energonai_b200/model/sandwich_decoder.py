"""The decoder of matrix-memory and grouped-attention layers: a norm in front of and behind every
sublayer, a gate on the sublayer's result, a scale per element:

    x += norm_out(mixer(h) * sigmoid(W h + b)) * scale,  h = norm_in(x)

and the same for the feed-forward.  Everything between two sublayers is one launch (stream_update): gate,
norm, scale and residual sum of the one, norm of the next.  The scale is multiplied into the output
norm's weight, in fp32."""
import torch
from torch import nn

from ..norm import stream_update
from .config import GroupedAttentionConfig
from .grouped_attention import GroupedAttention, padded_head
from .layered_decoder import LayeredDecoder
from .matrix_memory import MatrixMemory
from .mlp import XIELUFeedForward

class SandwichBlock(nn.Module):
    def __init__(self, mixer, mlp, padded, dtype, device=None):
        super().__init__()
        ones = lambda t: nn.Parameter(torch.ones(padded, dtype=t, device=device), requires_grad=False)
        self.mixer, self.norm1, self.out1 = mixer, ones(dtype), ones(torch.float32)
        self.mlp = mlp
        if mlp is not None:
            self.norm2, self.out2 = ones(dtype), ones(torch.float32)


class SandwichDecoder(LayeredDecoder):
    def build_layers(self, config, **kw):
        Wp, eps, dtype = self.hidden_size, config.eps, kw["dtype"]
        shared = [m for m in (lc.mixer for lc in config.layers) if isinstance(m, GroupedAttentionConfig) and m.v_mix]
        for i, lc in enumerate(config.layers):
            m = lc.mixer
            if isinstance(m, GroupedAttentionConfig):
                mixer = GroupedAttention(i, Wp, m, padded_head([d for s in (shared if m.v_mix else [m]) for d in (s.dim, s.vdim)], dtype), eps, **kw)
            else:
                mixer = MatrixMemory(i, Wp, m.heads, m.dim, m.vdim, m.gate_cap, eps, **kw)
            mlp = XIELUFeedForward(Wp, lc.mlp.ff, **kw) if lc.mlp is not None else None
            self.layers.append(SandwichBlock(mixer, mlp, Wp, **kw))

    def caches(self):
        return {i: blk.mixer.cache() for i, blk in enumerate(self.layers)}

    def run(self, rows, ctx, on_layer=None):
        eps, count = self.config.eps, self.width
        x = torch.empty(rows.shape, dtype=torch.float32, device=rows.device)
        # behind the last layer: the final norm of a step (of a prompt only some rows go on to the head)
        into = [blk.norm1 for blk in self.layers] + [None if ctx.is_prompt else self.norm.weight]
        h = stream_update(x, eps, count, src=rows, src_scale=self.config.embed_scale, w_next=into[0])
        for i, blk in enumerate(self.layers):
            y, gate = blk.mixer(h, ctx)
            w_out = blk.out1
            if blk.mlp is not None:
                h = stream_update(x, eps, count, y=y, gate=gate, w_out=w_out, w_next=blk.norm2)
                y, gate = blk.mlp(h)
                w_out = blk.out2
            h = stream_update(x, eps, count, y=y, gate=gate, w_out=w_out, w_next=into[i + 1])
            if on_layer is not None:
                on_layer(i, x)
        return x, h
