"""A feed-forward without a gate: x += W_down max(W_up h, 0)^2, no bias.  The square is the epilogue of the up product, the
residual sum that of the down product."""
from ..config.base import ConfigError
from . import linear
from .base import Part, as_matrix, nbytes
from .registry import register_ffn


@register_ffn("squared_relu")
class SquaredReLU(Part):
    graph_safe = True
    takes_normed_input = True

    def __init__(self, spec, env):
        self.hidden, self.inter = spec["hidden_size"], spec["intermediate_size"]
        self.names = dict(spec["names"])
        self.dtype = env.dtype
        if self.inter < 1:
            raise ConfigError(f"squared_relu: {self.inter} inner channels")
        self.w_up = self.w_down = None

    def sizes(self):
        return {"intermediate": self.inter}

    def flops(self, n_tokens, attended):
        return 4.0 * n_tokens * self.hidden * self.inter

    def weight_shapes(self, prefix):
        n = self.names
        return {prefix + n["up"]: (self.inter, self.hidden), prefix + n["down"]: (self.hidden, self.inter)}

    def load(self, tensors, prefix, device):
        n = self.names
        self.w_up = as_matrix(tensors[prefix + n["up"]], self.dtype, device)
        self.w_down = as_matrix(tensors[prefix + n["down"]], self.dtype, device)

    def workspace_bytes(self, n_tokens, n_seqs):
        return nbytes((n_tokens, self.inter), self.dtype) + nbytes((n_tokens, self.hidden), self.dtype)

    def first_weights(self):
        return (self.w_up,)

    def forward(self, ctx, h, x, accumulate=True):
        """x += feed_forward(h); with `accumulate` False, x = feed_forward(h) (float32)."""
        mid = ctx.ws.alloc((h.shape[0], self.inter), self.dtype)
        with ctx.prof("up_relu2"):
            linear.matmul(ctx, h, self.w_up, mid, epilogue=linear.EPI_RELU2, prefetch=(self.w_down,))
        with ctx.prof("down_proj_residual"):
            linear.matmul(ctx, mid, self.w_down, x, epilogue=linear.EPI_RESIDUAL if accumulate else linear.EPI_STORE,
                          residual=x if accumulate else None, prefetch=ctx.weights_after)
