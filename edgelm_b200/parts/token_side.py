"""A feed-forward that reads the token as well as the stream: x += W_proj (gelu_tanh(W_gate h) * e), gelu_tanh(z) =
z/2 (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), where e is the layer's slice of the token's row of a second embedding table.

The table is one tensor [vocab, columns] for the whole model (`names["table"]`, a name without the layer's prefix), of which this
layer reads the columns `first_column` .. `first_column + dim` - 1; it keeps only those.  The two projections have no biases; the
look-up and the product with the activation are one kernel between them, the activation in float32."""
import torch

from ..config.base import ConfigError
from ..csrc import ops
from . import linear
from .base import Part, as_matrix, nbytes
from .registry import register_ffn


@register_ffn("token_side")
class TokenSide(Part):
    graph_safe = True

    def __init__(self, spec, env):
        self.hidden, self.dim, self.vocab = spec["hidden_size"], spec["dim"], spec["vocab_size"]
        self.columns, self.first = spec["columns"], spec["first_column"]
        self.names = dict(spec["names"])
        self.dtype = env.dtype
        if self.dim < 1 or not 0 <= self.first <= self.columns - self.dim:
            raise ConfigError(f"token_side: columns {self.first} to {self.first + self.dim} of {self.columns}")
        self.table = self.w_gate = self.w_proj = None

    def sizes(self):
        return {"token_side": self.dim}

    def describe(self):
        return f"{self.kind}(dim {self.dim})"        # (which columns are the layer's own does not make it another kind of layer)

    def flops(self, n_tokens, attended):
        return 4.0 * n_tokens * self.hidden * self.dim

    def weight_shapes(self, prefix):
        n = self.names
        return {n["table"]: (self.vocab, self.columns), prefix + n["gate"]: (self.dim, self.hidden), prefix + n["proj"]: (self.hidden, self.dim)}

    def load(self, tensors, prefix, device):
        n = self.names
        self.table = as_matrix(tensors[n["table"]][:, self.first:self.first + self.dim], self.dtype, device)
        self.w_gate, self.w_proj = (as_matrix(tensors[prefix + n[k]], self.dtype, device) for k in ("gate", "proj"))

    def workspace_bytes(self, n_tokens, n_seqs):
        return nbytes((n_tokens, self.dim), torch.float32) + nbytes((n_tokens, self.dim), self.dtype) + nbytes((n_tokens, self.hidden), self.dtype)

    def first_weights(self):
        return (self.w_gate, self.w_proj)

    def forward(self, ctx, h, x, accumulate=True):
        h = linear.as_tensor(h)
        T, ws = h.shape[0], ctx.ws
        u = ws.alloc((T, self.dim), torch.float32)
        g = ws.alloc((T, self.dim), self.dtype)
        with ctx.prof("side_gate"):
            linear.matmul(ctx, h, self.w_gate, u, prefetch=(self.w_proj,))
            ops.token_gate(u, ctx.token_ids, self.table, g, ctx.err)
        with ctx.prof("side_proj"):
            linear.matmul(ctx, g, self.w_proj, x, epilogue=linear.EPI_RESIDUAL if accumulate else linear.EPI_STORE,
                          residual=x if accumulate else None, prefetch=ctx.weights_after)
