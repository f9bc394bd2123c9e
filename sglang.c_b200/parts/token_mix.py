"""Parts that mix what a sublayer reads with the tokens before it."""
from ..cache.needs import CacheNeed
from ..csrc import ops
from .base import Part
from .plan import WeightDecl
from .registry import register_part


@register_part("token_mix", "token_shift")
class TokenShift(Part):
    """h_t <- h_t + (h_(t-1) - h_t) * mu, element by element, on the normed rows a mixer reads; h_(t-1)
    is the row of the token before as it was before this change (zeros ahead of the first token).
    The last row of every request is kept, 32-bit, per request.  The norm ahead of the mixer, the
    shift and the norm ahead of a parallel feed-forward are one launch.  params: size."""

    @classmethod
    def declare_weights(cls, params):
        return {"mix": WeightDecl((params["size"],), "fraction")}

    def load(self, tensors, store):
        self.mix = store.vector(tensors["mix"])

    def cache_need(self):
        return CacheNeed.state((self.params["size"],), "float32", private=True)

    def forward(self, ctx, x, norm1, h1, norm2, h2, cache):
        ops.norm_pair_shift(x, norm1.weight, norm2.weight if norm2 is not None else None,
                            float(norm1.params["eps"]), h1, h2, shift=self.mix, prev=cache.tensor,
                            token_req=ctx.token_req, q_start=ctx.q_start, state_slots=ctx.state_slots)
