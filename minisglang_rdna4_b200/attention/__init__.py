"""Attention backends. ``--attention-backend`` is accepted for compatibility with the
reference's launch lines; every value maps to the one sm_100a paged backend."""
from .base import AttnMetadata, BaseAttnBackend
from .latent import LatentAttentionBackend
from .paged import PagedAttentionBackend


def create_attention_backend(name: str, num_q_heads: int, num_kv_heads: int, head_dim: int, device,
                             max_batch: int = 0, max_seq_len: int = 0, single_split: bool = False,
                             latent=None, heads=None, talk=None) -> BaseAttnBackend:
    """``latent``: the layers' sizes of a model with a latent pool; ``heads``: ``(query heads, row width)`` of every layer
    of a model whose attention layers have a geometry of their own; ``talk``: see ``PagedAttentionBackend``."""
    if latent:
        return LatentAttentionBackend(latent, device, max_seq_len, single_split)
    return PagedAttentionBackend(num_q_heads, num_kv_heads, head_dim, device, max_batch, max_seq_len,
                                 single_split, heads, talk)


__all__ = ["AttnMetadata", "BaseAttnBackend", "LatentAttentionBackend", "PagedAttentionBackend", "create_attention_backend"]
