"""Latent attention caches one row [latent | rotated key part] per position, shared by all heads.  A step attends over it in one of two
forms, whose choice is here for every model that has such layers:

  * ABSORBED: W_uk^T q against the cached rows themselves (one key head that is also the value), then W_uv per head;
  * EXPANDED: one tensor-core product turns the rows of the sequence into keys | values per head, then ordinary multi-head attention.
"""
from .. import abi

EXPAND_MIN_TOKENS = 128    # steps from this size on expand a latent layer's keys and values per head (bfloat16 sessions)


def expands(T: int, rank: int, rot_dim: int, dim: int, vdim: int, wdt: int, force_float32: bool = False) -> bool:
    """Whether a step of T tokens runs expanded.  Expanding costs 2 R (rank + rot_dim) H (dim + rot_dim + vdim) FLOPs on the tensor cores per step over
    R cached rows; the absorbed form costs (2 rank - dim - vdim) more multiply-adds per (query, key, head) in f32.  Worth it for long steps of
    bfloat16 sessions whose rows fit the tensor-core product (a multiple of 8 values, at least 64); float32 sessions, whose
    products are exact f32 tiles either way, and short steps stay absorbed."""
    row = rank + rot_dim
    return (wdt == abi.W_BF16 or force_float32) and T >= EXPAND_MIN_TOKENS and row % 8 == 0 and row >= 64 and 2 * rank > dim + vdim
