"""Latent attention: the keys and values of all heads come from ONE cached row per token, a normed latent ``c`` [R] and a rotated
key part [r] (``csrc/latent.cu``, ``csrc/latent_sm100.cu``).

Head h scores token j with ``(q_n . W_uk[h] c_j + q_r . k_r_j) * scale`` and takes its value ``W_uv[h] c_j``.  Two forms:

* absorbed (``latent_absorb`` -> ``latent_decode`` / ``latent_attention`` -> ``latent_out``): ``W_uk[h]^T q_n`` meets the cached rows
  themselves, the softmax mixes latents, ``W_uv[h]`` and the output gate follow.  Decoding, fp32, and sizes beyond the prompt kernel.
* expanded (``latent_rotate`` -> two GEMMs -> ``latent_prefill``): keys and transposed values of the visible tokens are
  materialised.  Prompts.

``z`` [T, columns] is the projection of the step's tokens: H heads of [d unrotated | r rotated] query columns, then (layers with
rows of their own) [R latent | r key part].  All sizes are padded to multiples of eight.  CPU tensors run the restatements here.
"""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from .. import _native
from .attention import tied_attention_simple

_FLAGS = {}         # one error flag per device, set by a tcgen05 launch whose waits gave up


def _rotate(x: torch.Tensor, cs: torch.Tensor) -> torch.Tensor:
    c, s = cs[..., 0::2], cs[..., 1::2]
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2)


def _store_rows(z, H, d, r, norm_w, R_real, eps, cs, dests):
    R = norm_w.numel()
    row = z[:, H * (d + r):H * (d + r) + R + r].float()
    c = row[:, :R]
    c = c / torch.sqrt(c.pow(2).sum(-1, keepdim=True) / R_real + eps) * norm_w
    row = torch.cat([c, _rotate(row[:, R:], cs)], dim=1).to(z.dtype)
    for store, rows in dests:
        ok = rows >= 0
        store.view(-1, R + r)[rows[ok]] = row[ok]


def latent_rotate(z: torch.Tensor, heads: int, d: int, r: int, norm_w: Optional[torch.Tensor], R: int, R_real: int, eps: float,
                  cos_sin: torch.Tensor, pos: torch.Tensor, home: Optional[Tuple[torch.Tensor, torch.Tensor]] = None,
                  ctx: Optional[Tuple[torch.Tensor, torch.Tensor]] = None) -> None:
    """In place: the queries' rotated parts turn to positions ``pos`` (int64 [T]).  With ``norm_w`` (fp32 [R]) the latent is normed
    (mean over ``R_real``), the key part rotated, and the row goes to rows ``home[1]`` of ``home[0]`` and ``ctx[1]`` of ``ctx[0]``."""
    if _native.use_native(z, cos_sin):
        _native.load(True).latent_rotate(z, int(heads), int(d), int(r), norm_w, int(R), int(R_real), float(eps), cos_sin, pos,
                                         *(home or (None, None)), *(ctx or (None, None)))
        return
    cs = cos_sin[pos]
    if norm_w is not None:
        _store_rows(z, heads, d, r, norm_w, R_real, eps, cs, [x for x in (home, ctx) if x is not None])
    q = z[:, :heads * (d + r)].view(z.shape[0], heads, d + r)
    q[..., d:] = _rotate(q[..., d:].float(), cs[:, None, :]).to(z.dtype)


def latent_absorb(z: torch.Tensor, uk_t: torch.Tensor, r: int, norm_w: Optional[torch.Tensor], R_real: int, eps: float,
                  cos_sin: torch.Tensor, pos: torch.Tensor, home: Optional[Tuple[torch.Tensor, torch.Tensor]] = None) -> torch.Tensor:
    """[T, H, R + r] = [W_uk^T q_unrotated | rotated part] of every head (``uk_t`` [H, R, d]); cache rows as in
    :func:`latent_rotate`.  One launch."""
    H, R, d = uk_t.shape
    if _native.use_native(z, uk_t):
        return _native.load(True).latent_absorb(z, uk_t, int(r), norm_w, int(R_real), float(eps), cos_sin, pos, *(home or (None, None)))
    cs = cos_sin[pos]
    if norm_w is not None:
        _store_rows(z, H, d, r, norm_w, R_real, eps, cs, [home])
    q = z[:, :H * (d + r)].reshape(z.shape[0], H, d + r).float()
    return torch.cat([torch.einsum("hrd,thd->thr", uk_t.float(), q[..., :d]), _rotate(q[..., d:], cs[:, None, :])], dim=-1).to(z.dtype)


def latent_out(o: torch.Tensor, ml: Optional[torch.Tensor], uv: torch.Tensor, gate: torch.Tensor) -> torch.Tensor:
    """[T, H dv] = sigmoid(gate) * W_uv[h] o[t, h] (``uv`` [H, dv, R]).  ``o`` fp32 [T, H, R], or split partials [T, H, splits, R]
    with ``ml`` [T, H, splits, 2] (reference maximum in the log2 domain, sum) that are merged first."""
    if _native.use_native(o, uv):
        return _native.load(True).latent_out(o, ml, uv, gate)
    if ml is not None:
        w = torch.exp2(ml[..., 0] - ml[..., 0].amax(-1, keepdim=True))
        o = torch.where(ml[..., 1:] > 0, o, torch.zeros_like(o))
        o = (o * w.unsqueeze(-1)).sum(2) / (w * ml[..., 1]).sum(-1).unsqueeze(-1)
    y = torch.einsum("hvr,thr->thv", uv.float(), o.to(uv.dtype).float()).flatten(1)
    return (y * torch.sigmoid(gate[:, :y.shape[1]].float())).to(uv.dtype)


def latent_attention(q_eff: torch.Tensor, cache: torch.Tensor, row0: torch.Tensor, n_keys: torch.Tensor, rank: int,
                     scale: float) -> torch.Tensor:
    """fp32 [T, H, R]: absorbed attention in fp32 arithmetic, token t over rows ``row0[t] .. + n_keys[t]`` of ``cache`` (rows of
    R + r, up to 1024): fp32 models, sizes beyond the tensor-core kernels, and the check of those."""
    return tied_attention_simple(q_eff, cache.view(-1, 1, cache.shape[-1]), None, row0, n_keys, None, None, scale, rank, True)


def latent_prefill_supported(d: int, r: int, dv: int, scale: float = 1.0) -> bool:
    """Sizes of the tcgen05 prompt kernel."""
    return d <= 128 and r <= 64 and dv <= 128 and scale > 0


def latent_decode_supported(R: int, r: int, scale: float = 1.0) -> bool:
    """Sizes of the tcgen05 decode kernel."""
    return R <= 512 and r <= 64 and scale > 0


def _error_flag(device) -> torch.Tensor:
    key = str(device)
    if key not in _FLAGS:
        _FLAGS[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return _FLAGS[key]


def check_latent_errors() -> None:
    """Raise if a bounded wait inside a tcgen05 latent-attention kernel gave up since the last check (synchronises)."""
    for flag in _FLAGS.values():
        if int(flag.item()) != 0:
            flag.zero_()
            raise RuntimeError("latent attention: a wait inside the kernel timed out")


def latent_prefill(z: torch.Tensor, k: torch.Tensor, ctx: torch.Tensor, vt: torch.Tensor, cu: torch.Tensor, q_pos0: torch.Tensor,
                   kv_lens: torch.Tensor, ctx0: torch.Tensor, max_q: int, heads: int, d: int, r: int, dv: int, scale: float,
                   gate: torch.Tensor) -> torch.Tensor:
    """Causal prompt attention in the expanded form with the output gate, [T, H dv] (GPU, bf16, tcgen05): queries in ``z``
    (rotated), keys ``k`` [L, H d] and the rotated part in the packed rows ``ctx`` [L, R + r], values ``vt`` [H dv, L].  Sequence b's
    queries are rows ``cu[b] .. cu[b + 1]`` from position ``q_pos0[b]`` on, its ``kv_lens[b]`` visible tokens start at packed row
    ``ctx0[b]`` (a multiple of 64, like L)."""
    return _native.load(True).latent_prefill(z, k, ctx, vt, cu, q_pos0, kv_lens, ctx0, int(max_q), int(heads), int(d), int(r),
                                             ctx.shape[1] - int(r), int(dv), float(scale), gate, _error_flag(z.device))


DECODE_TILE, DECODE_HEADS = 64, 32     # tokens per tile and heads per CTA of the decode kernel


def pick_latent_splits(batch: int, heads: int, rows: int, num_sms: int = 148) -> int:
    """KV splits of :func:`latent_decode`, one CTA per SM: as many as one wave holds, at most one per tile of tokens."""
    tiles = max(1, (rows + DECODE_TILE - 1) // DECODE_TILE)
    ctas = batch * ((heads + DECODE_HEADS - 1) // DECODE_HEADS)
    return int(max(1, min(num_sms // max(1, ctas), tiles, 64)))


def latent_decode(q_eff: torch.Tensor, cache: torch.Tensor, slots: torch.Tensor, kv_lens: torch.Tensor, rank: int, scale: float,
                  splits: int = 0) -> Tuple[torch.Tensor, torch.Tensor]:
    """Absorbed attention of one token per sequence over ``cache`` [slots, max_len, R + r] (GPU, bf16, tcgen05): split partials
    and their (maximum, sum) for :func:`latent_out`."""
    splits = splits or pick_latent_splits(q_eff.shape[0], q_eff.shape[1], cache.shape[1])
    return tuple(_native.load(True).latent_decode(q_eff, cache, slots, kv_lens, int(rank), float(scale), int(splits),
                                                  _error_flag(q_eff.device)))
