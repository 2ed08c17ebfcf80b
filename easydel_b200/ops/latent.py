"""Latent attention over paged rows ``[latent | rotary key]`` for fp32-stream layers (``csrc/latent_ops.cu``,
``csrc/attention_mla_decode.cu``, ``csrc/attention_fwd.cu``).

A packed projection row holds a token's query heads (``D`` unrotated and ``R`` rotary elements each), its latent (``L``) and
its rotary key (``R``). :func:`prologue` rotates the queries in place and appends the cache row; :func:`attend` then runs one
of three forms of the same attention, all of them with a sliding window and a sink per head:

* single-token sequences: the absorbed form on the tensor cores. The key up-projection is folded into the query, the
  kernel reads the pages as they are, the value up-projection follows;
* portions of several tokens: the visible pages are gathered and one product expands them into keys and values per head
  (the weight has an identity block for the rotary key, so a cache row becomes a complete key row), then the paged
  flash-attention kernel runs over them;
* 32-bit models and sizes outside the tiles: the absorbed form on the general-purpose cores.
"""

from __future__ import annotations

import torch

from . import _lib, kernels as K, serving as S, stream
from .rotation import rotate

vp, i32, i64, f32 = _lib.vp, _lib.i32, _lib.i64, _lib.f32
_lib.register("edl_latent_prologue", i32, [vp, i32, i64, vp, vp, vp, vp, f32, i32, i32, i32, i32, i32, i32, i32, vp, i64, i64,
                                           vp, vp])
_lib.register("edl_latent_spans", i32, [vp, vp, vp, i32, i32, i32, i32, i32, i32, vp, vp, vp, vp])
_lib.register("edl_gather_pages", i32, [vp, vp, vp, i32, i64, vp])
_lib.register("edl_head_gate", i32, [vp, i32, i64, i64, vp, i64, vp, i64, i32, i32, i32, vp])


def split_packed(proj: torch.Tensor, H: int, D: int, R: int, L: int):
    """Views of the packed rows: queries ``[T, H, D + R]``, latent ``[T, L]``, rotary key ``[T, R]``, the rest."""
    n = H * (D + R)
    return proj[:, :n].unflatten(1, (H, D + R)), proj[:, n:n + L], proj[:, n + L:n + L + R], proj[:, n + L + R:]


def latent_norm(c: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    cf = c.float()
    return (cf * torch.rsqrt(cf.pow(2).mean(-1, keepdim=True) + eps) * w.float()).to(c.dtype)


def prologue(proj: torch.Tensor, heads: tuple[int, int, int, int], norm_w: torch.Tensor, eps: float, freq: torch.Tensor,
             positions: torch.Tensor, slot_mapping: torch.Tensor, pages: torch.Tensor, layout: str = "neighbours") -> None:
    """Rotates the queries inside ``proj [T, ld]`` and writes the cache rows to ``pages [P, page, 1, L + R]``.
    ``heads = (H, D, R, L)``; ``layout``: see :mod:`.rotation`."""
    H, D, R, L = heads
    T = proj.shape[0]
    if stream.on_kernels(proj):
        pos = positions.reshape(-1).to(torch.int32)
        _lib.call("edl_latent_prologue", proj.data_ptr(), stream._f32flag(proj.dtype), proj.stride(0), pos.data_ptr(),
                  slot_mapping.data_ptr(), norm_w.data_ptr(), freq.data_ptr(), float(eps), T, H, D, R, L, freq.numel() // 2,
                  int(layout == "halves"), pages.data_ptr(), pages.stride(1), pages.shape[0] * pages.shape[1],
                  _lib.status_word(proj.device).data_ptr(), _lib.stream_ptr())
        return
    q, c, kr, _ = split_packed(proj, H, D, R, L)
    q[..., D:] = rotate(q[..., D:], positions, freq, layout)
    row = torch.cat([latent_norm(c, norm_w, eps), rotate(kr, positions, freq, layout)], -1)
    S.kv_append(row[:, None], row[:, None], pages, pages, slot_mapping)


def head_gate(o: torch.Tensor, gate: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """``out [T, H V] = o [T, H, V] * sigmoid(gate [T, H V])``; ``o`` may be strided."""
    T, H, V = o.shape
    if stream.on_kernels(o):
        assert o.stride(2) == 1 and gate.stride(1) == 1 and out.stride(1) == 1
        _lib.call("edl_head_gate", o.data_ptr(), stream._f32flag(o.dtype), o.stride(0), o.stride(1), gate.data_ptr(),
                  gate.stride(0), out.data_ptr(), out.stride(0), T, H, V, _lib.stream_ptr())
        return out
    return out.copy_((o.reshape(T, H * V).float() * torch.sigmoid(gate.float())).to(o.dtype))


def decode_splits(batch: int, heads: int, window: int | None, max_keys: int, sms: int) -> int:
    """Key splits of a decode step: enough (sequence, 16-head group, split) units to fill the SMs, each with some tiles
    of 32 keys. Depends on sizes only, so that a captured step keeps its value."""
    units = batch * ((heads + 15) // 16)
    tiles = (min(window or max_keys, max_keys) + 31) // 32
    return int(max(1, min(8, sms // max(1, units), tiles // 4)))


def expansion_weight(up: torch.Tensor, H: int, D: int, R: int, V: int, L: int) -> torch.Tensor:
    """``[H (D + R) + H V, L + R]``: turns cache rows into per-head keys (unrotated part from the latent, the shared
    rotary part copied by an identity block) and values. ``up [H D + H V, L]`` stacks both up-projections."""
    w = up.new_zeros(H * (D + R) + H * V, L + R)
    keys = w[:H * (D + R)].view(H, D + R, L + R)
    keys[:, :D, :L] = up[:H * D].view(H, D, L)
    keys[:, D:, L:] = torch.eye(R, dtype=up.dtype, device=up.device)
    w[H * (D + R):, :L] = up[H * D:]
    return w


def tiles_support(attn) -> bool:
    """Sizes the bf16 tensor-core forms take."""
    H, D, R, L, V = attn.heads, attn.dim, attn.rot_dim, attn.kv_rank, attn.vdim
    return (all(n % 8 == 0 for n in (D, R, L, V)) and D + R <= S.MAX_QK_DIM and V <= 128 and L <= 512 and L + R <= 576)


def attend(attn, proj: torch.Tensor, pages: torch.Tensor, meta, table: torch.Tensor, group: int = 0) -> torch.Tensor:
    """Attention of the step's rows over pages that hold them already -> gated heads ``[T, H V]``. ``attn``: the layer
    (:class:`..layers.mla.LatentStreamAttention`); ``meta``: :class:`..caching.paged.PagedBatchMeta`."""
    H, D, R, L, V = attn.heads, attn.dim, attn.rot_dim, attn.kv_rank, attn.vdim
    T = proj.shape[0]
    q, _, _, gate = split_packed(proj, H, D, R, L)
    up = attn.ukv_proj.weight
    uk, uv = up[:H * D].view(H, D, L), up[H * D:].view(H, V, L)
    out = torch.empty(T, H * V, dtype=proj.dtype, device=proj.device)
    window = attn.sliding_window or 0

    def finish(o, rows):
        """o [T', H, V] of the rows ``rows``."""
        if attn.output_gate:
            head_gate(o, gate[rows], out[rows])
        else:
            out[rows] = o.reshape(o.shape[0], H * V)

    if not proj.is_cuda:
        finish(_attend_reference(attn, q, pages, meta, table, uk, uv), slice(0, T))
        return out
    if proj.dtype != torch.bfloat16 or not attn.tiles:
        q_abs = torch.cat([stream.bmm(q[..., :D].transpose(0, 1), uk).transpose(0, 1), q[..., D:]], -1).contiguous()
        o = S.simt_attention(q_abs, pages, pages, meta.cu_q, meta.kv_lens, table, scale=attn.scale, window=window,
                             sinks=attn.sinks, v_dim=L)
        finish(stream.bmm(o.transpose(0, 1), uv.transpose(1, 2)).transpose(0, 1), slice(0, T))
        return out
    B = meta.num_seqs
    single = B if meta.max_q == 1 and T == B else meta.leading_singles()
    if single:
        rows = slice(0, single)
        q_lat = torch.bmm(q[rows, :, :D].transpose(0, 1), uk)                                    # [H, n, L]
        n = decode_splits(single, H, window, table.shape[1] * S.PAGE_SIZE, K.sm_count(proj.device))
        o = S.latent_decode(q_lat.transpose(0, 1), q[rows, :, D:], pages, meta.kv_lens, table, scale=attn.scale,
                            window=window, sinks=attn.sinks, num_splits=n)                       # [n, H, L]
        finish(torch.bmm(o.transpose(0, 1), uv.transpose(1, 2)).transpose(0, 1), rows)
    if single < B:
        rows = slice(single, T)
        compact, src, n_pages = visible_pages(meta, table, window, single, group, pages)
        ctx = torch.empty(n_pages * S.PAGE_SIZE, L + R, dtype=pages.dtype, device=pages.device)
        _lib.call("edl_gather_pages", pages.data_ptr(), src.data_ptr(), ctx.data_ptr(), n_pages,
                  S.PAGE_SIZE * (L + R) * pages.element_size(), _lib.stream_ptr())
        kv = K.gemm(ctx, attn.expansion())                                                       # [rows, H (D + R) + H V]
        o = torch.empty(T, H, V, dtype=proj.dtype, device=proj.device)
        k_width = H * (D + R)
        _lib.call("edl_attn_paged", proj.data_ptr(), kv.data_ptr(), kv.data_ptr() + 2 * k_width, o.data_ptr(),
                  proj.stride(0), kv.stride(0), kv.stride(0), H * V, meta.cu_q.data_ptr() + 4 * single,
                  meta.kv_lens.data_ptr() + 4 * single, compact.data_ptr(), compact.stride(0), B - single,
                  int(meta.max_q), T, n_pages, H, H, D + R, V, float(attn.scale), 1, window, 0, 0.0, _lib.ptr(attn.sinks),
                  _lib.status_word(proj.device).data_ptr(), _lib.stream_ptr())
        finish(o[rows], rows)
    return out


def visible_pages(meta, table, window: int, first_seq: int, group: int, pages):
    """Compact page table and page list of what the sequences from ``first_seq`` on can see in this step; the layers of
    a step with the same window share it."""
    key = (group, window, first_seq)
    hit = meta.visible.get(key)
    if hit is None:
        page, n = S.PAGE_SIZE, 0
        for new, keys in meta.spans[first_seq:]:
            first = max(0, keys - new - window + 1) // page if window else 0
            n += (keys + page - 1) // page - first if new else 0
        B, dev = meta.num_seqs - first_seq, table.device
        n = max(1, n)
        compact = torch.empty(B, table.shape[1], dtype=torch.int32, device=dev)
        src = torch.zeros(n, dtype=torch.int32, device=dev)
        _lib.call("edl_latent_spans", meta.cu_q.data_ptr() + 4 * first_seq, meta.kv_lens.data_ptr() + 4 * first_seq,
                  table.data_ptr() + 4 * first_seq * table.stride(0), table.stride(0), B, window, page, n, pages.shape[0],
                  compact.data_ptr(), src.data_ptr(), _lib.status_word(dev).data_ptr(), _lib.stream_ptr())
        hit = meta.visible[key] = (compact, src, n)
    return hit


def _attend_reference(attn, q, pages, meta, table, uk, uv):
    """Tensor form over the gathered pages of every sequence, keys and values expanded per head."""
    from . import reference as R

    D, L = attn.dim, attn.kv_rank
    page, cu, outs = pages.shape[1], meta.cu_q.tolist(), []
    for b, n in enumerate(meta.kv_lens.tolist()):
        qs = q[cu[b]:cu[b + 1]]
        if not qs.shape[0]:
            continue
        kv = pages[table[b, :(n + page - 1) // page].long(), :, 0].reshape(-1, pages.shape[-1])[:n].to(q.dtype)
        outs.append(expanded_attention(attn, qs[None], kv[None, :, :L], kv[None, :, L:], uk, uv)[0])
    return torch.cat(outs)


def expanded_attention(attn, q, c, kr, uk, uv, segment_ids=None):
    """q ``[B, Tq, H, D + R]``, latents ``c [B, Tk, L]``, rotary keys ``kr [B, Tk, R]`` -> ``[B, Tq, H, V]``."""
    from . import reference as R

    k = torch.einsum("btl,hdl->bthd", c, uk)
    k = torch.cat([k, kr[:, :, None].expand(*k.shape[:3], kr.shape[-1])], -1)
    v = torch.einsum("btl,hvl->bthv", c, uv)
    return R.attention(q, k, v, causal=True, scale=attn.scale, segment_ids=segment_ids, sinks=attn.sinks,
                       sliding_window=attn.sliding_window)
