"""Python entry points of the serving kernels (paged attention, KV append, sampling)."""

from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from . import _lib

vp, i32, i64, f32 = _lib.vp, _lib.i32, _lib.i64, _lib.f32
_lib.register("edl_attn_paged_lse", i32, [vp, vp, vp, vp, vp, i64, i64, i64, i64, vp, vp, vp, i32, i32, i32, i64, i64,
                                          i32, i32, i32, i32, _lib.f32, i32, i32, _lib.f32, vp, vp, vp])
_lib.register("edl_attn_combine", i32, [vp, i64, vp, i32, i32, i32, i32, vp, vp, vp, vp])
_lib.register("edl_attn_paged", i32, [vp, vp, vp, vp, i64, i64, i64, i64, vp, vp, vp, i32, i32, i32, i64, i64, i32, i32,
                                      i32, i32, f32, i32, i32, i32, f32, vp, vp, vp])
_lib.register("edl_attn_paged_sigmoid", i32, [vp, vp, vp, vp, i64, i64, i64, i64, vp, vp, vp, i32, i32, i32, i64, i64, i32, i32,
                                              i32, i32, f32, i32, i32, vp, vp, i64, f32, vp, vp])
_lib.register("edl_paged_kv_append", i32, [vp, vp, vp, vp, vp, i32, i32, i64, i64, i64, i64, vp, vp])
_lib.register("edl_sample", i32, [vp, i32, i64, i32, i32, vp, vp, vp, vp, vp, vp, vp, vp, i64, vp, vp, vp, vp, vp])
_lib.register("edl_count_update", i32, [vp, i64, vp, vp, i32, i32, vp])
_lib.register("edl_gather_rows", i32, [vp, vp, vp, i32, i32, i64, vp])
_lib.register("edl_attn_decode", i32, [vp, vp, vp, vp, vp, i64, i64, i64, i64, vp, vp, i32, i32, i64, i32, i32, i32, i32,
                                       f32,
                                       i32, i32, i32, f32, vp, vp, vp])
_lib.register("edl_attn_decode_sigmoid", i32, [vp, vp, vp, vp, vp, i64, i64, i64, i64, vp, vp, i32, i32, i64, i32, i32, i32, i32,
                                               f32, i32, i32, i32, vp, vp, i64, f32, vp, vp])
_lib.register("edl_attn_mla_decode", i32, [vp, i64, i64, vp, i64, i64, vp, vp, vp, i64, vp, vp, i32, i32, i64, i32, i32, i32,
                                            f32, i32, vp, i32, vp, vp])

@dataclass
class SigmoidWeights:
    """Attention without a softmax: a visible key's weight is ``sigmoid(score + bias[h])``, not normalised over keys; head h's
    output is multiplied by ``out_scale`` and, with a ``gate [T, H]`` (rows may be strided), by ``sigmoid(gate[t, h])``."""

    bias: torch.Tensor                    # fp32 [H]
    gate: torch.Tensor | None = None
    out_scale: float = 1.0

    def args(self) -> tuple:
        g = self.gate
        assert self.bias.dtype == torch.float32 and (g is None or g.stride(1) == 1)
        return _lib.ptr(self.bias), _lib.ptr(g), g.stride(0) if g is not None else 0, float(self.out_scale)

    def finish(self, o: torch.Tensor) -> torch.Tensor:
        """Tensor form of the last step: ``o [T, H, Dv]`` scaled and gated."""
        f = self.out_scale if self.gate is None else torch.sigmoid(self.gate.float())[..., None] * self.out_scale
        return (o.float() * f).to(o.dtype)


PAGE_SIZE = 128
MAX_QK_DIM = 192      # widest query / key head of the tensor-core prefill kernel


def kv_append(k: torch.Tensor, v: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor,
              slot_mapping: torch.Tensor) -> None:
    """Writes new key/value rows ``[T, Hkv, D]`` into the page pools ``[P, page, Hkv, D]`` at flat slots."""
    T = k.shape[0]
    width = k.shape[-2] * k.shape[-1]
    if k.is_cuda:
        assert v.shape == k.shape, "keys and values of different widths are appended by stream.qkv_prologue"
        assert k.stride(-1) == 1 and k.stride(-2) == k.shape[-1] and v.stride(-2) == v.shape[-1]
        ld_page = k_pages.stride(1)
        _lib.call("edl_paged_kv_append", k.data_ptr(), v.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(),
                  slot_mapping.data_ptr(), T, width, k.stride(0), v.stride(0), ld_page,
                  k_pages.shape[0] * k_pages.shape[1], _lib.status_word(k.device).data_ptr(), _lib.stream_ptr())
        return
    flat_k = k_pages.view(-1, *k_pages.shape[2:])
    flat_v = v_pages.view(-1, *v_pages.shape[2:])
    ok = slot_mapping >= 0
    idx = slot_mapping[ok].long()
    flat_k[idx] = k[ok].to(flat_k.dtype)
    flat_v[idx] = v[ok].to(flat_v.dtype)


def paged_attention(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, cu_q: torch.Tensor,
                    kv_lens: torch.Tensor, page_table: torch.Tensor, max_q: int, *, scale: float | None = None,
                    causal: bool = True, window: int = 0, softcap: float = 0.0, sinks=None,
                    out: torch.Tensor | None = None, keep_first: int = 0,
                    sigmoid: SigmoidWeights | None = None) -> torch.Tensor:
    """Mixed prefill/decode attention over a paged KV cache.

    q ``[T, Hq, D]`` (new tokens of all sequences, concatenated), key pages ``[P, 128, Hkv, D]``, value pages
    ``[P, 128, Hkv, Dv]`` (``Dv`` may differ from ``D``), ``cu_q`` int32 ``[B+1]``, ``kv_lens`` int32 ``[B]`` (cached +
    new keys), ``page_table`` int32 ``[B, maxP]``. Layouts outside :func:`paged_kernel_supports` (32-bit floats,
    heads wider than 128) run the plain SIMT kernel. ``keep_first``: keys that stay visible when ``window`` has moved past
    them; ``sigmoid``: weights without a softmax; ``out [T, Hq, Dv]`` may have a row pitch of its own.
    """
    T, Hq, D = q.shape
    Hkv, Dv = k_pages.shape[2], v_pages.shape[-1]
    B = kv_lens.numel()
    scale = scale if scale is not None else 1.0 / math.sqrt(D)
    if q.is_cuda and not paged_kernel_supports(q, k_pages, v_pages):
        if not causal:
            raise NotImplementedError("the SIMT attention kernel is causal")
        return simt_attention(q, k_pages, v_pages, cu_q, kv_lens, page_table, scale=scale, window=window, sinks=sinks,
                              out=out, softcap=softcap, keep_first=keep_first, sigmoid=sigmoid)
    if q.is_cuda:
        assert k_pages.shape[1] == PAGE_SIZE, "the paged kernels use pages of 128 tokens"
        assert q.stride(-1) == 1 and q.stride(-2) == D
        if out is None:
            out = torch.empty((T, Hq, Dv), dtype=q.dtype, device=q.device)
        elif not _aligned_rows(out):
            return out.copy_(paged_attention(q, k_pages, v_pages, cu_q, kv_lens, page_table, max_q, scale=scale, causal=causal,
                                             window=window, softcap=softcap, sinks=sinks, keep_first=keep_first,
                                             sigmoid=sigmoid))
        if sigmoid is not None:
            assert causal and not softcap and sinks is None
            _lib.call("edl_attn_paged_sigmoid", q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), out.data_ptr(),
                      q.stride(0), k_pages.stride(1), v_pages.stride(1), out.stride(0), cu_q.data_ptr(),
                      kv_lens.data_ptr(), page_table.data_ptr(), page_table.stride(0), B, int(max_q), T, k_pages.shape[0],
                      Hq, Hkv, D, Dv, float(scale), int(window or 0), int(keep_first), *sigmoid.args(),
                      _lib.status_word(q.device).data_ptr(), _lib.stream_ptr())
            return out
        _lib.call("edl_attn_paged", q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), out.data_ptr(),
                  q.stride(0), k_pages.stride(1), v_pages.stride(1), out.stride(0), cu_q.data_ptr(),
                  kv_lens.data_ptr(), page_table.data_ptr(), page_table.stride(0), B, int(max_q), T, k_pages.shape[0],
                  Hq, Hkv, D, Dv, float(scale), int(causal), int(window or 0), int(keep_first), float(softcap or 0.0),
                  _lib.ptr(sinks),
                  _lib.status_word(q.device).data_ptr(), _lib.stream_ptr())
        return out
    o = paged_attention_reference(q, k_pages, v_pages, cu_q, kv_lens, page_table, scale=scale, causal=causal,
                                  window=window, softcap=softcap, sinks=sinks, keep_first=keep_first, sigmoid=sigmoid)
    return o if out is None else out.copy_(o)


_lib.register("edl_attn_simt", i32, [vp, vp, vp, vp, i32, i64, i64, i64, i64, vp, vp, vp, i32, i32, i32, i64, i32, i32, i32, i32,
                                     f32, i32, i32, f32, vp, vp, vp, i64, f32, vp, vp])


def simt_attention(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, cu_q: torch.Tensor,
                   kv_lens: torch.Tensor, page_table: torch.Tensor, *, scale: float, window: int = 0, sinks=None,
                   out: torch.Tensor | None = None, v_dim: int | None = None, softcap: float = 0.0, keep_first: int = 0,
                   sigmoid: SigmoidWeights | None = None) -> torch.Tensor:
    """Causal paged attention in fp32 arithmetic (``csrc/attention_simt.cu``): fp32 models, and head sizes outside the
    tensor-core kernels'. Arguments as :func:`paged_attention`; ``v_dim``: only the first elements of a value row count
    (latent rows, which are keys and values at once; one KV head)."""
    T, Hq, D = q.shape
    Hkv, Dv = k_pages.shape[2], v_dim or v_pages.shape[-1]
    assert v_dim is None or Hkv == 1
    if q.dtype != k_pages.dtype or q.dtype != v_pages.dtype or q.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"queries and pages must share one type (bf16 or fp32), got {q.dtype} / {k_pages.dtype}")
    assert k_pages.shape[1] == PAGE_SIZE and q.stride(-1) == 1 and q.stride(-2) == D
    if out is None:
        out = torch.empty((T, Hq, Dv), dtype=q.dtype, device=q.device)
    assert out.stride(2) == 1 and out.stride(1) == Dv
    assert sigmoid is None or (sinks is None and (sigmoid.gate is None or sigmoid.gate.dtype == q.dtype))
    _lib.call("edl_attn_simt", q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), out.data_ptr(),
              int(q.dtype == torch.float32), q.stride(0), k_pages.stride(1), v_pages.stride(1), out.stride(0), cu_q.data_ptr(),
              kv_lens.data_ptr(), page_table.data_ptr(), page_table.stride(0), kv_lens.numel(), T, k_pages.shape[0], Hq,
              Hkv, D, Dv, float(scale), int(window or 0), int(keep_first), float(softcap or 0.0), _lib.ptr(sinks),
              *(sigmoid.args() if sigmoid is not None else (None, None, 0, 1.0)), _lib.status_word(q.device).data_ptr(), _lib.stream_ptr())
    return out


def decode_attention(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, kv_lens: torch.Tensor,
                     page_table: torch.Tensor, *, scale: float | None = None, window: int = 0, sinks=None,
                     num_splits: int = 1, softcap: float = 0.0, keep_first: int = 0,
                     sigmoid: SigmoidWeights | None = None, out: torch.Tensor | None = None) -> torch.Tensor:
    """Decode-step attention (one query token per sequence) with the streaming kernel of
    ``csrc/attention_decode.cu``. q ``[B, Hq, D]``; pages ``[P, 128, Hkv, D]`` (values may have another width than
    keys); ``num_splits`` cuts every
    sequence's keys into that many parts that run as separate CTAs and are merged by :func:`attn_combine`; ``softcap``:
    scores become ``softcap * tanh(score / softcap)``; ``keep_first``, ``sigmoid``: as for :func:`paged_attention`.
    ``out [B, Hq, Dv]`` may have a row pitch of its own (without a softmax, or without key splits)."""
    B, Hq, D = q.shape
    Hkv, Dv = k_pages.shape[2], v_pages.shape[-1]
    scale = scale if scale is not None else 1.0 / math.sqrt(D)
    S_ = max(1, int(num_splits))
    if sigmoid is not None and (out is None or _aligned_rows(out)):
        assert not softcap and sinks is None
        if out is None:
            out = torch.empty((B, Hq, Dv), dtype=q.dtype, device=q.device)
        parts = torch.empty((S_, B, Hq, Dv), dtype=torch.float32, device=q.device) if S_ > 1 else None
        _lib.call("edl_attn_decode_sigmoid", q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), out.data_ptr(),
                  _lib.ptr(parts), q.stride(0), k_pages.stride(1), v_pages.stride(1), out.stride(0), kv_lens.data_ptr(),
                  page_table.data_ptr(), page_table.stride(0), B, k_pages.shape[0], Hq, Hkv, D, Dv, float(scale),
                  int(window or 0), int(keep_first), S_, *sigmoid.args(), _lib.status_word(q.device).data_ptr(),
                  _lib.stream_ptr())
        return out
    if out is not None:
        return out.copy_(decode_attention(q, k_pages, v_pages, kv_lens, page_table, scale=scale, window=window, sinks=sinks,
                                          num_splits=S_, softcap=softcap, keep_first=keep_first, sigmoid=sigmoid))
    out = torch.empty((S_, B, Hq, Dv), dtype=q.dtype, device=q.device)
    lse = torch.empty((S_, Hq, B), dtype=torch.float32, device=q.device) if S_ > 1 else None
    _lib.call("edl_attn_decode", q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), out.data_ptr(), _lib.ptr(lse),
              q.stride(0), k_pages.stride(1), v_pages.stride(1), Hq * Dv, kv_lens.data_ptr(), page_table.data_ptr(),
              page_table.stride(0), B, k_pages.shape[0], Hq, Hkv, D, Dv, float(scale), int(window or 0), int(keep_first), S_,
              float(softcap or 0.0), _lib.ptr(sinks) if S_ == 1 else None, _lib.status_word(q.device).data_ptr(), _lib.stream_ptr())
    if S_ == 1:
        return out[0]
    return attn_combine(out, lse, sinks=sinks)


def mla_decode_attention(q: torch.Tensor, pages: torch.Tensor, kv_lens: torch.Tensor, page_table: torch.Tensor, *,
                         scale: float, num_splits: int = 1) -> torch.Tensor:
    """Decode-step latent attention in the absorbed form (``csrc/attention_mla_decode.cu``).

    q ``[B, H, 576]`` = (query folded through the key up-projection (512) | rotated rotary query (64)); pages
    ``[P, 128, 1, 576]`` rows (compressed key/value | rotated rotary key). Returns ``[B, H, 512]``: the
    softmax-weighted sums of the rows' compressed part, to be sent through the value up-projection."""
    B, H, W = q.shape
    assert W == 576 and pages.shape[-1] == 576 and q.is_contiguous()
    return latent_decode(q[..., :512], q[..., 512:], pages, kv_lens, page_table, scale=scale, num_splits=num_splits)


def latent_decode(q_lat: torch.Tensor, q_rot: torch.Tensor, pages: torch.Tensor, kv_lens: torch.Tensor,
                  page_table: torch.Tensor, *, scale: float, window: int = 0, sinks=None,
                  num_splits: int = 1) -> torch.Tensor:
    """One absorbed query token per sequence over pages of latent rows: ``q_lat [B, H, L]`` (folded through the key
    up-projection), ``q_rot [B, H, R]`` (rotated), pages ``[P, 128, 1, L + R]``; the views may be strided. ``window``: a
    query sees its latest ``window`` keys; ``sinks [H]`` join the denominators. Returns ``[B, H, L]``."""
    B, H, L = q_lat.shape
    R = q_rot.shape[-1]
    assert pages.shape[-1] == L + R and pages.shape[1] == PAGE_SIZE and pages.is_contiguous()
    assert q_lat.stride(2) == 1 and q_rot.stride(2) == 1
    S_ = max(1, int(num_splits))
    out = torch.empty((S_, B, H, L), dtype=q_lat.dtype, device=q_lat.device)
    lse = torch.empty((S_, H, B), dtype=torch.float32, device=q_lat.device) if S_ > 1 else None
    _lib.call("edl_attn_mla_decode", q_lat.data_ptr(), q_lat.stride(0), q_lat.stride(1), q_rot.data_ptr(), q_rot.stride(0),
              q_rot.stride(1), pages.data_ptr(), out.data_ptr(), _lib.ptr(lse), H * L, kv_lens.data_ptr(),
              page_table.data_ptr(), page_table.stride(0), B, pages.shape[0], H, L, R, float(scale), int(window or 0),
              _lib.ptr(sinks) if S_ == 1 else None, S_, _lib.status_word(q_lat.device).data_ptr(), _lib.stream_ptr())
    return out[0] if S_ == 1 else attn_combine(out, lse, sinks=sinks)


def mla_decode_kernel_supports(q: torch.Tensor, pages: torch.Tensor) -> bool:
    return (q.is_cuda and q.dtype == torch.bfloat16 and pages.dtype == torch.bfloat16 and q.shape[-1] == 576
            and pages.shape[-1] == 576 and pages.shape[1] == PAGE_SIZE and pages.is_contiguous())


def _aligned_rows(out: torch.Tensor) -> bool:
    """The tensor-core kernels store 16 bytes at a time."""
    return out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0


def _tile_width(n: int) -> bool:
    return 8 <= n <= 128 and n % 8 == 0


def paged_kernel_supports(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor) -> bool:
    """Layouts of the tensor-core paged attention kernels: bf16, head sizes that are multiples of 8 up to 128."""
    return (q.is_cuda and q.dtype == torch.bfloat16 and k_pages.dtype == torch.bfloat16
            and _tile_width(q.shape[-1]) and _tile_width(v_pages.shape[-1]) and q.stride(0) % 8 == 0)


def decode_splits(splits: int, window: int | None, keep_first: int = 0) -> int:
    """Key splits of a layer's decode step: as many as planned for the whole context, but under a sliding window (with
    ``keep_first`` kept keys) no more than leave every split some tiles of 32 keys."""
    return splits if not window else int(max(1, min(splits, (window + keep_first + 31) // 32 // 4)))


def decode_kernel_supports(q: torch.Tensor, k_pages: torch.Tensor, v_dim: int | None = None) -> bool:
    Hq, D = q.shape[-2], q.shape[-1]
    Hkv = k_pages.shape[2]
    return (q.is_cuda and q.dtype == torch.bfloat16 and _tile_width(D) and _tile_width(v_dim or D) and Hq % Hkv == 0
            and Hq // Hkv <= 16 and k_pages.shape[1] == PAGE_SIZE and q.stride(-1) == 1 and q.stride(-2) == D)


def attn_combine(o_parts: torch.Tensor, lse_parts: torch.Tensor, sinks=None, want_lse: bool = False):
    """Merges ``o_parts [S, R, H, D]`` with ``lse_parts [S, H, R]`` (disjoint key ranges) into ``[R, H, D]``."""
    S_, R_, H, D = o_parts.shape
    if o_parts.is_cuda:
        o_parts = o_parts.contiguous()      # strides of size-1 dimensions are arbitrary: pass the dense pitch
        out = torch.empty(R_, H, D, dtype=o_parts.dtype, device=o_parts.device)
        lse = torch.empty(H, R_, dtype=torch.float32, device=o_parts.device) if want_lse else None
        _lib.call("edl_attn_combine", o_parts.data_ptr(), R_ * H * D, lse_parts.contiguous().data_ptr(), S_, R_,
                  H, D, _lib.ptr(sinks), out.data_ptr(), _lib.ptr(lse), _lib.stream_ptr())
        return (out, lse) if want_lse else out
    l = lse_parts.float().permute(0, 2, 1)                      # [S, R, H]
    if sinks is not None:
        l_all = torch.cat([l, sinks.float()[None, None].expand(1, R_, H)], 0)
    else:
        l_all = l
    tot = torch.logsumexp(l_all, 0)                             # [R, H]
    w = torch.exp(l - tot[None]).nan_to_num(0.0)
    out = (w[..., None] * o_parts.float()).sum(0).to(o_parts.dtype)
    return (out, tot.t().contiguous()) if want_lse else out


def paged_attention_splitkv(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, kv_lens: torch.Tensor,
                            page_table: torch.Tensor, num_splits: int, *, scale: float | None = None,
                            softcap: float = 0.0, sinks=None) -> torch.Tensor:
    """Decode attention (one query token per sequence) with every sequence's keys cut into ``num_splits`` page
    ranges that run as independent rows of the paged kernel and are merged by :func:`attn_combine`.

    With few sequences and long contexts the plain kernel has ``B * Hkv`` CTAs walking thousands of keys each;
    splitting gives the idle SMs work. q ``[B, Hq, D]``; the page table's width is padded to a multiple of
    ``num_splits`` pages so that each split is a strided view of it.
    """
    B, Hq, D = q.shape
    S_ = int(num_splits)
    MP = page_table.shape[1]
    cp = (MP + S_ - 1) // S_
    if cp * S_ != MP:
        page_table = torch.nn.functional.pad(page_table, (0, cp * S_ - MP))
    pt = page_table.contiguous().view(B * S_, cp)
    chunk = cp * PAGE_SIZE
    starts = torch.arange(S_, device=q.device, dtype=torch.int32) * chunk
    lens = (kv_lens.to(torch.int32)[:, None] - starts[None]).clamp(0, chunk).reshape(-1).contiguous()
    scale = scale if scale is not None else 1.0 / math.sqrt(D)
    if not q.is_cuda:
        o = paged_attention_reference(q, k_pages, v_pages, torch.arange(B + 1, dtype=torch.int32), kv_lens,
                                      page_table[:, :MP], scale=scale, causal=True, softcap=softcap, sinks=sinks)
        return o
    qr = q.repeat_interleave(S_, 0).contiguous()
    cu = torch.arange(B * S_ + 1, device=q.device, dtype=torch.int32)
    o_parts = torch.empty(B * S_, Hq, D, dtype=q.dtype, device=q.device)
    lse = torch.empty(Hq, B * S_, dtype=torch.float32, device=q.device)
    _lib.call("edl_attn_paged_lse", qr.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), o_parts.data_ptr(),
              lse.data_ptr(), qr.stride(0), k_pages.stride(1), v_pages.stride(1), o_parts.stride(0), cu.data_ptr(),
              lens.data_ptr(), pt.data_ptr(), pt.stride(0), B * S_, 1, B * S_, k_pages.shape[0], Hq, k_pages.shape[2],
              D, D, float(scale), 1, 0, float(softcap or 0.0), None, _lib.status_word(q.device).data_ptr(), _lib.stream_ptr())
    # [B*S, Hq, D] -> [S, B, Hq, D]; lse [Hq, B*S] -> [S, Hq, B]
    op = o_parts.view(B, S_, Hq, D).transpose(0, 1).contiguous()
    lp = lse.view(Hq, B, S_).permute(2, 0, 1).contiguous()
    return attn_combine(op, lp, sinks)


def paged_attention_reference(q, k_pages, v_pages, cu_q, kv_lens, page_table, *, scale=None, causal=True, window=0,
                              softcap=0.0, sinks=None, keep_first=0, sigmoid=None):
    """Dense oracle: gathers each sequence's keys/values from its pages and runs reference attention."""
    from . import reference as R

    page = k_pages.shape[1]
    outs = []
    cu = cu_q.tolist()
    for b, L in enumerate(kv_lens.tolist()):
        qs = q[cu[b]:cu[b + 1]]
        if qs.shape[0] == 0:
            continue
        n_pages = (L + page - 1) // page
        ids = page_table[b, :n_pages].long()
        ks = k_pages[ids].reshape(-1, *k_pages.shape[2:])[:L]
        vs = v_pages[ids].reshape(-1, *v_pages.shape[2:])[:L]
        o = R.attention(qs[None], ks[None].to(qs.dtype), vs[None].to(qs.dtype), causal=causal, scale=scale,
                        sliding_window=window or None, softcap=softcap, sinks=sinks, keep_first=keep_first,
                        score_bias=None if sigmoid is None else sigmoid.bias)
        outs.append(o[0])
    o = torch.cat(outs, dim=0)
    return o if sigmoid is None else sigmoid.finish(o)


def sample(logits: torch.Tensor, *, temperature=None, top_k=None, top_p=None, min_p=None, presence=None,
           frequency=None, repetition=None, counts=None, seeds=None, steps=None, want_logprob: bool = False):
    """Samples one token per row of ``[R, V]`` logits. All per-row parameter tensors are optional
    (absent = greedy, no penalties). Returns (tokens int32 [R], logprobs fp32 [R] or None)."""
    R_, V = logits.shape
    if logits.is_cuda:
        assert logits.stride(1) == 1 and logits.dtype in (torch.bfloat16, torch.float32)
        out = torch.empty(R_, dtype=torch.int32, device=logits.device)
        lp = torch.empty(R_, dtype=torch.float32, device=logits.device) if want_logprob else None
        _lib.call("edl_sample", logits.data_ptr(), int(logits.dtype == torch.float32), logits.stride(0), R_, V,
                  _lib.ptr(temperature), _lib.ptr(top_k), _lib.ptr(top_p), _lib.ptr(min_p), _lib.ptr(presence),
                  _lib.ptr(frequency), _lib.ptr(repetition), _lib.ptr(counts),
                  counts.stride(0) if counts is not None else 0, _lib.ptr(seeds), _lib.ptr(steps), out.data_ptr(),
                  _lib.ptr(lp), _lib.stream_ptr())
        return out, lp
    return sample_reference(logits, temperature=temperature, top_k=top_k, top_p=top_p, min_p=min_p,
                            presence=presence, frequency=frequency, repetition=repetition, counts=counts,
                            seeds=seeds, steps=steps, want_logprob=want_logprob)


def apply_penalties_reference(z: torch.Tensor, counts, presence, frequency, repetition) -> torch.Tensor:
    z = z.float().clone()
    if counts is None:
        return z
    seen = counts[: z.shape[0], : z.shape[1]] > 0
    if repetition is not None:
        rep = repetition[:, None]
        z = torch.where(seen, torch.where(z > 0, z / rep, z * rep), z)
    c = counts[: z.shape[0], : z.shape[1]].float()
    if presence is not None:
        z = z - presence[:, None] * seen
    if frequency is not None:
        z = z - frequency[:, None] * c
    return z


def sample_reference(logits, *, temperature=None, top_k=None, top_p=None, min_p=None, presence=None, frequency=None,
                     repetition=None, counts=None, seeds=None, steps=None, want_logprob=False):
    """CPU oracle with the kernel's order: penalties -> top-k (<= 64) -> temperature -> top-p -> min-p -> draw."""
    z = apply_penalties_reference(logits, counts, presence, frequency, repetition)
    R_, V = z.shape
    out = torch.empty(R_, dtype=torch.int32)
    lps = torch.empty(R_, dtype=torch.float32)
    for r in range(R_):
        t = float(temperature[r]) if temperature is not None else 0.0
        k = int(top_k[r]) if top_k is not None else 0
        if t <= 0 or k == 1:
            i = int(torch.argmax(z[r]))
            out[r] = i
            lps[r] = torch.log_softmax(z[r], -1)[i]
            continue
        k = 64 if (k <= 0 or k > 64) else k
        vals, idx = torch.topk(z[r], min(k, V))
        p = torch.softmax(vals / t, -1)
        keep = torch.ones_like(p, dtype=torch.bool)
        tp = float(top_p[r]) if top_p is not None else 1.0
        mp = float(min_p[r]) if min_p is not None else 0.0
        cum = torch.cumsum(p, 0) - p
        keep &= (cum < tp)
        keep &= p >= mp * p[0]
        keep[0] = True
        p = torch.where(keep, p, torch.zeros_like(p))
        g = torch.Generator().manual_seed(int(seeds[r]) + 7919 * int(steps[r] if steps is not None else 0)
                                          if seeds is not None else r)
        j = int(torch.multinomial(p / p.sum(), 1, generator=g))
        out[r] = int(idx[j])
        lps[r] = torch.log_softmax(z[r] / t, -1)[idx[j]]
    return out, (lps if want_logprob else None)


def count_update(counts: torch.Tensor, tokens: torch.Tensor, row_slots: torch.Tensor | None = None) -> None:
    if counts.is_cuda:
        _lib.call("edl_count_update", counts.data_ptr(), counts.stride(0), tokens.data_ptr(), _lib.ptr(row_slots),
                  tokens.numel(), counts.shape[1], _lib.stream_ptr())
        return
    rows = row_slots.long() if row_slots is not None else torch.arange(tokens.numel())
    ok = (tokens >= 0) & (rows >= 0)
    counts.index_put_((rows[ok], tokens[ok].long()), torch.ones(int(ok.sum()), dtype=counts.dtype), accumulate=True)


def gather_rows(src: torch.Tensor, idx: torch.Tensor) -> torch.Tensor:
    """``src[idx]`` for a 2-D bf16 matrix (last hidden state of every sequence)."""
    if src.is_cuda and src.dtype == torch.bfloat16 and src.shape[1] % 8 == 0:
        out = torch.empty((idx.numel(), src.shape[1]), dtype=src.dtype, device=src.device)
        _lib.call("edl_gather_rows", src.data_ptr(), idx.data_ptr(), out.data_ptr(), idx.numel(), src.shape[1],
                  src.stride(0), _lib.stream_ptr())
        return out
    return src[idx.long()]
