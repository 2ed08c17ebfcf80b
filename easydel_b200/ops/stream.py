"""Operations around an fp32 residual stream (``csrc/stream_ops.cu``).

Models that keep the sum of their branches in 32 bits hold ``x [T, W]`` as fp32: branches read it through
:func:`norm_shift` (RMS norm, optionally blended with the previous token's row) and add their output projection into
it with :func:`linear_add_`. CUDA tensors run the kernels (inference only: the stream is updated in place); CPU tensors
and calls under autograd run the tensor forms below, which return new tensors.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as tF

from . import _lib, kernels as K, reference as R, rotation

vp, i32, i64, f32 = _lib.vp, _lib.i32, _lib.i64, _lib.f32
_lib.register("edl_embed_stream", i32, [vp, i32, vp, f32, vp, vp, i64, i32, i32, i32, vp, vp])
_lib.register("edl_cast_rows", i32, [vp, vp, i32, i64, i32, i32, vp])
_lib.register("edl_norm_shift", i32, [vp, vp, vp, f32, i32, i32, vp, i32, vp, vp, i64, f32, vp, i32, vp])
_lib.register("edl_head_norm", i32, [vp, vp, f32, i64, i32, vp, i32, vp])
_lib.register("edl_xielu", i32, [vp, vp, vp, i32, i64, vp])
_lib.register("edl_gelu_erf", i32, [vp, vp, i32, i64, vp])
_lib.register("edl_post_norm", i32, [vp, vp, vp, vp, vp, i32, f32, f32, i32, vp, f32, f32, vp, i32, i32, i32, vp])
_lib.register("edl_scale_cap", i32, [vp, i64, f32, f32, vp])
_lib.register("edl_qkv_prologue", i32, [vp, i32, i64, vp, vp, vp, vp, f32, f32, f32, i32, i32, i32, i32, i32, vp, vp, vp,
                                        i64, i64, i64, vp, vp])
_lib.register("edl_qkv_rotary_prologue", i32, [vp, i32, i64, vp, vp, vp, vp, f32, vp, i32, i32, f32, vp, vp, i64, vp, i32, i32,
                                               i32, i32, i32, vp, vp, vp, i64, i64, i64, vp, vp])
_lib.register("edl_branch_norm", i32, [vp, vp, vp, vp, f32, vp, f32, vp, i32, i32, i32, vp])
_lib.register("edl_gated_unit", i32, [vp, i32, i64, vp, i32, i32, i32, vp])


def on_kernels(t: torch.Tensor) -> bool:
    """Kernels for CUDA tensors outside autograd."""
    return _lib.use_kernels(t) and not torch.is_grad_enabled()


def _f32flag(dtype: torch.dtype) -> int:
    if dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"fp32-stream operations take bf16 or fp32 operands, got {dtype}")
    return int(dtype == torch.float32)


# ---------------------------------------------------------------------------------------------- products
def _fp32_product(x: torch.Tensor, w: torch.Tensor, bias, out: torch.Tensor | None) -> torch.Tensor:
    """True 32-bit product (no TF32), through the vendor library: the tensor cores have no fp32 mode."""
    allow = torch.backends.cuda.matmul.allow_tf32
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        if out is not None:
            return out.addmm_(x, w.t()) if bias is None else out.addmm_(x, w.t()).add_(bias)
        return tF.linear(x, w, bias)
    finally:
        torch.backends.cuda.matmul.allow_tf32 = allow


def _tile_ok(x: torch.Tensor, w: torch.Tensor) -> bool:
    return w.shape[0] % 8 == 0 and w.shape[1] % 8 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0


def linear(x: torch.Tensor, w: torch.Tensor, bias: torch.Tensor | None = None,
           out_dtype: torch.dtype | None = None) -> torch.Tensor:
    """``x @ w.T (+ bias)`` for a 2-D ``x`` in the operand type, result in ``out_dtype`` (default: the operand type;
    fp32 results of bf16 products come straight from the fp32 accumulators)."""
    out_dtype = out_dtype or x.dtype
    if on_kernels(x) and x.dtype == torch.bfloat16 and _tile_ok(x, w):
        return K.gemm(x, w, bias=bias, out_dtype=out_dtype)
    if x.dtype == torch.float32 and x.is_cuda:
        return _fp32_product(x, w, bias, None).to(out_dtype)
    if out_dtype == torch.float32 and x.dtype != torch.float32:
        # sizes outside the GEMM's 16-byte rows, CPU and autograd
        return tF.linear(x.float(), w.float(), None if bias is None else bias.float())
    return tF.linear(x, w, bias).to(out_dtype)


def linear_add_(stream: torch.Tensor, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``stream + x @ w.T`` with fp32 accumulation into the fp32 ``stream [T, W]`` (in place on the kernels); returns
    the updated stream."""
    if on_kernels(x):
        if x.dtype == torch.bfloat16 and _tile_ok(x, w):
            K.gemm(x, w, out=stream, accumulate=True)
            return stream
        if x.dtype == torch.float32:
            return _fp32_product(x, w, None, stream)
        return stream.add_(tF.linear(x.float(), w.float()))
    return stream + tF.linear(x, w).float()


def branch_product(x: torch.Tensor, w: torch.Tensor, base: torch.Tensor | None = None,
                   bias: torch.Tensor | None = None) -> torch.Tensor:
    """``x @ w.T (+ bias)`` as fp32 rows, added to the fp32 rows ``base`` (in place on the kernels) if there are any."""
    if base is None:
        return linear(x, w, bias, torch.float32)
    out = linear_add_(base, x, w)
    return out if bias is None else out + bias.float()


def bmm(a: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """Batched product in the operand type, true 32-bit for fp32 (vendor library)."""
    allow = torch.backends.cuda.matmul.allow_tf32
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        return torch.bmm(a, b)
    finally:
        torch.backends.cuda.matmul.allow_tf32 = allow


# ---------------------------------------------------------------------------------------------- rows of the stream
def embed(table: torch.Tensor, ids: torch.Tensor, right: torch.Tensor | None = None, scale: float = 1.0) -> torch.Tensor:
    """fp32 rows ``table[ids] * scale`` ``[T, W]``; ``right`` (a view ``[T, W]`` of the right half of a ``[x ; x0]``
    operand) receives the same rows in the table's type."""
    ids = ids.reshape(-1)
    W = table.shape[1]
    if on_kernels(table):
        ids = ids.to(torch.int64).contiguous()
        x = torch.empty(ids.numel(), W, dtype=torch.float32, device=table.device)
        _lib.call("edl_embed_stream", table.data_ptr(), _f32flag(table.dtype), ids.data_ptr(), float(scale), x.data_ptr(),
                  _lib.ptr(right), right.stride(0) if right is not None else 0, ids.numel(), W, table.shape[0],
                  _lib.status_word(table.device).data_ptr(), _lib.stream_ptr())
        return x
    rows = table[ids.long()].float() * scale
    if right is not None:
        right.copy_(rows)
    return rows


def cast_rows(x: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """Writes the fp32 rows ``x [T, W]`` into the view ``out [T, W]`` in its type."""
    if on_kernels(x):
        _lib.call("edl_cast_rows", x.data_ptr(), out.data_ptr(), _f32flag(out.dtype), out.stride(0), x.shape[0],
                  x.shape[1], _lib.stream_ptr())
        return out
    out.copy_(x)
    return out


def norm_shift_reference(x, w, eps, out_dtype, mu=None, cu=None, slots=None, state=None):
    h = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w
    if mu is None:
        return h.to(out_dtype)
    before = torch.cat([h.new_zeros(1, h.shape[1]), h[:-1]])
    bounds = cu.tolist()
    rows = list(range(len(bounds) - 1)) if slots is None else slots.tolist()
    first = [(b, s) for b, s in enumerate(bounds[:-1]) if bounds[b + 1] > s]
    if first:
        idx = torch.tensor([s for _, s in first], device=x.device)
        init = torch.stack([state[rows[b]] if state is not None else torch.zeros_like(h[0]) for b, _ in first])
        before = before.index_copy(0, idx, init.to(h.dtype))
    if state is not None:
        with torch.no_grad():
            for b, _ in first:
                state[rows[b]] = h[bounds[b + 1] - 1]
    return (h + (before - h) * mu).to(out_dtype)


def norm_shift(x: torch.Tensor, w: torch.Tensor, eps: float, out_dtype: torch.dtype, mu: torch.Tensor | None = None,
               cu: torch.Tensor | None = None, slots: torch.Tensor | None = None,
               state: torch.Tensor | None = None, offset: float = 0.0) -> torch.Tensor:
    """RMS norm of the fp32 stream ``x [T, W]`` times ``w + offset`` (fp32), in 32 bits, cast once to ``out_dtype``.

    ``mu`` (fp32 ``[W]``): token shift. Row t becomes ``h_t + (h_{t-1} - h_t) * mu`` inside the sequences bounded by
    ``cu`` (int32 ``[B + 1]``); the row before a sequence's first one comes from ``state[slots[b]]`` (fp32
    ``[*, W]``, zeros without a state), which then receives the sequence's last unshifted row."""
    if on_kernels(x):
        out = torch.empty(x.shape, dtype=out_dtype, device=x.device)
        nseq = cu.numel() - 1 if cu is not None else 0
        _lib.call("edl_norm_shift", x.data_ptr(), w.data_ptr(), _lib.ptr(mu), float(eps), x.shape[0], x.shape[1],
                  _lib.ptr(cu), nseq, _lib.ptr(slots), _lib.ptr(state), state.stride(0) if state is not None else 0,
                  float(offset), out.data_ptr(), _f32flag(out_dtype), _lib.stream_ptr())
        return out
    return norm_shift_reference(x, w.float() + offset, eps, out_dtype, None if mu is None else mu.float(), cu, slots, state)


def head_norm(o: torch.Tensor, w: torch.Tensor, eps: float, out_dtype: torch.dtype) -> torch.Tensor:
    """RMS norm of fp32 ``o [T, H, V]`` over V with one weight vector for all heads."""
    if on_kernels(o):
        out = torch.empty(o.shape, dtype=out_dtype, device=o.device)
        _lib.call("edl_head_norm", o.data_ptr(), w.data_ptr(), float(eps), o.numel() // o.shape[-1], o.shape[-1],
                  out.data_ptr(), _f32flag(out_dtype), _lib.stream_ptr())
        return out
    return (o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * w.float()).to(out_dtype)


def xielu(z: torch.Tensor, act: torch.Tensor) -> torch.Tensor:
    """xIELU with raw parameters ``act = (p, q)``: ``softplus(p) z^2 + z / 2`` for z > 0, else
    ``(1/2 + softplus(q)) (e^z - 1 - z) + z / 2``."""
    if on_kernels(z):
        z = z if z.is_contiguous() else z.contiguous()
        y = torch.empty_like(z)
        _lib.call("edl_xielu", z.data_ptr(), act.data_ptr(), y.data_ptr(), _f32flag(z.dtype), z.numel(),
                  _lib.stream_ptr())
        return y
    zf, a = z.float(), act.float()
    ap, an = tF.softplus(a[0]), 0.5 + tF.softplus(a[1])
    neg = zf.clamp(max=0.0)
    return torch.where(zf > 0, ap * zf * zf + 0.5 * zf, an * (torch.expm1(neg) - neg) + 0.5 * neg).to(z.dtype)


def gelu_erf(z: torch.Tensor) -> torch.Tensor:
    """Exact GELU, ``z / 2 (1 + erf(z / sqrt 2))``."""
    if on_kernels(z):
        z = z if z.is_contiguous() else z.contiguous()
        y = torch.empty_like(z)
        _lib.call("edl_gelu_erf", z.data_ptr(), y.data_ptr(), _f32flag(z.dtype), z.numel(), _lib.stream_ptr())
        return y
    return tF.gelu(z)


def gated_unit(gu: torch.Tensor, act: str = "silu") -> torch.Tensor:
    """``act(gate) * up`` for rows ``gu [T, 2 F] = [gate | up]``."""
    if on_kernels(gu):
        F = gu.shape[1] // 2
        if gu.dtype == torch.bfloat16 and F % 8 == 0 and gu.stride(0) % 8 == 0 and act in K.ACT_IDS:
            return K.gated_act_fwd(gu, act)
        if act in K.ACT_IDS and gu.stride(1) == 1:
            out = torch.empty(gu.shape[0], F, dtype=gu.dtype, device=gu.device)
            _lib.call("edl_gated_unit", gu.data_ptr(), _f32flag(gu.dtype), gu.stride(0), out.data_ptr(), gu.shape[0], F,
                      K.ACT_IDS[act], _lib.stream_ptr())
            return out
    return R.gated_act(gu, act)


def scale_cap(z: torch.Tensor, scale: float = 1.0, cap: float = 0.0) -> torch.Tensor:
    """``cap tanh(scale z / cap)`` for fp32 ``z`` (``scale z`` without a cap), in place on the kernels."""
    if on_kernels(z):
        assert z.dtype == torch.float32 and z.is_contiguous()
        _lib.call("edl_scale_cap", z.data_ptr(), z.numel(), float(scale), float(cap), _lib.stream_ptr())
        return z
    z = z * scale
    return torch.tanh(z / cap) * cap if cap else z


# ---------------------------------------------------------------------------------------------- norm after the sum
def _sum_and_norm(x, branch, alpha, beta, keep_sum, w, eps, out_dtype, offset):
    rows = None if isinstance(branch, torch.Tensor) else branch
    if on_kernels(x):
        h = torch.empty(x.shape, dtype=out_dtype, device=x.device)
        y = branch if rows is None else rows.base
        if y is not None and (y.dtype != torch.float32 or not y.is_contiguous()):
            y = y.float().contiguous()
        assert x.is_contiguous() and (rows is None or rows.ys.dtype == out_dtype)
        _lib.call("edl_post_norm", x.data_ptr(), _lib.ptr(y), _lib.ptr(rows.ys) if rows else None,
                  _lib.ptr(rows.weights) if rows else None, _lib.ptr(rows.pos) if rows else None, rows.k if rows else 0,
                  float(alpha), float(beta), int(keep_sum), w.data_ptr(), float(offset), float(eps), h.data_ptr(),
                  _f32flag(out_dtype), x.shape[0], x.shape[1], _lib.stream_ptr())
        return x, h
    s = x * alpha + branch_rows(branch) * beta
    v = s * torch.rsqrt(s.pow(2).mean(-1, keepdim=True) + eps) * (w.float() + offset)
    return s if keep_sum else v, v.to(out_dtype)


@dataclass
class NormedBranch:
    """A branch that is RMS-normed before it joins the stream: ``rms_norm(rows) * weight * scale`` (all fp32; ``scale [W]``:
    one factor per channel, or None)."""

    rows: torch.Tensor
    weight: torch.Tensor
    eps: float
    scale: torch.Tensor | None = None

    def combine(self) -> torch.Tensor:
        f = self.rows.float()
        y = f * torch.rsqrt(f.pow(2).mean(-1, keepdim=True) + self.eps) * self.weight.float()
        return y if self.scale is None else y * self.scale.float()


def branch_rows(branch) -> torch.Tensor:
    """A branch (fp32 rows, expert rows or a normed branch) as fp32 rows."""
    return branch.float() if isinstance(branch, torch.Tensor) else branch.combine()


def post_norm(x: torch.Tensor, branch, alpha: float, w: torch.Tensor, eps: float, out_dtype: torch.dtype,
              offset: float = 0.0) -> tuple[torch.Tensor, torch.Tensor]:
    """``rms_norm(alpha x + branch) * (w + offset)`` over the fp32 stream ``x [T, W]`` in 32 bits: the new stream (in place
    on the kernels) and the same rows as the operand of the next product. ``branch``: fp32 rows ``[T, W]``, or an
    :class:`..ops.moe_kernels.ExpertRows`, whose weighted sum over each token's experts happens in the same pass."""
    return _sum_and_norm(x, branch, alpha, 1.0, False, w, eps, out_dtype, offset)


def add_norm(x: torch.Tensor, branch, mult: float, w: torch.Tensor, eps: float, out_dtype: torch.dtype,
             offset: float = 0.0) -> tuple[torch.Tensor, torch.Tensor]:
    """``x + mult branch`` (in place on the kernels; ``branch`` as in :func:`post_norm`, a :class:`NormedBranch`, or None) and
    the RMS norm of the sum, ``* (w + offset)``, as the operand of the next products."""
    if branch is None:
        return x, norm_shift(x, w, eps, out_dtype, offset=offset)
    if isinstance(branch, NormedBranch) and on_kernels(x) and mult == 1.0 and offset == 0.0:
        y = branch.rows
        assert x.is_contiguous() and y.is_contiguous() and y.dtype == torch.float32 and branch.weight.dtype == torch.float32
        h = torch.empty(x.shape, dtype=out_dtype, device=x.device)
        _lib.call("edl_branch_norm", x.data_ptr(), y.data_ptr(), branch.weight.data_ptr(), _lib.ptr(branch.scale),
                  float(branch.eps), w.data_ptr(), float(eps), h.data_ptr(), _f32flag(out_dtype), x.shape[0], x.shape[1],
                  _lib.stream_ptr())
        return x, h
    if isinstance(branch, NormedBranch):
        branch = branch.combine()
    return _sum_and_norm(x, branch, 1.0, mult, True, w, eps, out_dtype, offset)


# ---------------------------------------------------------------------------------------------- attention prologue
def query_temperature(positions: torch.Tensor, temp: tuple[float, float]) -> torch.Tensor:
    """``1 + coef * ln(floor((p + 1) / every) + 1)`` in fp32; ``temp = (coef, every)``."""
    coef, every = temp
    return torch.log(torch.floor((positions.float() + 1.0) / every) + 1.0) * coef + 1.0


def qk_norm_temper(q, k, qw, kw, eps, positions=None, temp=None):
    """Tensor form of the q / k half of the prologue: ``q [T, H, D]``, ``k [T, G, D]`` -> the same, normed and tempered
    in fp32 and cast back."""
    def norm(x, w):
        xf = x.float()
        return xf if w is None else xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w.float()

    qf = norm(q, qw)
    if temp is not None:
        qf = qf * query_temperature(positions.reshape(-1), temp)[:, None, None]
    return qf.to(q.dtype), norm(k, kw).to(k.dtype)


def qkv_prologue(qkv: torch.Tensor, heads: tuple[int, int, int, int], qw, kw, eps: float, positions: torch.Tensor,
                 temp: tuple[float, float] | None, slot_mapping: torch.Tensor, k_pages: torch.Tensor,
                 v_pages: torch.Tensor) -> torch.Tensor:
    """Packed projection rows ``qkv [T, Hq D + Hkv D + Hkv Dv]`` -> normed, tempered queries ``[T, Hq, D]``; the normed
    keys and the values are appended to their pages. ``heads = (Hq, Hkv, D, Dv)``."""
    Hq, Hkv, D, Dv = heads
    T = qkv.shape[0]
    if on_kernels(qkv):
        q = torch.empty(T, Hq, D, dtype=qkv.dtype, device=qkv.device)
        pos = positions.reshape(-1).to(torch.int32)
        coef, every = temp if temp is not None else (0.0, 0.0)
        _lib.call("edl_qkv_prologue", qkv.data_ptr(), _f32flag(qkv.dtype), qkv.stride(0), pos.data_ptr(),
                  slot_mapping.data_ptr(), _lib.ptr(qw), _lib.ptr(kw), float(eps), float(coef), float(every), T, Hq, Hkv,
                  D, Dv, q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), k_pages.stride(1), v_pages.stride(1),
                  k_pages.shape[0] * k_pages.shape[1], _lib.status_word(qkv.device).data_ptr(), _lib.stream_ptr())
        return q
    from . import serving as S

    q, k, v = torch.split(qkv, [Hq * D, Hkv * D, Hkv * Dv], -1)
    q, k = qk_norm_temper(q.reshape(T, Hq, D), k.reshape(T, Hkv, D), qw, kw, eps, positions, temp)
    S.kv_append(k, v.reshape(T, Hkv, Dv), k_pages, v_pages, slot_mapping)
    return q


def qkv_rotary_prologue(qkv: torch.Tensor, heads: tuple[int, int, int, int], qw, kw, eps: float, positions: torch.Tensor,
                        freq: torch.Tensor | None, slot_mapping: torch.Tensor, k_pages: torch.Tensor,
                        v_pages: torch.Tensor, layout: str = "halves", mag: float = 1.0, bias: torch.Tensor | None = None,
                        first: torch.Tensor | None = None, lam: torch.Tensor | None = None) -> torch.Tensor:
    """:func:`qkv_prologue` for queries and keys that are normed over the whole projection (all heads at once; weights
    ``qw [Hq D]``, ``kw [Hkv D]``, None: no norm) and then rotated: the pairs of every head (``layout``, ``freq``: see
    :mod:`.rotation`; None: no rotation) by the position times their frequency, cosines and sines times ``mag``.
    ``bias`` fp32 ``[Hq D + Hkv (D + Dv)]`` is added first. ``lam`` (fp32 scalar): the cached values are ``(1 - lam) v + lam
    first``, ``first [T, Hkv, Dv]`` in the operand type (rows may be strided)."""
    Hq, Hkv, D, Dv = heads
    T = qkv.shape[0]
    if on_kernels(qkv):
        q = torch.empty(T, Hq, D, dtype=qkv.dtype, device=qkv.device)
        pos = positions.reshape(-1).to(torch.int32)
        _lib.call("edl_qkv_rotary_prologue", qkv.data_ptr(), _f32flag(qkv.dtype), qkv.stride(0), pos.data_ptr(),
                  slot_mapping.data_ptr(), _lib.ptr(qw), _lib.ptr(kw), float(eps), _lib.ptr(freq),
                  freq.numel() // 2 if freq is not None else 0, int(layout == "neighbours"), float(mag), _lib.ptr(bias),
                  _lib.ptr(first), first.stride(0) if first is not None else 0, _lib.ptr(lam), T, Hq, Hkv, D, Dv,
                  q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), k_pages.stride(1), v_pages.stride(1),
                  k_pages.shape[0] * k_pages.shape[1], _lib.status_word(qkv.device).data_ptr(), _lib.stream_ptr())
        return q
    from . import serving as S

    q, k, v = rotary_rows(qkv, heads, qw, kw, eps, positions, freq, layout, mag, bias, first, lam)
    S.kv_append(k, v, k_pages, v_pages, slot_mapping)
    return q


def rotary_rows(qkv, heads, qw, kw, eps: float, positions, freq, layout="halves", mag=1.0, bias=None, first=None, lam=None):
    """Tensor form of :func:`qkv_rotary_prologue` without the pages: ``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, Dv]``."""
    Hq, Hkv, D, Dv = heads
    dt = qkv.dtype
    if bias is not None:
        qkv = qkv.float() + bias.float()
    q, k, v = torch.split(qkv, [Hq * D, Hkv * D, Hkv * Dv], -1)
    q, k = qk_norm_rotate(q, k, D, qw, kw, eps, positions, freq, layout, mag)
    if lam is not None:
        v = (1.0 - lam.float()) * v.float() + lam.float() * first.float().flatten(1)
    return q.to(dt), k.to(dt), v.to(dt).reshape(-1, Hkv, Dv)


def qk_norm_rotate(q, k, D: int, qw, kw, eps: float, positions, freq, layout: str = "halves", mag: float = 1.0):
    """The q / k half of :func:`rotary_rows`: flat rows -> ``[T, H, D]`` and ``[T, G, D]``."""
    def one(x, w):
        xf = x.float()
        if w is not None:
            xf = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w.float()
        xf = xf.reshape(x.shape[0], -1, D)
        return (xf if freq is None else rotation.rotate(xf, positions.reshape(-1), freq, layout, mag)).to(x.dtype)

    return one(q, qw), one(k, kw)
