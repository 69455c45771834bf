"""Torch-facing wrappers of the C-ABI kernels.

Each function validates what only the Python side can know (device, dtype, contiguity of
the innermost dimension), passes raw device pointers, element strides and torch's current
stream to the library, and returns torch tensors.  CUDA tensors only.
"""
from typing import Optional, Tuple

import torch

from . import _capi
from ._capi import BASED_BF16, BASED_F32, IMPL_AUTO, IMPL_DECODE, IMPL_SIMT, IMPL_TCGEN05  # noqa: F401

EXPANDED_DIM = 273
_IMPLS = {"auto": IMPL_AUTO, "simt": IMPL_SIMT, "tcgen05": IMPL_TCGEN05, "decode": IMPL_DECODE}


def _dt(t: torch.dtype) -> int:
    if t == torch.float32:
        return BASED_F32
    if t == torch.bfloat16:
        return BASED_BF16
    raise TypeError(f"unsupported dtype {t}: the kernels take float32 or bfloat16")


def _need_cuda(*ts):
    """Every op starts here: CUDA tensors only, and no autograd.  The kernels write into fresh buffers through
    raw pointers and register no backward, so under grad mode the result would silently be cut off from the
    graph (the projections before a mixer would get no gradient and nothing would say so)."""
    for t in ts:
        if t is not None and not t.is_cuda:
            raise RuntimeError("based_b200 ops run on CUDA tensors only (there is no CPU path)")
    if torch.is_grad_enabled():
        for t in ts:
            if t is not None and t.requires_grad:
                raise RuntimeError(
                    "based_b200 kernels are inference-only (no backward): call them under torch.no_grad() or "
                    "torch.inference_mode(), or detach the inputs")


def check_status(reset: bool = True) -> int:
    """Read the tensor-core kernels' status word and raise if a bounded in-kernel wait ever expired (the results
    of that launch are then meaningless).  It synchronises the device, so call it where the caller synchronises
    anyway: after a generation loop, at the end of a timed region."""
    code = _capi.read_status(reset)
    if code != 0:
        raise _capi.BasedLibraryError(f"a bounded wait expired inside a tensor-core kernel (status 0x{code:x}); "
                                      "the outputs of that launch are not valid")
    return code


def _inner_contig(t, name):
    if t.stride(-1) != 1:
        raise ValueError(f"{name}: innermost stride must be 1")


def _rows(t, width):
    """``t [..., width]`` as a ``[M, width]`` view of the same memory (rows one constant stride apart)."""
    if t.shape[-1] != width or t.stride(-1) != 1:
        raise ValueError(f"out must be a [..., {width}] tensor with contiguous rows")
    return flat_rows(t)


def flat_rows(t):
    """``t [..., W]`` as ``[M, W]`` without a copy; raises when its rows are not one constant stride apart."""
    dims = [(n, st) for n, st in zip(t.shape[:-1], t.stride()[:-1]) if n != 1]
    for (_, outer), (n, inner) in zip(dims, dims[1:]):
        if outer != inner * n:
            raise ValueError("rows are not one constant stride apart")
    m = 1
    for n, _ in dims:
        m *= n
    return t.as_strided((m, t.shape[-1]), (dims[-1][1] if dims else t.shape[-1], t.stride(-1)))


def _position(pos, like):
    """(device pointer or None, scalar) of a call's first position: an int, or an int32 CUDA tensor with one per row."""
    if torch.is_tensor(pos):
        if pos.dtype != torch.int32 or pos.device != like.device or not pos.is_contiguous():
            raise TypeError("positions must be a contiguous int32 tensor on the inputs' device")
        if pos.numel() < like.shape[0]:
            raise ValueError("positions: one per batch row is needed")
        return pos.data_ptr(), 0
    return None, int(pos)


def _ptr(t):
    return None if t is None else t.data_ptr()


def _stream():
    return torch.cuda.current_stream().cuda_stream


def linattn_prefill(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, *, eps: float = 1e-12,
                    return_state: bool = True, state_dtype: Optional[torch.dtype] = None,
                    out: Optional[torch.Tensor] = None, impl: str = "auto",
                    kv_state: Optional[torch.Tensor] = None, k_state: Optional[torch.Tensor] = None,
                    nseg: Optional[int] = None, scratch: Optional[torch.Tensor] = None,
                    ) -> Tuple[torch.Tensor, Optional[torch.Tensor], Optional[torch.Tensor]]:
    """Causal Taylor linear attention over a whole sequence.

    q, k ``[B, H, L, 16]`` (raw), v ``[B, H, L, dv]``; any batch/head/seq strides (e.g. the
    transposed views LinearAttention.forward makes, linear_attention.py:127-129).
    Returns ``y`` as a ``[B, H, L, dv]`` view of a ``[B, L, H, dv]`` buffer (so the reference's
    ``'b h l d -> b l (h d)'`` rearrange is free), ``kv_state [B, H, 1, dv, 273]`` and
    ``k_state [B, H, 1, 1, 273]`` (linear_attention.py:220-222), or ``None`` for the states
    when ``return_state`` is false.  ``kv_state``/``k_state`` may be given to be filled in place.

    ``nseg`` splits the SEQUENCE into that many segments that run on different SMs (bf16, tensor-core
    kernel only): ``None`` lets the library choose (it splits only when ``B*H`` is below half the SM
    count and ``L >= 1024``), ``1`` never splits.  The split needs a workspace of
    ``based_linattn_prefill_scratch_bytes`` bytes; ``scratch`` (a CUDA uint8/float tensor at least that
    large) may be given to reuse one, else it is taken from torch's caching allocator.
    """
    _need_cuda(q, k, v)
    B, H, L, d = q.shape
    dv = v.shape[-1]
    if k.shape != q.shape or v.shape[:3] != q.shape[:3]:
        raise ValueError("q, k, v shapes disagree")
    if not (q.dtype == k.dtype == v.dtype):
        raise TypeError("q, k, v must share a dtype")
    for t, n in ((q, "q"), (k, "k"), (v, "v")):
        _inner_contig(t, n)
    if out is None:
        out = torch.empty(B, L, H, dv, dtype=q.dtype, device=q.device).permute(0, 2, 1, 3)
    else:
        _inner_contig(out, "out")
    sdt = kv_state.dtype if kv_state is not None else (state_dtype or q.dtype)
    if return_state:
        if kv_state is None:
            kv_state = torch.empty(B, H, 1, dv, EXPANDED_DIM, dtype=sdt, device=q.device)
            k_state = torch.empty(B, H, 1, 1, EXPANDED_DIM, dtype=sdt, device=q.device)
        elif not (kv_state.is_contiguous() and k_state.is_contiguous()):
            raise ValueError("kv_state / k_state must be contiguous")
    if L == 0 or B == 0 or H == 0:  # empty tensors have no device pointer to pass
        if return_state:
            kv_state.zero_()
            k_state.zero_()
        return out, (kv_state if return_state else None), (k_state if return_state else None)
    lib = _capi.lib()
    can_split = q.dtype == torch.bfloat16 and dv <= 112 and impl in ("auto", "tcgen05")
    if nseg is not None and nseg > 1 and not can_split:
        raise ValueError("nseg > 1 needs bf16 inputs, dv <= 112 and the tensor-core kernel")
    with torch.cuda.device(q.device):
        if nseg is None:
            nseg = lib.based_linattn_prefill_segments(B, H, L) if can_split else 1
        if nseg > 1:
            need = lib.based_linattn_prefill_scratch_bytes(B, H, L, dv, nseg)
            if scratch is None:
                scratch = torch.empty(max(need, 16), dtype=torch.uint8, device=q.device)
            elif scratch.device != q.device or not scratch.is_contiguous():
                raise ValueError("scratch must be a contiguous tensor on the inputs' device")
            code = lib.based_linattn_prefill_split(
                q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(),
                kv_state.data_ptr() if return_state else None, k_state.data_ptr() if return_state else None,
                B, H, L, d, dv,
                _capi.strides(*q.stride()[:3]), _capi.strides(*k.stride()[:3]),
                _capi.strides(*v.stride()[:3]), _capi.strides(*out.stride()[:3]),
                _dt(sdt), float(eps), int(nseg), scratch.data_ptr(), scratch.numel() * scratch.element_size(),
                _stream())
            _capi.check(code, "based_linattn_prefill_split")
            return out, (kv_state if return_state else None), (k_state if return_state else None)
        code = lib.based_linattn_prefill(
            q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(),
            kv_state.data_ptr() if return_state else None, k_state.data_ptr() if return_state else None,
            B, H, L, d, dv,
            _capi.strides(*q.stride()[:3]), _capi.strides(*k.stride()[:3]),
            _capi.strides(*v.stride()[:3]), _capi.strides(*out.stride()[:3]),
            _dt(q.dtype), _dt(sdt), float(eps), _IMPLS[impl], _stream())
    _capi.check(code, "based_linattn_prefill")
    return out, (kv_state if return_state else None), (k_state if return_state else None)


def linattn_decode(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, kv_state: torch.Tensor,
                   k_state: torch.Tensor, *, eps: float = 1e-12, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One recurrent step; ``kv_state``/``k_state`` are updated IN PLACE.

    q, k ``[B, H, 1, 16]`` or ``[B, H, 16]`` (raw), v ``[B, H, 1, dv]`` or ``[B, H, dv]``;
    ``kv_state [B, H, 1, dv, 273]``, ``k_state [B, H, 1, 1, 273]`` (fp32 or bf16).
    Returns ``y [B, 1, H*dv]`` in ``q.dtype`` (the layout recurrent_forward hands to out_proj,
    linear_attention.py:251).
    """
    _need_cuda(q, k, v, kv_state, k_state)
    if q.dim() == 4:
        q, k, v = q[:, :, 0], k[:, :, 0], v[:, :, 0]
    B, H, d = q.shape
    dv = v.shape[-1]
    if kv_state.shape != (B, H, 1, dv, EXPANDED_DIM) or k_state.shape != (B, H, 1, 1, EXPANDED_DIM):
        raise ValueError(f"state shapes {tuple(kv_state.shape)}, {tuple(k_state.shape)} do not match B={B} H={H} dv={dv}")
    if not (kv_state.is_contiguous() and k_state.is_contiguous()):
        raise ValueError("kv_state / k_state must be contiguous")
    if kv_state.dtype != k_state.dtype:
        raise TypeError("kv_state and k_state must share a dtype")
    for t, n in ((q, "q"), (k, "k"), (v, "v")):
        _inner_contig(t, n)
    if out is None:
        out = torch.empty(B, 1, H * dv, dtype=q.dtype, device=q.device)
    y = out.view(B, H, dv)
    with torch.cuda.device(q.device):
        code = _capi.lib().based_linattn_decode(
            q.data_ptr(), k.data_ptr(), v.data_ptr(), y.data_ptr(), kv_state.data_ptr(), k_state.data_ptr(),
            B, H, d, dv, _capi.strides(*q.stride()[:2]), _capi.strides(*k.stride()[:2]),
            _capi.strides(*v.stride()[:2]), _capi.strides(*y.stride()[:2]),
            _dt(q.dtype), _dt(kv_state.dtype), float(eps), _stream())
    _capi.check(code, "based_linattn_decode")
    return out


def swa_prefill(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, window_left: int,
                softmax_scale: Optional[float] = None, *, impl: str = "auto",
                out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal sliding-window softmax attention; q, k, v ``[B, L, H, hd]`` (views into a packed
    qkv tensor are fine).  Query i sees keys ``[i - window_left, i]`` (slide_attention.py:97)."""
    _need_cuda(q, k, v)
    B, L, H, hd = q.shape
    if k.shape != q.shape or v.shape != q.shape:
        raise ValueError("q, k, v shapes disagree")
    for t, n in ((q, "q"), (k, "k"), (v, "v")):
        _inner_contig(t, n)
    if out is None:
        out = torch.empty(B, L, H, hd, dtype=q.dtype, device=q.device)
    scale = hd ** -0.5 if softmax_scale is None else float(softmax_scale)
    if out.numel() == 0:
        return out
    with torch.cuda.device(q.device):
        code = _capi.lib().based_swa_prefill(
            q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), B, L, H, hd,
            _capi.strides(*q.stride()[:3]), _capi.strides(*k.stride()[:3]),
            _capi.strides(*v.stride()[:3]), _capi.strides(*out.stride()[:3]),
            int(window_left), scale, _dt(q.dtype), _IMPLS[impl], _stream())
    _capi.check(code, "based_swa_prefill")
    return out


def swa_decode(q: torch.Tensor, k_new: torch.Tensor, v_new: torch.Tensor, kv_cache: torch.Tensor,
               cache_seqlens, window_left: int, softmax_scale: Optional[float] = None, *,
               rotary_cos: Optional[torch.Tensor] = None, rotary_sin: Optional[torch.Tensor] = None,
               out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One decode step: optional RoPE at the new position, append to ``kv_cache
    [B, maxL, 2, H, hd]`` IN PLACE, attend over the window (slide_attention.py:414-427).
    q, k_new, v_new ``[B, 1, H, hd]``; ``cache_seqlens`` an int or an int32 ``[B]`` CUDA tensor."""
    _need_cuda(q, k_new, v_new, kv_cache)
    B, one, H, hd = q.shape
    assert one == 1
    if not kv_cache.is_contiguous() or kv_cache.shape[0] < B or kv_cache.shape[2:] != (2, H, hd):
        raise ValueError("kv_cache must be contiguous [B, maxL, 2, H, hd]")
    if kv_cache.dtype != q.dtype:
        raise TypeError("kv_cache and q must share a dtype")
    q3, k3, v3 = q[:, 0], k_new[:, 0], v_new[:, 0]
    for t, n in ((q3, "q"), (k3, "k_new"), (v3, "v_new")):
        _inner_contig(t, n)
    if out is None:
        out = torch.empty(B, 1, H, hd, dtype=q.dtype, device=q.device)
    o3 = out[:, 0]
    if torch.is_tensor(cache_seqlens):
        if cache_seqlens.dtype != torch.int32 or not cache_seqlens.is_cuda or not cache_seqlens.is_contiguous():
            raise TypeError("cache_seqlens must be a contiguous int32 CUDA tensor")
        import ctypes
        lens_ptr = ctypes.cast(cache_seqlens.data_ptr(), ctypes.POINTER(ctypes.c_int32))
        lens_scalar = 0
    else:
        lens_ptr, lens_scalar = None, int(cache_seqlens)
    rdim = 0
    if rotary_cos is not None:
        if rotary_cos.dtype != q.dtype or rotary_sin.dtype != q.dtype:
            raise TypeError("rotary tables must be in the q dtype")
        if not (rotary_cos.is_contiguous() and rotary_sin.is_contiguous()):
            raise ValueError("rotary tables must be contiguous")
        rdim = 2 * rotary_cos.shape[-1]
    scale = hd ** -0.5 if softmax_scale is None else float(softmax_scale)
    with torch.cuda.device(q.device):
        code = _capi.lib().based_swa_decode(
            q3.data_ptr(), k3.data_ptr(), v3.data_ptr(), o3.data_ptr(), kv_cache.data_ptr(), lens_ptr, lens_scalar,
            rotary_cos.data_ptr() if rotary_cos is not None else None,
            rotary_sin.data_ptr() if rotary_sin is not None else None, rdim,
            B, H, hd, kv_cache.shape[1], _capi.strides(*q3.stride()[:2]), _capi.strides(*k3.stride()[:2]),
            _capi.strides(*v3.stride()[:2]), _capi.strides(*o3.stride()[:2]),
            int(window_left), scale, _dt(q.dtype), _stream())
    _capi.check(code, "based_swa_decode")
    return out


def rotary_apply_(x: torch.Tensor, rotary_cos: torch.Tensor, rotary_sin: torch.Tensor, seqlen_offset=0) -> torch.Tensor:
    """In-place non-interleaved RoPE on ``x [B, L, H, hd]`` (a view into packed qkv is fine);
    ``seqlen_offset`` an int or an int32 ``[B]`` CUDA tensor (based/ops/triton/rotary.py:68-105)."""
    _need_cuda(x, rotary_cos, rotary_sin)
    B, L, H, hd = x.shape
    _inner_contig(x, "x")
    if rotary_cos.dtype != x.dtype or rotary_sin.dtype != x.dtype:
        raise TypeError("rotary tables must be in the dtype of x")
    if not (rotary_cos.is_contiguous() and rotary_sin.is_contiguous()):
        raise ValueError("rotary tables must be contiguous")
    if x.numel() == 0:
        return x
    if torch.is_tensor(seqlen_offset):
        import ctypes
        if seqlen_offset.dtype != torch.int32 or not seqlen_offset.is_cuda:
            raise TypeError("seqlen_offset tensor must be int32 on CUDA")
        off_ptr, off_scalar = ctypes.cast(seqlen_offset.data_ptr(), ctypes.POINTER(ctypes.c_int32)), 0
        max_pos = None
    else:
        off_ptr, off_scalar = None, int(seqlen_offset)
        if off_scalar + L > rotary_cos.shape[0]:
            raise ValueError("rotary tables are shorter than seqlen_offset + L")
    with torch.cuda.device(x.device):
        code = _capi.lib().based_rotary_apply(
            x.data_ptr(), B, L, H, hd, _capi.strides(*x.stride()[:3]), rotary_cos.data_ptr(), rotary_sin.data_ptr(),
            2 * rotary_cos.shape[-1], off_ptr, off_scalar, _dt(x.dtype), _stream())
    _capi.check(code, "based_rotary_apply")
    return x


def gated_conv_prefill(u: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None, *,
                       state: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``silu(causal_depthwise_conv(u1) + bias) * u2`` with ``u1, u2`` the halves of ``u [B, L, 2*di]``.

    ``weight [di, k]`` (or ``[di, 1, k]`` as nn.Conv1d stores it), ``bias [di]`` or None, both in one
    dtype (float32 or bfloat16).  ``state [B, di, k]`` (dtype of ``u``), when given, receives the
    last k inputs of the convolution (convolution.py:63-67).  Returns ``v [B, L, di]``.
    """
    _need_cuda(u, weight, bias, state)
    B, L, two_di = u.shape
    di = two_di // 2
    weight = weight.reshape(weight.shape[0], -1)
    k = weight.shape[1]
    if weight.shape[0] != di or two_di != 2 * di:
        raise ValueError("u must be [B, L, 2*di] and weight [di, k]")
    _inner_contig(u, "u")
    weight = weight.contiguous()
    if bias is not None:
        bias = bias.to(weight.dtype).contiguous()
    if out is None:
        out = torch.empty(B, L, di, dtype=u.dtype, device=u.device)
    else:
        _inner_contig(out, "out")
    if state is not None and (state.shape != (B, di, k) or state.dtype != u.dtype or not state.is_contiguous()):
        raise ValueError("state must be a contiguous [B, di, k] tensor of u's dtype")
    if B == 0 or L == 0:
        if state is not None:
            state.zero_()
        return out
    u1, u2 = u[..., :di], u[..., di:]
    with torch.cuda.device(u.device):
        code = _capi.lib().based_gated_conv_prefill(
            u1.data_ptr(), u2.data_ptr(), out.data_ptr(), state.data_ptr() if state is not None else None,
            weight.data_ptr(), bias.data_ptr() if bias is not None else None, B, L, di, k,
            _capi.strides(*u1.stride()[:2]), _capi.strides(*u2.stride()[:2]), _capi.strides(*out.stride()[:2]),
            _dt(u.dtype), _dt(weight.dtype), _stream())
    _capi.check(code, "based_gated_conv_prefill")
    return out


def gated_conv_step(u: torch.Tensor, state: torch.Tensor, weight: torch.Tensor,
                    bias: Optional[torch.Tensor] = None, *, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One decode step of :func:`gated_conv_prefill`; ``state [B, di, k]`` is updated IN PLACE
    (convolution.py:104-107).  ``u [B, 2*di]`` or ``[B, 1, 2*di]``; returns ``[B, di]``."""
    _need_cuda(u, state, weight, bias)
    if u.dim() == 3:
        u = u[:, 0]
    B, two_di = u.shape
    di = two_di // 2
    weight = weight.reshape(weight.shape[0], -1).contiguous()
    k = weight.shape[1]
    _inner_contig(u, "u")
    if bias is not None:
        bias = bias.to(weight.dtype).contiguous()
    if state.shape != (B, di, k) or state.dtype != u.dtype or not state.is_contiguous():
        raise ValueError("state must be a contiguous [B, di, k] tensor of u's dtype")
    if out is None:
        out = torch.empty(B, di, dtype=u.dtype, device=u.device)
    if B == 0:
        return out
    u1, u2 = u[:, :di], u[:, di:]
    with torch.cuda.device(u.device):
        code = _capi.lib().based_gated_conv_step(
            u1.data_ptr(), u2.data_ptr(), out.data_ptr(), state.data_ptr(), weight.data_ptr(),
            bias.data_ptr() if bias is not None else None, B, di, k, u1.stride(0), u2.stride(0), out.stride(0),
            _dt(u.dtype), _dt(weight.dtype), _stream())
    _capi.check(code, "based_gated_conv_step")
    return out


def add_rmsnorm(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None,
                residual: Optional[torch.Tensor] = None, *, eps: float = 1e-6, prenorm: bool = False,
                residual_in_fp32: bool = False, round_input: bool = False):
    """``z = x + residual``; ``out = rmsnorm(z) * weight (+ bias)`` in one pass; with ``prenorm`` returns
    ``(out, z)`` like rms_norm_fn (layer_norm.py:926-953).  ``z`` is fp32 when ``residual_in_fp32`` or
    when ``residual`` already is, else x's dtype.  ``round_input`` rounds ``z`` to x's dtype before the
    norm (the unfused ``norm(residual.to(weight.dtype))`` of block.py:134-137).  x ``[..., D]``."""
    _need_cuda(x, weight, bias, residual)
    D = x.shape[-1]
    x2 = x.reshape(-1, D)
    _inner_contig(x2, "x")
    M = x2.shape[0]
    res2 = None
    if residual is not None:
        if residual.shape != x.shape:
            raise ValueError("residual must have x's shape")
        res2 = residual.reshape(-1, D)
        _inner_contig(res2, "residual")
    res_dtype = torch.float32 if (residual_in_fp32 or (residual is not None and residual.dtype == torch.float32)) else x.dtype
    if res2 is not None and res2.dtype != res_dtype:
        res2 = res2.to(res_dtype)
    weight = weight.contiguous()
    if bias is not None:
        bias = bias.to(weight.dtype).contiguous()
    out = torch.empty(M, D, dtype=x.dtype, device=x.device)
    res_out = torch.empty(M, D, dtype=res_dtype, device=x.device) if prenorm else None
    if M > 0:
        with torch.cuda.device(x.device):
            code = _capi.lib().based_add_rmsnorm(
                x2.data_ptr(), res2.data_ptr() if res2 is not None else None, weight.data_ptr(),
                bias.data_ptr() if bias is not None else None, out.data_ptr(),
                res_out.data_ptr() if res_out is not None else None, M, D, x2.stride(0),
                res2.stride(0) if res2 is not None else 0, out.stride(0), res_out.stride(0) if res_out is not None else 0,
                float(eps), _dt(x.dtype), _dt(res_dtype), _dt(weight.dtype), int(round_input), _stream())
        _capi.check(code, "based_add_rmsnorm")
    out = out.reshape(x.shape)
    return (out, res_out.reshape(x.shape)) if prenorm else out


_ACTS = {"silu": 0, "swiglu": 0, "sigmoid": 1, "glu": 1}


def gated_act(y: torch.Tensor, activation: str = "silu", out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``first_half * act(second_half)`` over the last dim of ``y [..., 2F]`` (mlp.py:141-154).  ``out``: a ``[..., F]``
    tensor or column slice to write (rows one constant stride apart)."""
    _need_cuda(y, out)
    F2 = y.shape[-1]
    F = F2 // 2
    y2 = y.reshape(-1, F2)
    _inner_contig(y2, "y")
    M = y2.shape[0]
    out = torch.empty(M, F, dtype=y.dtype, device=y.device) if out is None else _rows(out, F)
    if M > 0:
        a, g = y2[:, :F], y2[:, F:]
        with torch.cuda.device(y.device):
            code = _capi.lib().based_gated_act(a.data_ptr(), g.data_ptr(), out.data_ptr(), M, F, a.stride(0),
                                               g.stride(0), out.stride(0), _ACTS[activation], _dt(y.dtype), _stream())
        _capi.check(code, "based_gated_act")
    return out.reshape(*y.shape[:-1], F)


DECODE_LINEAR_MAX_ROWS = 64  # beyond this the library GEMM is the better tool
# Which decode-step products the mixers and the MLP hand to decode_linear instead of cuBLAS (+ a separate
# elementwise launch).  Measured on the 360M model at batch 16 with the weights streaming from HBM
# (ms per decode step): none 1.146, gated 1.089, gated + conv 1.145, all three 1.329 -- only fc1 + SwiGLU pays.
DECODE_LINEAR_USE = {"plain": False, "gated": True, "conv": False}


def decode_linear(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None, *,
                  epilogue: str = "plain", activation: str = "silu", conv_state: Optional[torch.Tensor] = None,
                  conv_weight: Optional[torch.Tensor] = None, conv_bias: Optional[torch.Tensor] = None,
                  out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``x W^T (+ bias)`` for the few rows of a decode step (bf16), with a fused epilogue:
    ``"plain"``; ``"gated"`` -> ``first_half * act(second_half)`` (mlp.py:146-154); ``"conv"`` -> the BaseConv
    decode step on the first half (``conv_state [M, N/2, k]`` updated in place), silu, gate by the second half
    (convolution.py:88-109, :205-211).  x ``[..., K]``; returns ``[..., N]`` or ``[..., N/2]``."""
    _need_cuda(x, weight, bias, conv_state, conv_weight, conv_bias)
    if x.dtype != torch.bfloat16 or weight.dtype != torch.bfloat16:
        raise TypeError("decode_linear takes bfloat16 activations and weights")
    K = x.shape[-1]
    x2 = x.reshape(-1, K)
    _inner_contig(x2, "x")
    M, N = x2.shape[0], weight.shape[0]
    if weight.shape[1] != K or not weight.is_contiguous():
        raise ValueError("weight must be a contiguous [N, K] tensor")
    epi = {"plain": 0, "gated": 1, "conv": 2}[epilogue]
    n_out = N if epi == 0 else N // 2
    out = torch.empty(M, n_out, dtype=torch.bfloat16, device=x.device) if out is None else _rows(out, n_out)
    if bias is not None:
        bias = bias.to(torch.bfloat16).contiguous()
    ck, cw_dt = 0, BASED_BF16
    if epi == 2:
        conv_weight = conv_weight.reshape(conv_weight.shape[0], -1).contiguous()
        ck, cw_dt = conv_weight.shape[1], _dt(conv_weight.dtype)
        if conv_bias is not None:
            conv_bias = conv_bias.to(conv_weight.dtype).contiguous()
        if conv_state.shape != (M, n_out, ck) or conv_state.dtype != torch.bfloat16 or not conv_state.is_contiguous():
            raise ValueError("conv_state must be a contiguous bfloat16 [M, N/2, k] tensor")
    if M > 0:
        with torch.cuda.device(x.device):
            code = _capi.lib().based_decode_linear(
                x2.data_ptr(), weight.data_ptr(), bias.data_ptr() if bias is not None else None, out.data_ptr(),
                M, N, K, x2.stride(0), out.stride(0), epi, _ACTS[activation],
                conv_state.data_ptr() if epi == 2 else None, conv_weight.data_ptr() if epi == 2 else None,
                conv_bias.data_ptr() if (epi == 2 and conv_bias is not None) else None, ck, cw_dt, _stream())
        _capi.check(code, "based_decode_linear")
    return out.reshape(*x.shape[:-1], n_out)


def _decode_rows(x: torch.Tensor, weight: torch.Tensor) -> bool:
    """True when ``x W^T`` is a decode-step product the library's own kernel should run."""
    rows = x.numel() // x.shape[-1] if x.numel() else 0
    return (x.is_cuda and x.dtype == torch.bfloat16 and weight.dtype == torch.bfloat16 and 0 < rows <= DECODE_LINEAR_MAX_ROWS
            and x.shape[-1] % 32 == 0 and weight.shape[0] % 8 == 0 and weight.is_contiguous() and x.stride(-1) == 1
            and not torch.is_grad_enabled())


def linear(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``nn.functional.linear`` for the mixers: the decode-step kernel for a few bf16 rows, cuBLAS otherwise."""
    if DECODE_LINEAR_USE["plain"] and _decode_rows(x, weight):
        return decode_linear(x, weight, bias)
    return torch.nn.functional.linear(x, weight, bias)


def rotary_qkv_cache_(qkv: torch.Tensor, rotary_cos: torch.Tensor, rotary_sin: torch.Tensor,
                      kv_cache: torch.Tensor) -> torch.Tensor:
    """Prompt pass of the sliding-window mixer: whole-head RoPE on q and k of packed ``qkv [B, L, 3, H, hd]`` in
    place, and rotated k plus v written to ``kv_cache[:B, :L]`` (``[*, max_seqlen, 2, H, hd]``) in the same launch
    (slide_attention.py:553-556 and :255-281).  bf16 only; returns ``qkv``."""
    _need_cuda(qkv, rotary_cos, rotary_sin, kv_cache)
    B, L, three, H, hd = qkv.shape
    if three != 3 or qkv.dtype != torch.bfloat16 or kv_cache.dtype != torch.bfloat16:
        raise TypeError("rotary_qkv_cache_ takes a bfloat16 [B, L, 3, H, hd] tensor and a bfloat16 cache")
    _inner_contig(qkv, "qkv")
    if rotary_cos.shape[-1] * 2 != hd or rotary_cos.shape[0] < L or rotary_cos.dtype != torch.bfloat16:
        raise ValueError("rotary tables must be bfloat16 [>= L, hd/2]")
    if not (rotary_cos.is_contiguous() and rotary_sin.is_contiguous()):
        raise ValueError("rotary tables must be contiguous")
    if (kv_cache.shape[0] < B or kv_cache.shape[1] < L or tuple(kv_cache.shape[2:]) != (2, H, hd)
            or kv_cache.stride()[2:] != (H * hd, hd, 1)):
        raise ValueError("kv_cache must be [>= B, >= L, 2, H, hd] with the last three dims contiguous")
    if qkv.numel() == 0:
        return qkv
    with torch.cuda.device(qkv.device):
        code = _capi.lib().based_rotary_qkv_cache(
            qkv.data_ptr(), B, L, H, hd, _capi.strides(*qkv.stride()[:4]), rotary_cos.data_ptr(), rotary_sin.data_ptr(),
            kv_cache.data_ptr(), _capi.strides(*kv_cache.stride()[:2]), _stream())
    _capi.check(code, "based_rotary_qkv_cache")
    return qkv


def tp_outproj_workspace_bytes(world: int, max_rows: int, n_out: int) -> int:
    """Size of one rank's receive workspace for :func:`tp_outproj_allreduce`."""
    n = _capi.lib().based_tp_outproj_workspace_bytes(int(world), int(max_rows), int(n_out))
    if n == 0:
        raise ValueError("tp_outproj: world must be 1..8, max_rows >= 1 and n_out a multiple of 8")
    return n


def tp_outproj_workspace_init_(ws: torch.Tensor) -> torch.Tensor:
    """Prepare a workspace (zero flags, call counter = 1).  Once, by its owner, before any rank's first call."""
    _need_cuda(ws)
    with torch.cuda.device(ws.device):
        _capi.check(_capi.lib().based_tp_outproj_workspace_init(ws.data_ptr(), ws.numel() * ws.element_size(), _stream()),
                    "based_tp_outproj_workspace_init")
    return ws


def tp_outproj_allreduce(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor], workspace_ptrs, max_rows: int,
                         rank: int, world: int, *, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Row-parallel ``x W^T`` summed over the tensor-parallel ranks (+ bias), one kernel per rank
    (based/ops/fused_dense.py:239-246 as GEMM + all-reduce in one launch).  ``x [..., K_local]`` bf16 with at most
    ``max_rows`` rows, ``weight [N, K_local]`` bf16 contiguous; ``workspace_ptrs`` the device addresses of every rank's
    workspace as mapped in this process.  A collective: every rank calls it with the same shapes."""
    _need_cuda(x, weight, bias)
    if x.dtype != torch.bfloat16 or weight.dtype != torch.bfloat16:
        raise TypeError("tp_outproj_allreduce takes bfloat16 activations and weights")
    K = x.shape[-1]
    x2 = x.reshape(-1, K)
    _inner_contig(x2, "x")
    M, N = x2.shape[0], weight.shape[0]
    if weight.shape[1] != K or not weight.is_contiguous():
        raise ValueError("weight must be a contiguous [N, K] tensor")
    if not 0 < M <= max_rows:
        raise ValueError(f"tp_outproj_allreduce: {M} rows, workspace built for at most {max_rows}")
    if len(workspace_ptrs) != world:
        raise ValueError("one workspace address per rank is needed")
    if bias is not None:
        bias = bias.to(torch.bfloat16).contiguous()
    if out is None:
        out = torch.empty(M, N, dtype=torch.bfloat16, device=x.device)
    o2 = out.reshape(-1, N)
    with torch.cuda.device(x.device):
        code = _capi.lib().based_tp_outproj_allreduce(
            x2.data_ptr(), weight.data_ptr(), bias.data_ptr() if bias is not None else None, o2.data_ptr(), M, N, K,
            x2.stride(0), o2.stride(0), _capi.pointers(workspace_ptrs), int(max_rows), int(rank), int(world), _stream())
    _capi.check(code, "based_tp_outproj_allreduce")
    return out.reshape(*x.shape[:-1], N)


def tp_outproj_allreduce_emulated(xs, weights, bias, workspaces, max_rows: int):
    """All ranks of :func:`tp_outproj_allreduce` inside one cooperative launch on one GPU: ``xs[r] [M, K]``,
    ``weights[r] [N, K]``, ``workspaces[r]`` (prepared uint8 tensors), all on the same device.  Returns the list of the
    ranks' outputs.  For checking the exchange protocol with a single GPU."""
    world = len(xs)
    _need_cuda(*xs, *weights, bias, *workspaces)
    M, K = xs[0].shape
    N = weights[0].shape[0]
    outs = [torch.empty(M, N, dtype=torch.bfloat16, device=xs[0].device) for _ in range(world)]
    if bias is not None:
        bias = bias.to(torch.bfloat16).contiguous()
    with torch.cuda.device(xs[0].device):
        code = _capi.lib().based_tp_outproj_allreduce_emulated(
            _capi.pointers([t.data_ptr() for t in xs]), _capi.pointers([t.data_ptr() for t in weights]),
            bias.data_ptr() if bias is not None else None, _capi.pointers([t.data_ptr() for t in outs]), M, N, K,
            xs[0].stride(0), outs[0].stride(0), _capi.pointers([t.data_ptr() for t in workspaces]), int(max_rows), world,
            _stream())
    _capi.check(code, "based_tp_outproj_allreduce_emulated")
    return outs


# --------------------------------------------------------------------------- stateful mixers of hybrid stacks
# ``pos``: position of a call's first token, an int or an int32 CUDA tensor with one entry per batch row.  A sequence
# that starts (position 0) reads no state, so state tensors need no clearing between sequences.

def linear_f32(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``x W^T`` with an fp32 result (fp32 accumulation of the operands' products, not rounded to their dtype)."""
    _need_cuda(x, weight)
    if x.dtype == torch.float32:
        return torch.nn.functional.linear(x, weight)
    y = torch.mm(x.reshape(-1, x.shape[-1]), weight.t(), out_dtype=torch.float32)
    return y.view(*x.shape[:-1], weight.shape[0])


def stream_norm(residual: torch.Tensor, w1: torch.Tensor, w2: Optional[torch.Tensor] = None, *,
                branch: Optional[torch.Tensor] = None, mult: float = 1.0, tokens: Optional[torch.Tensor] = None,
                table: Optional[torch.Tensor] = None, table_norm: Optional[torch.Tensor] = None, eps: float = 1e-6):
    """The norm step of a parallel block: the fp32 stream ``residual [..., D]`` becomes ``residual + mult * branch`` (or,
    with ``tokens``, ``rmsnorm(table[token]) * table_norm``) IN PLACE; returns its RMSNorm scaled by ``w1`` and by ``w2``
    (None without ``w2``), in the weights' dtype."""
    _need_cuda(residual, w1, w2, branch, tokens, table, table_norm)
    D = residual.shape[-1]
    if residual.dtype != torch.float32 or not residual.is_contiguous():
        raise TypeError("residual must be a contiguous float32 tensor")
    M = residual.numel() // D if D else 0
    out1 = torch.empty(residual.shape, dtype=w1.dtype, device=residual.device)
    out2 = torch.empty_like(out1) if w2 is not None else None
    sb = 0
    if branch is not None:
        branch = branch.reshape(-1, D)
        _inner_contig(branch, "branch")
        sb = branch.stride(0)
    V = 0
    if tokens is not None:
        if tokens.dtype != torch.int64 or tokens.numel() != M:
            raise TypeError("tokens must be int64, one per row")
        tokens, V = tokens.contiguous(), table.shape[0]
    for t in (w1, w2, branch, table, table_norm):
        if t is not None and (t.dtype != w1.dtype or (t is not branch and not t.is_contiguous())):
            raise TypeError("weights, table and branch must share a dtype and be contiguous")
    if M > 0:
        with torch.cuda.device(residual.device):
            code = _capi.lib().based_stream_norm(
                _ptr(tokens), _ptr(table), _ptr(table_norm), V, _ptr(branch), sb, float(mult), residual.data_ptr(),
                w1.data_ptr(), _ptr(w2), out1.data_ptr(), _ptr(out2), M, D, float(eps), _dt(w1.dtype), _stream())
        _capi.check(code, "based_stream_norm")
    return out1, out2


def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """``x / sqrt(mean(x^2) + eps) * weight`` over the last dim of ``x [..., D]`` (a column slice is fine), contiguous."""
    _need_cuda(x, weight)
    D = x.shape[-1]
    x2 = flat_rows(x) if x.dim() > 1 else x.view(1, D)
    _inner_contig(x2, "x")
    out = torch.empty(x.shape, dtype=x.dtype, device=x.device)
    if weight.dtype != x.dtype:
        raise TypeError("weight must be in x's dtype")
    if out.numel() > 0:
        with torch.cuda.device(x.device):
            code = _capi.lib().based_rmsnorm(x2.data_ptr(), weight.data_ptr(), out.data_ptr(), x2.shape[0], D, x2.stride(0), D,
                                             float(eps), _dt(x.dtype), _stream())
        _capi.check(code, "based_rmsnorm")
    return out


def short_conv(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None, *,
               ring: Optional[torch.Tensor] = None, pos=0, silu: bool = False) -> torch.Tensor:
    """Depthwise causal convolution ``x [B, L, C]`` by ``weight [C, taps]`` for tokens that start at ``pos``; ``ring
    [B, taps, C]`` carries earlier inputs (position p in slot p mod taps) and is updated.  Contiguous ``[B, L, C]``."""
    _need_cuda(x, weight, bias, ring)
    B, L, C = x.shape
    taps = weight.shape[1]
    _inner_contig(x, "x")
    if weight.shape[0] != C or weight.dtype != x.dtype or not weight.is_contiguous() or (bias is not None and bias.dtype != x.dtype):
        raise ValueError("weight must be a contiguous [C, taps] tensor in x's dtype (bias [C] too)")
    if ring is not None and (ring.shape[0] < B or ring.shape[1:] != (taps, C) or ring.dtype != x.dtype or not ring.is_contiguous()):
        raise ValueError("ring must be a contiguous [>= B, taps, C] tensor in x's dtype")
    y = torch.empty(B, L, C, dtype=x.dtype, device=x.device)
    if y.numel() == 0:
        return y
    off, scalar = _position(pos, x)
    with torch.cuda.device(x.device):
        code = _capi.lib().based_short_conv(x.data_ptr(), y.data_ptr(), _ptr(ring), weight.data_ptr(), _ptr(bias), B, L, C, taps,
                                            _capi.strides(*x.stride()[:2]), _capi.strides(*y.stride()[:2]), off, scalar,
                                            int(silu), _dt(x.dtype), _stream())
    _capi.check(code, "based_short_conv")
    return y


def latent_prepare_(q: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, dim: int, *, z: Optional[torch.Tensor] = None,
                    norm_weight: Optional[torch.Tensor] = None, cache: Optional[torch.Tensor] = None, kv_rank: int = 1,
                    pos=0, eps: float = 1e-6) -> torch.Tensor:
    """Rotate the last dims of every head of ``q [B, L, H, dim + rot]`` IN PLACE and, with ``z [B, L, kv_rank + rot]``,
    append the normed latent and the rotated shared key to ``cache [B, max_len, kv_rank + rot]``.  fp32 tables."""
    _need_cuda(q, cos, sin, z, norm_weight, cache)
    B, L, H, dq = q.shape
    rd = dq - dim
    if not q.is_contiguous() or cos.dtype != torch.float32 or cos.shape[1] * 2 != rd or not (cos.is_contiguous() and sin.is_contiguous()):
        raise ValueError("q must be contiguous and the tables float32 [positions, rot / 2]")
    zs = cs = None
    max_len = 2147483647
    if z is not None:
        _inner_contig(z, "z")
        if z.dtype != q.dtype or cache.dtype != q.dtype or cache.shape[0] < B or cache.shape[2] != kv_rank + rd or cache.stride(2) != 1:
            raise ValueError("cache must be [>= B, max_len, kv_rank + rot] in the inputs' dtype")
        zs, cs, max_len = _capi.strides(*z.stride()[:2]), _capi.strides(*cache.stride()[:2]), cache.shape[1]
    if q.numel() == 0:
        return q
    off, scalar = _position(pos, q)
    with torch.cuda.device(q.device):
        code = _capi.lib().based_latent_prepare(_ptr(z), _ptr(norm_weight), _ptr(cache), q.data_ptr(), cos.data_ptr(), sin.data_ptr(),
                                                cos.shape[0], B, L, H, int(kv_rank), rd, int(dim), max_len, zs, cs,
                                                _capi.strides(*q.stride()[:2]), off, scalar, float(eps), _dt(q.dtype), _stream())
    _capi.check(code, "based_latent_prepare")
    return q


def split_key_attention(q1, q2, k1, k2, v, scale: float, *, gate: Optional[torch.Tensor] = None, pos=0,
                        out: torch.Tensor) -> torch.Tensor:
    """Causal attention with score ``(q1 . k1 + q2 . k2) * scale`` on CUDA cores (fp32 arithmetic): q1, q2 ``[B, L, H, .]``,
    k1, k2, v ``[B, T, H, .]`` (expand the head dim to share keys), ``gate [B, L, H]`` pre-sigmoid, ``out [B, L, H, dv]``."""
    _need_cuda(q1, q2, k1, k2, v, gate, out)
    B, L, H, d1 = q1.shape
    for t, n in ((q1, "q1"), (q2, "q2"), (k1, "k1"), (k2, "k2"), (v, "v"), (out, "out")):
        _inner_contig(t, n)
        if t.dtype != q1.dtype:
            raise TypeError("all tensors must share a dtype")
    off, scalar = _position(pos, q1)
    if off is None and k1.shape[1] < scalar + L:
        raise ValueError("fewer keys than the last query sees")
    gs = _capi.strides(*gate.stride()[:2]) if gate is not None else None
    if gate is not None:
        _inner_contig(gate, "gate")
    if out.numel() == 0:
        return out
    with torch.cuda.device(q1.device):
        code = _capi.lib().based_split_key_attention(
            q1.data_ptr(), q2.data_ptr(), k1.data_ptr(), k2.data_ptr(), v.data_ptr(), _ptr(gate), out.data_ptr(), B, L, H, d1,
            q2.shape[-1], v.shape[-1], _capi.strides(*q1.stride()[:3]), _capi.strides(*q2.stride()[:3]),
            _capi.strides(*k1.stride()[:3]), _capi.strides(*k2.stride()[:3]), _capi.strides(*v.stride()[:3]),
            _capi.strides(*out.stride()[:3]), gs, off, scalar, float(scale), _dt(q1.dtype), _stream())
    _capi.check(code, "based_split_key_attention")
    return out


def latent_prefill(q1, q2, k1, k2, v, scale: float, *, gate: Optional[torch.Tensor] = None, pos: int = 0,
                   out: torch.Tensor, impl: str = "auto") -> torch.Tensor:
    """Expanded latent attention over a prompt or portion: q1, q2 ``[B, L, H, .]`` at positions ``pos ..``, per-head keys
    k1 and values v ``[B, T, H, .]``, shared key part k2 ``[B, T, d2]``, ``gate [B, L, H]`` pre-sigmoid -> ``out [B, L, H, dv]``."""
    _need_cuda(q1, q2, k1, k2, v, gate, out)
    B, L, H, d1 = q1.shape
    for t, n in ((q1, "q1"), (q2, "q2"), (k1, "k1"), (k2, "k2"), (v, "v"), (out, "out")):
        _inner_contig(t, n)
        if t.dtype != q1.dtype:
            raise TypeError("all tensors must share a dtype")
    if gate is not None:
        _inner_contig(gate, "gate")
    if out.numel() == 0:
        return out
    with torch.cuda.device(q1.device):
        code = _capi.lib().based_latent_prefill(
            q1.data_ptr(), q2.data_ptr(), k1.data_ptr(), k2.data_ptr(), v.data_ptr(), _ptr(gate), out.data_ptr(), B, L, k1.shape[1],
            H, d1, q2.shape[-1], v.shape[-1], _capi.strides(*q1.stride()[:3]), _capi.strides(*q2.stride()[:3]),
            _capi.strides(*k1.stride()[:3]), _capi.strides(*k2.stride()[:2]), _capi.strides(*v.stride()[:3]),
            _capi.strides(*out.stride()[:3]), _capi.strides(*gate.stride()[:2]) if gate is not None else None, int(pos),
            float(scale), _dt(q1.dtype), _IMPLS[impl], _stream())
    _capi.check(code, "based_latent_prefill")
    return out


def latent_decode(qa, qr, cache, scale: float, *, gate: Optional[torch.Tensor] = None, pos=0,
                  out: torch.Tensor) -> torch.Tensor:
    """Absorbed latent attention for a few query rows: qa ``[B, L, H, kv_rank]``, qr ``[B, L, H, rot]``, ``cache [B, max_len,
    kv_rank + rot]`` -> gated context ``out [B, L, H, kv_rank]``."""
    _need_cuda(qa, qr, cache, gate, out)
    B, L, H, r = qa.shape
    rd = qr.shape[-1]
    for t, n in ((qa, "qa"), (qr, "qr"), (cache, "cache"), (out, "out")):
        _inner_contig(t, n)
        if t.dtype != qa.dtype:
            raise TypeError("all tensors must share a dtype")
    if cache.shape[0] < B or cache.shape[2] != r + rd:
        raise ValueError("cache must be [>= B, max_len, kv_rank + rot]")
    if gate is not None:
        _inner_contig(gate, "gate")
    if out.numel() == 0:
        return out
    off, scalar = _position(pos, qa)
    with torch.cuda.device(qa.device):
        lib = _capi.lib()
        need = lib.based_latent_decode_scratch_bytes(B, L, H, r, cache.shape[1])
        scratch = torch.empty(need, dtype=torch.uint8, device=qa.device) if need else None
        code = lib.based_latent_decode(
            qa.data_ptr(), qr.data_ptr(), cache.data_ptr(), _ptr(gate), out.data_ptr(), _ptr(scratch), need, B, L, H, r, rd,
            cache.shape[1], _capi.strides(*qa.stride()[:3]), _capi.strides(*qr.stride()[:3]), _capi.strides(*cache.stride()[:2]),
            _capi.strides(*out.stride()[:3]), _capi.strides(*gate.stride()[:2]) if gate is not None else None, off, scalar,
            float(scale), _dt(qa.dtype), _stream())
    _capi.check(code, "based_latent_decode")
    return out


def _check_delta(state, B, H, d, dv, *params):
    if state.shape[0] < B or state.shape[1:] != (H, d, dv) or state.dtype != torch.float32 or not state.is_contiguous():
        raise ValueError("state must be a contiguous float32 [>= B, H, d, dv] tensor")
    for t in params:
        if t.dtype != torch.float32 or t.stride(-1) != 1:
            raise TypeError("decay and step-size inputs must be float32")


def delta_prefill(q, k, v, z, a, b, A_log, dt_bias, norm_weight, state, *, pos=0, eps: float = 1e-6,
                  out: torch.Tensor, impl: str = "auto") -> torch.Tensor:
    """Gated delta rule over ``L`` tokens: q, k ``[B, L, Hk, d]``, v, z ``[B, L, H, dv]`` (token-strided views, heads
    contiguous), a, b ``[B, L, H]`` fp32 pre-activations, ``state [B, H, d, dv]`` fp32 updated IN PLACE; ``out [B, L, H * dv]``."""
    _need_cuda(q, k, v, z, a, b, A_log, dt_bias, norm_weight, state, out)
    B, L, Hk, d = q.shape
    H, dv = v.shape[2:]
    _check_delta(state, B, H, d, dv, a, b, A_log, dt_bias)
    for t, w in ((q, d), (k, d), (v, dv), (z, dv)):
        if t.stride(3) != 1 or (t.shape[2] > 1 and t.stride(2) != w) or t.dtype != q.dtype:
            raise ValueError("q, k, v, z: heads must be contiguous inside a token and share a dtype")
    if a.stride()[:2] != b.stride()[:2]:
        raise ValueError("a and b must have the same strides")
    _inner_contig(out, "out")
    off, scalar = _position(pos, q)
    if out.numel() == 0:
        return out
    with torch.cuda.device(q.device):
        need = _capi.lib().based_delta_prefill_scratch_bytes(B, L, H, d, dv) if q.dtype == torch.bfloat16 and impl != "simt" else 0
        scratch = torch.empty(need, dtype=torch.uint8, device=q.device) if need else None
        code = _capi.lib().based_delta_prefill(
            q.data_ptr(), k.data_ptr(), v.data_ptr(), z.data_ptr(), a.data_ptr(), b.data_ptr(), A_log.data_ptr(), dt_bias.data_ptr(),
            norm_weight.data_ptr(), state.data_ptr(), out.data_ptr(), B, L, H, Hk, d, dv, _capi.strides(*q.stride()[:2]),
            _capi.strides(*k.stride()[:2]), _capi.strides(*v.stride()[:2]), _capi.strides(*z.stride()[:2]),
            _capi.strides(*a.stride()[:2]), _capi.strides(*out.stride()[:2]), off, scalar, float(eps), _dt(q.dtype), _IMPLS[impl],
            _ptr(scratch), need, _stream())
    _capi.check(code, "based_delta_prefill")
    return out


def delta_step(x, conv_weight, ring, a, b, A_log, dt_bias, norm_weight, state, kv_heads: int, *, pos, eps: float = 1e-6,
               out: torch.Tensor) -> bool:
    """One token per row in one launch: packed projection ``x [B, q | k | v | z]``, ``ring [B, taps, C]`` and ``state
    [B, H, d, dv]`` updated IN PLACE, ``out [B, H * dv]``.  Returns False, nothing launched, for sizes it does not take."""
    _need_cuda(x, conv_weight, ring, a, b, A_log, dt_bias, norm_weight, state, out)
    B, (_, H, d, dv) = x.shape[0], state.shape
    _check_delta(state, B, H, d, dv, a, b, A_log, dt_bias)
    C, taps = conv_weight.shape
    if C != 2 * kv_heads * d + H * dv or x.shape[1] < C + H * dv or x.stride(1) != 1 or out.stride(1) != 1 or a.stride(0) != b.stride(0):
        raise ValueError("x must be [B, >= 2 kv_heads d + 2 H dv] and conv_weight [2 kv_heads d + H dv, taps]")
    if ring.shape[0] < B or ring.shape[1:] != (taps, C) or ring.dtype != x.dtype or not ring.is_contiguous() or not conv_weight.is_contiguous():
        raise ValueError("ring must be a contiguous [>= B, taps, C] tensor in x's dtype")
    off, scalar = _position(pos, x)
    if B == 0:
        return True
    with torch.cuda.device(x.device):
        code = _capi.lib().based_delta_step(
            x.data_ptr(), conv_weight.data_ptr(), ring.data_ptr(), a.data_ptr(), b.data_ptr(), A_log.data_ptr(), dt_bias.data_ptr(),
            norm_weight.data_ptr(), state.data_ptr(), out.data_ptr(), B, H, int(kv_heads), d, dv, taps, x.stride(0), a.stride(0),
            out.stride(0), off, scalar, float(eps), _dt(x.dtype), _stream())
    if code == _capi.ERR_IMPL:
        return False
    _capi.check(code, "based_delta_step")
    return True


def block_gates(u: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """Block-diagonal gate products with an fp32 result: ``u [B, L, blocks * n]`` by ``weight [blocks, 2, n, n]`` (r and i
    matrices, stored [out, in]) -> ``[blocks, B * L, 2 n]``."""
    _need_cuda(u, weight)
    nb, _, n, _ = weight.shape
    x, w = u.reshape(-1, nb, n).transpose(0, 1), weight.view(nb, 2 * n, n).transpose(1, 2)
    if u.dtype == torch.float32:
        return torch.bmm(x, w)
    return torch.bmm(x, w, out_dtype=torch.float32)


def rglru(u, y, gates, r_bias, i_bias, lam, state, *, pos=0, out: torch.Tensor) -> torch.Tensor:
    """Real-gated linear recurrent unit: u, y ``[B, L, W]``, ``gates [blocks, B * L, 2 n]`` fp32 (r half, i half),
    ``lam [W]`` fp32, ``state [B, W]`` fp32 updated IN PLACE; ``out [B, L, W] = S * gelu_tanh(y)``."""
    _need_cuda(u, y, gates, r_bias, i_bias, lam, state, out)
    B, L, W = u.shape
    nb, rows, n2 = gates.shape
    if rows != B * L or nb * n2 != 2 * W or gates.dtype != torch.float32 or gates.stride(2) != 1:
        raise ValueError("gates must be float32 [blocks, B * L, 2 * W / blocks]")
    if state.shape[0] < B or state.shape[1] != W or state.dtype != torch.float32 or lam.dtype != torch.float32 or not state.is_contiguous():
        raise ValueError("state must be a contiguous float32 [>= B, W] tensor and lam float32")
    for t, n in ((u, "u"), (y, "y"), (out, "out")):
        _inner_contig(t, n)
    off, scalar = _position(pos, u)
    if out.numel() == 0:
        return out
    with torch.cuda.device(u.device):
        code = _capi.lib().based_rglru(
            u.data_ptr(), y.data_ptr(), gates.data_ptr(), r_bias.data_ptr(), i_bias.data_ptr(), lam.data_ptr(), state.data_ptr(),
            out.data_ptr(), B, L, W, n2 // 2, _capi.strides(*u.stride()[:2]), _capi.strides(*y.stride()[:2]),
            _capi.strides(*out.stride()[:2]), _capi.strides(gates.stride(0), gates.stride(1)), off, scalar, _dt(u.dtype), _stream())
    _capi.check(code, "based_rglru")
    return out


# tokens from which the one-pass kernel is used; below it, the gate products and the recurrence are two launches
RGLRU_FUSED_MIN_TOKENS = 8


def rglru_gated(u, y, gate_weight, r_bias, i_bias, lam, state, *, pos=0, out: torch.Tensor) -> torch.Tensor:
    """The recurrent unit with its gate products (``gate_weight`` as in :func:`block_gates`): one pass on the tensor cores
    for bf16 prompts and portions, else :func:`block_gates` and :func:`rglru`."""
    _need_cuda(u, y, gate_weight, r_bias, i_bias, lam, state, out)
    B, L, W = u.shape
    nb, _, n, _ = gate_weight.shape
    if u.dtype == torch.bfloat16 and L >= RGLRU_FUSED_MIN_TOKENS and B > 0:
        if (nb * n != W or not gate_weight.is_contiguous() or gate_weight.dtype != u.dtype or lam.dtype != torch.float32
                or state.dtype != torch.float32 or state.shape[0] < B or state.shape[1] != W or not state.is_contiguous()):
            raise ValueError("gate_weight must be [blocks, 2, n, n] in u's dtype, state [>= B, W] and lam float32, contiguous")
        for t, name in ((u, "u"), (y, "y"), (out, "out")):
            _inner_contig(t, name)
        off, scalar = _position(pos, u)
        with torch.cuda.device(u.device):
            code = _capi.lib().based_rglru_gated(
                u.data_ptr(), y.data_ptr(), gate_weight.data_ptr(), r_bias.data_ptr(), i_bias.data_ptr(), lam.data_ptr(),
                state.data_ptr(), out.data_ptr(), B, L, W, n, _capi.strides(*u.stride()[:2]), _capi.strides(*y.stride()[:2]),
                _capi.strides(*out.stride()[:2]), off, scalar, _dt(u.dtype), _stream())
        if code != _capi.ERR_IMPL:
            _capi.check(code, "based_rglru_gated")
            return out
    return rglru(u, y, block_gates(u, gate_weight), r_bias, i_bias, lam, state, pos=pos, out=out)


# --------------------------------------------------------------------------- post-norm stacks

def _strides_bl(t):
    return _capi.strides(*t.stride()[:2])


def _same_dtype(like, **tensors):
    for name, t in tensors.items():
        if t is not None and (t.dtype != like.dtype or t.stride(-1) != 1):
            raise TypeError(f"{name} must be in the inputs' dtype with an innermost stride of 1")


def stream_embed(residual: torch.Tensor, tokens: torch.Tensor, table: torch.Tensor, scale: float, pos_table: torch.Tensor,
                 pos=0) -> torch.Tensor:
    """Start of a stream: the fp32 ``residual [B, L, D]`` becomes ``table[token] * scale + pos_table[position]`` IN PLACE;
    returns it in the table's dtype (fp32: the stream itself)."""
    _need_cuda(residual, tokens, table, pos_table)
    B, L, D = residual.shape
    if residual.dtype != torch.float32 or not residual.is_contiguous():
        raise TypeError("residual must be a contiguous float32 tensor")
    if tokens.dtype != torch.int64 or tokens.shape != (B, L):
        raise TypeError("tokens must be int64 [B, L]")
    if table.dtype != pos_table.dtype or not (table.is_contiguous() and pos_table.is_contiguous()) or table.shape[1] != D or pos_table.shape[1] != D:
        raise ValueError("table and pos_table must be contiguous [rows, D] of one dtype")
    out = residual if table.dtype == torch.float32 else torch.empty(B, L, D, dtype=table.dtype, device=residual.device)
    off, scalar = _position(pos, residual)
    if residual.numel() > 0:
        tokens = tokens.contiguous()
        with torch.cuda.device(residual.device):
            code = _capi.lib().based_stream_embed(
                tokens.data_ptr(), table.data_ptr(), table.shape[0], float(scale), pos_table.data_ptr(), pos_table.shape[0],
                residual.data_ptr(), None if out is residual else out.data_ptr(), B, L, D, off, scalar, _dt(table.dtype), _stream())
        _capi.check(code, "based_stream_embed")
    return out


def stream_post_norm(residual: torch.Tensor, branch: torch.Tensor, weight: torch.Tensor, *,
                     out_weight: Optional[torch.Tensor] = None, eps: float = 1e-6) -> torch.Tensor:
    """The norm step of a post-norm block: the fp32 stream ``residual [..., D]`` becomes ``residual + rmsnorm(branch) * weight``
    IN PLACE; returns it in the branch's dtype (fp32: the stream itself), or its RMSNorm scaled by ``out_weight``."""
    _need_cuda(residual, branch, weight, out_weight)
    D = residual.shape[-1]
    if residual.dtype != torch.float32 or not residual.is_contiguous():
        raise TypeError("residual must be a contiguous float32 tensor")
    b2 = flat_rows(branch)
    _same_dtype(branch, branch=branch, weight=weight, out_weight=out_weight)
    M = residual.numel() // D if D else 0
    if b2.shape != (M, D) or weight.shape != (D,) or (out_weight is not None and out_weight.shape != (D,)):
        raise ValueError("branch must have the stream's shape and the weights its width")
    alias = out_weight is None and branch.dtype == torch.float32
    out = residual if alias else torch.empty(residual.shape, dtype=branch.dtype, device=residual.device)
    if M > 0:
        with torch.cuda.device(residual.device):
            code = _capi.lib().based_stream_post_norm(b2.data_ptr(), b2.stride(0), weight.data_ptr(), residual.data_ptr(), _ptr(out_weight),
                                                      None if alias else out.data_ptr(), M, D, float(eps), _dt(branch.dtype), _stream())
        _capi.check(code, "based_stream_post_norm")
    return out


def norm_gate(x: torch.Tensor, weight: torch.Tensor, gate: torch.Tensor, eps: float, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``rmsnorm(x) * weight * sigmoid(gate)`` over the last dim; column slices are fine for all but the weight."""
    _need_cuda(x, weight, gate, out)
    D = x.shape[-1]
    out = torch.empty(x.shape, dtype=x.dtype, device=x.device) if out is None else out
    _same_dtype(x, x=x, weight=weight, gate=gate, out=out)
    x2, g2, o2 = flat_rows(x), flat_rows(gate), flat_rows(out)
    if g2.shape != x2.shape or o2.shape != x2.shape or weight.shape != (D,):
        raise ValueError("gate and out must have x's shape and the weight its width")
    if x2.numel() > 0:
        with torch.cuda.device(x.device):
            code = _capi.lib().based_norm_gate(x2.data_ptr(), x2.stride(0), weight.data_ptr(), g2.data_ptr(), g2.stride(0), o2.data_ptr(),
                                               o2.stride(0), x2.shape[0], D, float(eps), _dt(x.dtype), _stream())
        _capi.check(code, "based_norm_gate")
    return out


def token_gate(z: torch.Tensor, tokens: torch.Tensor, table: torch.Tensor, column: int) -> torch.Tensor:
    """``gelu_tanh(z) * table[token, column : column + n]`` for ``z [..., n]``, contiguous."""
    _need_cuda(z, tokens, table)
    n = z.shape[-1]
    z2 = flat_rows(z)
    _same_dtype(z, z=z, table=table)
    if tokens.dtype != torch.int64 or tokens.numel() != z2.shape[0] or not 0 <= column <= table.shape[1] - n:
        raise ValueError("tokens must be int64, one per row, and the slice inside the table")
    out = torch.empty(z.shape, dtype=z.dtype, device=z.device)
    if out.numel() > 0:
        tokens = tokens.contiguous()
        with torch.cuda.device(z.device):
            code = _capi.lib().based_token_gate(z2.data_ptr(), z2.stride(0), tokens.data_ptr(), table.data_ptr(), table.shape[0],
                                                table.stride(0), int(column), out.data_ptr(), z2.shape[0], n, _dt(z.dtype), _stream())
        _capi.check(code, "based_token_gate")
    return out


TOKEN_SIDE_MAX_WEIGHT = 200_000   # elements of one matrix up to which one cluster per 16 rows beats the separate launches


def token_side_step(residual: torch.Tensor, x: torch.Tensor, tokens: torch.Tensor, gate_weight: torch.Tensor, proj_weight: torch.Tensor,
                    table: torch.Tensor, column: int, norm_weight: torch.Tensor, *, out_weight: Optional[torch.Tensor] = None,
                    eps: float = 1e-6) -> Optional[torch.Tensor]:
    """A layer's token input for a few rows in one launch: ``x [..., W]`` through ``gate_weight [n, W]``, :func:`token_gate`,
    ``proj_weight [W, n]`` and :func:`stream_post_norm`.  None, nothing launched, for rows, sizes or dtypes it does not take."""
    _need_cuda(residual, x, tokens, gate_weight, proj_weight, table, norm_weight, out_weight)
    n, W = gate_weight.shape
    M = x.numel() // W if W else 0
    if x.dtype != torch.bfloat16 or not 0 < M <= DECODE_LINEAR_MAX_ROWS or n * W > TOKEN_SIDE_MAX_WEIGHT:
        return None
    _same_dtype(x, x=x, gate_weight=gate_weight, proj_weight=proj_weight, table=table, norm_weight=norm_weight, out_weight=out_weight)
    x2 = flat_rows(x)
    if residual.dtype != torch.float32 or not residual.is_contiguous() or residual.shape != x.shape:
        raise TypeError("residual must be a contiguous float32 tensor of x's shape")
    if proj_weight.shape != (W, n) or not (gate_weight.is_contiguous() and proj_weight.is_contiguous()):
        raise ValueError("gate_weight must be [n, W] and proj_weight [W, n], contiguous")
    if tokens.dtype != torch.int64 or tokens.numel() != M or not 0 <= column <= table.shape[1] - n:
        raise ValueError("tokens must be int64, one per row, and the slice inside the table")
    if norm_weight.shape != (W,) or (out_weight is not None and out_weight.shape != (W,)):
        raise ValueError("norm weights must have the stream's width")
    out = torch.empty(x.shape, dtype=x.dtype, device=x.device)
    tokens = tokens.contiguous()
    with torch.cuda.device(x.device):
        code = _capi.lib().based_token_side(
            x2.data_ptr(), x2.stride(0), tokens.data_ptr(), gate_weight.data_ptr(), proj_weight.data_ptr(), table.data_ptr(), table.shape[0],
            table.stride(0), int(column), norm_weight.data_ptr(), residual.data_ptr(), _ptr(out_weight), out.data_ptr(), M, W, n, float(eps),
            _dt(x.dtype), _stream())
    if code == _capi.ERR_IMPL:
        return None
    _capi.check(code, "based_token_side")
    return out


def _check_tied(q, cache, factor, B, H, G, d):
    if H % G or q.shape[2] != H * d or cache.shape[0] < B or cache.shape[2] != G * d or cache.dtype != q.dtype or cache.stride(2) != 1:
        raise ValueError("q must be [B, L, H d] and cache [>= B, max_len, G d] in its dtype, H a multiple of G")
    if factor.dtype != torch.float32 or factor.shape[0] < B or factor.shape[1] != G or factor.shape[2] < cache.shape[1] or factor.stride(2) != 1:
        raise ValueError("factor must be float32 [>= B, G, >= max_len]")


def tied_attention_state(batch: int, heads: int, kv_heads: int, dim: int, max_len: int, dtype, device) -> dict:
    """What :func:`tied_prepare_` and :func:`tied_attention` keep for ``batch`` sequences: the keys, their factors (rows padded to
    whole key tiles) and the zeroed counters of a decode step whose keys are split."""
    rows = max(_capi.TIED_DECODE_ROWS, heads // kv_heads)
    return {"keys": torch.zeros(batch, max_len, kv_heads * dim, dtype=dtype, device=device),
            "factor": torch.zeros(batch, kv_heads, (max_len + 127) // 128 * 128, dtype=torch.float32, device=device),
            "count": torch.zeros(batch * kv_heads * ((rows + 15) // 16), dtype=torch.int32, device=device)}


def tied_prepare_(q: torch.Tensor, k: torch.Tensor, q_weight: torch.Tensor, k_weight: torch.Tensor, cache: torch.Tensor,
                  factor: torch.Tensor, *, pos=0, eps: float = 1e-6, temp_coef: float = 0.0, temp_every: float = 1.0) -> torch.Tensor:
    """Queries ``q [B, L, H d]`` normed per head, times both norm weights and ``1 + temp_coef ln(floor((p + 1) / temp_every) +
    1)`` IN PLACE; keys ``k [B, L, G d]`` appended to ``cache [B, max_len, G d]`` as they are, their inverse root mean squares to
    ``factor [B, G, max_len]``."""
    _need_cuda(q, k, q_weight, k_weight, cache, factor)
    B, L, _ = q.shape
    d = q_weight.shape[0]
    H, G = q.shape[2] // d, k.shape[2] // d
    _same_dtype(q, q=q, k=k, q_weight=q_weight, k_weight=k_weight)
    _check_tied(q, cache, factor, B, H, G, d)
    if k.shape != (B, L, G * d) or k_weight.shape != (d,):
        raise ValueError("k must be [B, L, G d]")
    off, scalar = _position(pos, q)
    if q.numel() > 0:
        with torch.cuda.device(q.device):
            code = _capi.lib().based_tied_prepare(
                q.data_ptr(), k.data_ptr(), q_weight.data_ptr(), k_weight.data_ptr(), cache.data_ptr(), factor.data_ptr(), B, L, H, G, d,
                cache.shape[1], _strides_bl(q), _strides_bl(k), _strides_bl(cache), _strides_bl(factor), off, scalar, float(eps),
                float(temp_coef), float(temp_every), _dt(q.dtype), _stream())
        _capi.check(code, "based_tied_prepare")
    return q


def tied_attention(q: torch.Tensor, cache: torch.Tensor, factor: torch.Tensor, count: torch.Tensor, heads: int, scale: float, *,
                   gate: Optional[torch.Tensor] = None, pos=0, sink: float = 0.0, out: torch.Tensor, impl: str = "auto") -> torch.Tensor:
    """Causal attention of prepared queries ``q [B, L, H d]`` at positions ``pos ..`` over ``cache [B, max_len, G d]``, whose rows
    are keys (scores times ``factor``) and values; ``sink`` scores of 0 without a value in each softmax sum; ``out [B, L, H d]``
    times ``sigmoid(gate [B, L, H d])``.  ``count``: int32 zeros, see :func:`tied_attention_state`."""
    _need_cuda(q, cache, factor, count, gate, out)
    if count.dtype != torch.int32 or not count.is_contiguous():
        raise TypeError("count must be a contiguous int32 tensor")
    B, L, W = q.shape
    d = W // heads
    G = cache.shape[2] // d
    _same_dtype(q, q=q, gate=gate, out=out)
    _check_tied(q, cache, factor, B, heads, G, d)
    if out.shape != q.shape or (gate is not None and gate.shape != q.shape):
        raise ValueError("gate and out must have q's shape")
    off, scalar = _position(pos, q)
    if out.numel() == 0:
        return out
    with torch.cuda.device(q.device):
        need = 0
        if q.dtype == torch.bfloat16 and (impl == "decode" or impl == "auto" and (off is not None or L * (heads // G) <= _capi.TIED_DECODE_ROWS)):
            need = _capi.lib().based_tied_attention_scratch_bytes(B, L, heads, G, d, cache.shape[1])
        scratch = torch.empty(need, dtype=torch.uint8, device=q.device) if need else None
        code = _capi.lib().based_tied_attention(
            q.data_ptr(), cache.data_ptr(), factor.data_ptr(), _ptr(gate), out.data_ptr(), B, L, heads, G, d, cache.shape[1],
            _strides_bl(q), _strides_bl(cache), _strides_bl(factor), _strides_bl(gate) if gate is not None else None, _strides_bl(out),
            off, scalar, float(scale), float(sink), _dt(q.dtype), _IMPLS[impl], _ptr(scratch), need, count.data_ptr(), count.numel(), _stream())
    _capi.check(code, "based_tied_attention")
    return out


def _check_lightning(state, decay, B, H, d, dv):
    if state.shape[0] < B or state.shape[1:] != (H, d, dv) or state.dtype != torch.float32 or not state.is_contiguous():
        raise ValueError("state must be a contiguous float32 [>= B, H, d, dv] tensor")
    if decay.shape != (H,) or decay.dtype != torch.float32 or not decay.is_contiguous():
        raise ValueError("decay must be float32, one per head")


def lightning(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, state: torch.Tensor, *, pos=0,
              out: Optional[torch.Tensor] = None, impl: str = "auto") -> torch.Tensor:
    """Linear attention with a constant decay per head: q, k ``[B, L, H d]``, v ``[B, L, H dv]`` before silu, ``state [B, H, d,
    dv]`` fp32 updated IN PLACE; the read-out ``[B, L, H dv]``."""
    _need_cuda(q, k, v, decay, state, out)
    B, L, _ = q.shape
    _, H, d, dv = state.shape
    _check_lightning(state, decay, B, H, d, dv)
    out = torch.empty(B, L, H * dv, dtype=q.dtype, device=q.device) if out is None else out
    _same_dtype(q, q=q, k=k, v=v, out=out)
    if q.shape[2] != H * d or k.shape != q.shape or v.shape != (B, L, H * dv) or out.shape != v.shape:
        raise ValueError("q, k must be [B, L, H d] and v, out [B, L, H dv]")
    off, scalar = _position(pos, q)
    if out.numel() == 0:
        return out
    with torch.cuda.device(q.device):
        code = _capi.lib().based_lightning(q.data_ptr(), k.data_ptr(), v.data_ptr(), decay.data_ptr(), state.data_ptr(), out.data_ptr(), B, L,
                                           H, d, dv, _strides_bl(q), _strides_bl(k), _strides_bl(v), _strides_bl(out), off, scalar,
                                           _dt(q.dtype), _IMPLS[impl], _stream())
    _capi.check(code, "based_lightning")
    return out


def lightning_step(q, k, v, gate, decay, norm_weight, state, read, count, *, pos, eps: float, out: torch.Tensor) -> bool:
    """One token per row in one launch: q, k, v, gate are column slices ``[B, .]`` of one packed projection, ``state`` is updated
    IN PLACE, ``read [B, H dv]`` fp32 and ``count [B]`` int32 (zeros) are workspace; ``out [B, H dv]`` normed over all heads and
    gated.  Returns False, nothing launched, for sizes it does not take."""
    _need_cuda(q, k, v, gate, decay, norm_weight, state, read, count, out)
    B = q.shape[0]
    _, H, d, dv = state.shape
    _check_lightning(state, decay, B, H, d, dv)
    _same_dtype(q, q=q, k=k, v=v, gate=gate, norm_weight=norm_weight, out=out)
    if q.shape[1] != H * d or k.shape != q.shape or v.shape != (B, H * dv) or gate.shape != v.shape or out.shape != v.shape or norm_weight.shape != (H * dv,):
        raise ValueError("q, k must be [B, H d] and v, gate, out [B, H dv]")
    if len({t.stride(0) for t in (q, k, v, gate)}) > 1 and B > 1:
        raise ValueError("q, k, v and gate must be slices of one tensor")
    if read.dtype != torch.float32 or read.shape[0] < B or read.shape[1] != H * dv or not read.is_contiguous() or count.dtype != torch.int32 or count.numel() < B:
        raise ValueError("read must be contiguous float32 [>= B, H dv] and count int32 [>= B]")
    off, scalar = _position(pos, q)
    if B == 0:
        return True
    with torch.cuda.device(q.device):
        code = _capi.lib().based_lightning_step(
            q.data_ptr(), k.data_ptr(), v.data_ptr(), gate.data_ptr(), q.stride(0), decay.data_ptr(), norm_weight.data_ptr(),
            state.data_ptr(), read.data_ptr(), count.data_ptr(), out.data_ptr(), out.stride(0), B, H, d, dv, off, scalar, float(eps),
            _dt(q.dtype), _stream())
    if code == _capi.ERR_IMPL:
        return False
    _capi.check(code, "based_lightning_step")
    return True
