"""out = x . W^T for a weight [out, in] without bias: picks the kernel by dtype and row count.

float32: the CUDA-core sgemm for every size (a true 32-bit product). bfloat16: up to 8 rows the
streaming kernel (cp.async rings, weights read once); up to 128 rows the TMA + tcgen05 kernel in its
decode form (one tile of rows, K in slices); for more rows (prefill) the same kernel, always for the
gated product (SiLU*up fused into its epilogue) and otherwise when its 128 x 256 tiles fill the
GPU's waves, else the library matrix product (the reference uses the library for all of these,
engine/fused.py:993-995)."""
import torch

from ..csrc import api

STORE, STORE_F32, SILU, XIELU = api.MODE_STORE, api.MODE_STORE_F32, api.MODE_SILU, api.MODE_XIELU


def linear(x, w, mode=STORE, allow_partial=False, act=(0.0, 0.0)):
    """mode STORE: [M, N] in x's dtype; STORE_F32: float32 (logits); SILU: w = [gate; up] rows,
    returns silu(x.gate^T) * (x.up^T) of width N/2 (with ``act`` = ``api.GATE_GELU`` the gate goes through the tanh
    form of GELU instead, with ``api.gate_clamped(limit)`` through the clamped gate); XIELU: xielu(x.w^T) with the constants ``act`` =
    (alpha_pos, alpha_neg), in the product's epilogue wherever the product is this library's (after
    the library's product a row kernel applies it). ``allow_partial``: the caller can take
    ``csrc.api.Partial`` (split-K partial sums, added up by the kernel that consumes them) instead
    of a tensor (with STORE_F32 too: partial sums are float32)."""
    M, K = x.shape
    N = w.shape[0] // 2 if mode == SILU else w.shape[0]
    if x.dtype == torch.float32:
        out = torch.empty((M, N), dtype=torch.float32, device=x.device)
        api.sgemm(x, w, out, mode, act)
        return out
    if x.data_ptr() % 16:        # a single row cut out of a wider one is dense where it lies: the products read 16 bytes at a time
        x = x.clone()
    if K % 8:
        # an inner size the tensor-core kernels do not take (their rows sit on 16-byte boundaries): the library's
        # product, and the activation as a row kernel behind it
        if mode == STORE_F32:
            return torch.mm(x, w.t(), out_dtype=torch.float32)
        out = torch.mm(x, w.t())
        if mode == SILU:
            half = torch.empty((M, N), dtype=x.dtype, device=x.device)
            if act[0] > 1.5:
                api.act_mul(out, half, api.ACT_CLAMPED, act[1])
            else:
                api.act_mul(out, half, api.ACT_GELU_TANH if act[0] > 0.5 else api.ACT_SILU)
            return half
        if mode == XIELU:
            api.xielu(out, out, act[0], act[1])
        return out
    if M <= api.STREAM_BEST_ROWS and K % 16 == 0:
        plan = api.stream_plan(M, N, K, mode, allow_partial)
        if plan is not None:
            return api.gemv_stream(x, w, None, mode, plan, act)
    if M <= api.TC_SKINNY_MAX_ROWS:
        # a decode step of up to 128 rows: weights streamed once by TMA, one 128-row tile of x,
        # K in slices so that the few weight tiles still cover the SMs
        plan = api.skinny_tc_plan(M, N, K, STORE if mode == STORE_F32 and allow_partial else mode, allow_partial)
        return api.gemm_tc(x, w, STORE if mode == STORE_F32 and plan[1] > 1 else mode, None, plan, act)
    if mode == STORE_F32:
        return torch.mm(x, w.t(), out_dtype=torch.float32)
    if mode == SILU:
        return api.gemm_tc(x, w, mode, None, api.gated_tc_plan(M, N), act)   # TMA + tcgen05, SiLU*up fused into the epilogue
    if api.gemm_tc_fills_gpu(M, N):
        return api.gemm_tc(x, w, mode, act=act)
    out = torch.mm(x, w.t())
    if mode == XIELU:
        api.xielu(out, out, act[0], act[1])
    return out


def linear_partial(x, w):
    """x . w^T in float32 as a ``csrc.api.Partial`` (of one slice or more), for the kernels that put it into the stream."""
    y = linear(x, w, STORE_F32, allow_partial=True)
    return y if isinstance(y, api.Partial) else api.Partial(y.unsqueeze(0))
