"""Several residual streams per token (csrc/hyper_streams.cu): a sublayer's write into all streams and the next sublayer's normed read
of them in one kernel.  Streams, sums and the norm are fp32 for every storage dtype of the projections."""
import torch

from swiftllm_b200 import _lib


def stream_mix_norm(x: torch.Tensor, streams: int, y=None, mix=None, share=None, x_out=None, read=None, norm_w=None, eps: float = 0.0,
                    out_dtype: torch.dtype = None, rows=None):
    """x fp32 [T, streams, W], or [T, W] while all streams are equal.  With y ([T, W], out_dtype): x_t <- sum_s mix[s, t] x_s + share[t] y
    (mix fp32 [from, to], share fp32 [streams]).  x_out (fp32 [T, streams, W], may be x) receives the streams; with norm_w (fp32 [W])
    the result is h = rms(sum_s read[s] x_s) * norm_w [T, W] in out_dtype, else None.  rows (int32): only these tokens, h has one row for
    each."""
    one = x.dim() == 2
    T, W = x.shape[0], x.shape[-1]
    assert x.dtype == torch.float32 and x.is_contiguous() and (one or x.shape[1] == streams)
    assert y is None or (y.is_contiguous() and y.shape == (T, W) and y.dtype == out_dtype and mix.dtype == share.dtype == torch.float32
                         and mix.is_contiguous() and mix.shape == (streams, streams) and share.shape == (streams,))
    assert x_out is None or (x_out.dtype == torch.float32 and x_out.is_contiguous() and x_out.shape == (T, streams, W))
    assert norm_w is None or (norm_w.dtype == read.dtype == torch.float32 and norm_w.shape == (W,) and read.shape == (streams,))
    assert rows is None or rows.dtype == torch.int32
    _lib.require_device(x)
    n = T if rows is None else rows.shape[0]
    h = torch.empty((n, W), dtype=out_dtype, device=x.device) if norm_w is not None else None
    _lib.check(_lib.lib().sllm_stream_mix_norm(
        x.data_ptr(), 1 if one else 0, streams, _lib.ptr(y), _lib.ptr(mix), _lib.ptr(share), _lib.ptr(read), _lib.ptr(norm_w), eps,
        _lib.ptr(x_out), _lib.ptr(h), _lib.ptr(rows), n, W, _lib.dtype_tag_f32(out_dtype), _lib.stream()), "stream_mix_norm")
    return h
