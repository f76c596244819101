"""A sequential pre-norm decoder block on several residual streams (hyper-connections): a sublayer reads h = rms(sum_s in[s] x_s) * w, and
its output y goes back into all streams at once, x_t <- sum_s mix[s, t] x_s + share[t] y.  The kernel that writes a sublayer's output also
does the read of the sublayer that follows, so `forward` takes its first read's result and returns the read that comes after the
block.  One stream with all weights one is the plain residual sum."""
import torch

from swiftllm_b200.model_config import DeltaRuleSpec, MatrixMemorySpec, WindowAttentionSpec
from swiftllm_b200.worker.kernels.hyper_streams import stream_mix_norm
from swiftllm_b200.worker.layers.delta_rule import GatedDeltaRuleMixer
from swiftllm_b200.worker.layers.feed_forward import build_feed_forward
from swiftllm_b200.worker.layers.matrix_memory import MatrixMemoryMixer
from swiftllm_b200.worker.layers.window_attention import WholeNormAttentionMixer


class HyperStreamBlockLayer:
    def __init__(self, model_config, weight, layer_id: int):
        mc = model_config
        self.layer_id, self.weight, self.eps, self.streams = layer_id, weight, mc.rms_norm_eps, mc.num_streams
        spec = mc.mixers[layer_id]
        if isinstance(spec, DeltaRuleSpec):
            self.mixer = GatedDeltaRuleMixer(spec, weight, self.eps, layer_id)
        elif isinstance(spec, MatrixMemorySpec):
            self.mixer = MatrixMemoryMixer(spec, weight, self.eps, layer_id)
        else:
            assert isinstance(spec, WindowAttentionSpec)
            self.mixer = WholeNormAttentionMixer(spec, weight, self.eps, mc.cache_slot[layer_id])
        self.ff = build_feed_forward(mc.ffs[layer_id], weight)

    def _write_and_read(self, x, x_out, y, conn, read, rows=None):
        """conn: the sublayer's (mix, share); read: the next sublayer's (weights of the streams, norm weight), or None."""
        return stream_mix_norm(x, self.streams, y=y, mix=conn.mix, share=conn.share, x_out=x_out, read=None if read is None else read[0],
                               norm_w=None if read is None else read[1], eps=self.eps, out_dtype=y.dtype, rows=rows)

    def forward(self, x, x_out, h, caches, block_table, states, st, next_read, last_rows=None):
        """x fp32 [T, streams, W] (or [T, W]: all streams equal) before the block, x_out where they go (x itself once it has all streams);
        h = the first sublayer's read; next_read: the read that comes after the block.  last_rows: only these tokens are read
        afterwards and nothing needs the streams any more.  -> the read that comes after the block."""
        w = self.weight
        y = self.mixer.forward(h, caches, block_table, states, st)
        if self.ff is not None:
            h = self._write_and_read(x, x_out, y, w.conn1, (w.conn2.read, w.norm2))
            x, conn, y = x_out, w.conn2, self.ff.forward(h)
        else:
            conn = w.conn1
        return self._write_and_read(x, None if last_rows is not None else x_out, y, conn, next_read, rows=last_rows)
