"""VoreraxModel - worker of the Vorerax design: SEQUENTIAL pre-norm blocks on several fp32 residual streams (hyper-connections); mixers are
windowed attention whose values are its un-normed keys, with norms over the whole projections, partial rotation, a learned sink and a
gate per head (worker/layers/window_attention.py), the gated delta rule behind short convolutions (worker/layers/delta_rule.py) or a
matrix memory with exponential input gate (worker/layers/matrix_memory.py); feed-forwards are mixtures of SiLU-gated experts with
group-limited sigmoid routing; the embedding adds a hashed table of token pairs.

The public surface, the paged cache, the per-sequence state rows, the step's metadata and the CUDA-graph decode path are the shared
token-batch worker's (worker/token_model.py), the block is worker/layers/hyper_block.py.  Per sequence this design keeps, besides the
attention layers' cache rows: the previous token, every delta layer's state and convolution tail, every matrix memory's state,
normaliser and running maximum."""
from __future__ import annotations

import torch

from swiftllm_b200.model_config import VoreraxModelConfig
from swiftllm_b200.worker.kernels.hyper_streams import stream_mix_norm
from swiftllm_b200.worker.kernels.linear import linear_f32_out
from swiftllm_b200.worker.kernels.stream_ops import embed_pair_hash
from swiftllm_b200.worker.weight import load_vorerax_weights

from .infer_state import TokenInferState
from .layers.hyper_block import HyperStreamBlockLayer
from .token_model import TokenBatchModel

LAST_TOKEN = "last_token"


class VoreraxModel(TokenBatchModel):
    NATIVE_SOURCES = TokenBatchModel.NATIVE_SOURCES + ("stream_ops.cu", "hyper_streams.cu", "window_attn.cu", "scan_ops.cu", "delta_rule.cu",
                                                       "matrix_memory.cu")
    CONFIG_CLASS = VoreraxModelConfig

    @staticmethod
    def _load_weights(model_config, dtype, model_path, use_dummy, getter, device):
        return load_vorerax_weights(model_config, dtype, model_path, use_dummy, getter=getter, device=device)

    def _build_layers(self) -> list:
        layers = [HyperStreamBlockLayer(self.model_config, self.weight.layers[i], i) for i in range(self.model_config.num_layers)]
        for layer in layers:
            layer.mixer.register(self)
        return layers

    def _state_layout(self) -> dict:
        layout = {}
        if self.model_config.pair_hash is not None:
            layout[LAST_TOKEN] = ((), torch.int32)
        for layer in self.layers:
            layout.update(layer.mixer.state_layout())
        return layout

    @torch.inference_mode()
    def _forward(self, input_ids: torch.Tensor, st: TokenInferState) -> torch.Tensor:
        """-> fp32 logits of st.output_rows."""
        mc, w = self.model_config, self.weight
        T, S, layers = input_ids.shape[0], mc.num_streams, self.layers
        pair, states = mc.pair_hash, self.seq_states
        if pair is not None and not st.ignore_kvcache:
            x, _ = embed_pair_hash(input_ids, st, states[LAST_TOKEN], w.wte, w.pairs, pair.buckets, pair.mul_prev, pair.mul_cur,
                                   scale=mc.embedding_scale, want_h=False)
        else:
            x, _ = embed_pair_hash(input_ids, st, None, w.wte, None, 0, 0, 0, scale=mc.embedding_scale, want_h=False)
        self._wait_for_swaps()
        block_table = None if st.ignore_kvcache else self.gpu_block_manager.block_table
        keep = [] if self.keep_residuals else None
        reads = [(l.weight.conn1.read, l.weight.norm1) for l in layers] + [(w.final_read, w.final_norm)]
        h = stream_mix_norm(x, S, read=reads[0][0], norm_w=reads[0][1], eps=mc.rms_norm_eps, out_dtype=self.dtype)
        streams = torch.empty((T, S, mc.hidden_size), dtype=torch.float32, device=self.device)
        for i, layer in enumerate(layers):
            last = i + 1 == len(layers) and keep is None        # the streams end here: only the output rows are read once more
            h = layer.forward(x, streams, h, self.caches, block_table, states, st, reads[i + 1], st.output_rows if last else None)
            x = streams
            if keep is not None:
                keep.append(x.sum(dim=1))
        self.last_residuals = keep
        if keep is not None:
            h = h.index_select(0, st.output_rows)
        return linear_f32_out(h, w.lm_head)
