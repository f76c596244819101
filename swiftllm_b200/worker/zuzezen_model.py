"""ZuzezenModel - worker of the Zuzezen design: SEQUENTIAL blocks on an fp32 residual stream whose sublayers read the stream itself
and whose outputs go through an RMS norm and an element-wise scale before they are added; mixers are latent attention with a
learned softmax sink and an element-wise gate (worker/layers/latent_attention.py), windowed attention whose values are its un-normed
keys, with kept first positions and a bias on the distance (worker/layers/window_attention.py), or gated linear attention with a
decay per key channel and token (worker/layers/gated_linear_attention.py); feed-forwards are SiLU gated linear units with biases.

The public surface, the paged cache, the per-sequence state rows, the step's metadata and the CUDA-graph decode path are the
shared token-batch worker's (worker/token_model.py), the block is worker/layers/sequential_block.py.  Per sequence this design
keeps, besides the attention layers' cache rows, every linear attention's state."""
from __future__ import annotations

import torch

from swiftllm_b200.model_config import ZuzezenModelConfig
from swiftllm_b200.worker.kernels.linear import linear_f32_out
from swiftllm_b200.worker.kernels.parallel_block import add_rmsnorm_f32
from swiftllm_b200.worker.kernels.stream_ops import embed_pair_hash
from swiftllm_b200.worker.weight import load_zuzezen_weights

from .infer_state import TokenInferState
from .layers.sequential_block import PostNormBlockLayer
from .token_model import TokenBatchModel


class ZuzezenModel(TokenBatchModel):
    NATIVE_SOURCES = TokenBatchModel.NATIVE_SOURCES + ("parallel_block.cu", "stream_ops.cu", "latent_attn.cu", "window_attn.cu", "gla.cu")
    CONFIG_CLASS = ZuzezenModelConfig

    @staticmethod
    def _load_weights(model_config, dtype, model_path, use_dummy, getter, device):
        return load_zuzezen_weights(model_config, dtype, model_path, use_dummy, getter=getter, device=device)

    def _build_layers(self) -> list:
        layers = [PostNormBlockLayer(self.model_config, self.weight.layers[i], i) for i in range(self.model_config.num_layers)]
        for layer in layers:
            layer.mixer.register(self)
        return layers

    def _state_layout(self) -> dict:
        layout = {}
        for layer in self.layers:
            layout.update(layer.mixer.state_layout())
        return layout

    @torch.inference_mode()
    def _forward(self, input_ids: torch.Tensor, st: TokenInferState) -> torch.Tensor:
        """-> fp32 logits of st.output_rows."""
        mc, w = self.model_config, self.weight
        x, h = embed_pair_hash(input_ids, st, None, w.wte, None, 0, 0, 0, scale=mc.embedding_scale)
        self._wait_for_swaps()
        block_table = None if st.ignore_kvcache else self.gpu_block_manager.block_table
        keep = [] if self.keep_residuals else None
        for layer in self.layers:
            layer.forward(x, h, self.caches, block_table, self.seq_states, st)
            if keep is not None:
                keep.append(x.clone())
        self.last_residuals = keep
        rows = x.index_select(0, st.output_rows)
        hn = add_rmsnorm_f32(rows, None, None, w.final_norm, mc.rms_norm_eps, out_dtype=self.dtype)
        return linear_f32_out(hn, w.lm_head)
