"""Runner of decoders built from the layers of _C/_hybrid_layers.py: the Llama runner's interface (forward, generate with a
recorded decode step, beam_search) over caches of pages and recurrent states. A model family adds `_embed` (token ids to what
its first layer takes) and `_head`, and `_stream_rows` for inspection."""
import torch

from .._C import _hybrid_layers as hybrid
from .fused_llama_infer import LlamaRunner
from .llm_common import TppCache


class HybridRunner(LlamaRunner):
    packable = False

    def __init__(self, shape, embed, layers, norm_w, lm_head_w, dtype):
        super().__init__(shape, embed, layers, norm_w, lm_head_w, None)
        self.dtype = dtype
        self.layer_outputs = None  # a list: receives the stream [B * S, D] after every layer of the next forward calls

    def _wanted_rows(self, B, S, device):
        """Rows of a call's B * S tokens whose logits are wanted."""
        if self.logit_rows is not None:
            return self.logit_rows
        rows = torch.arange(B * S, device=device)
        return rows[S - 1::S].contiguous() if self.only_last_logit else rows

    def _logits(self, h, B):
        """fp32 logits of normed rows: [B, 1, V] (last token), [B, S, V], or [rows, V] with logit_rows."""
        logits = hybrid.linear(h, self.lm_head_w, out_f32=True)
        return logits if self.logit_rows is not None else logits.view(B, -1, logits.shape[-1])

    def _stream_rows(self, s, layer, cpp, past):
        """The residual stream behind `layer`, [B * S, D] fp32."""
        raise NotImplementedError

    def _pick(self, logits):
        return hybrid.argmax_rows_f32(logits[:, -1]).unsqueeze(-1)

    def _reserve(self, cpp, batch, tokens, device):
        for layer in self.layers:
            layer.reserve(cpp, batch, tokens, device)

    def _decode_mask(self, cpp, mask, past, cap):
        return cpp.start

    @staticmethod
    def _padding(attention_mask):
        """Leading padding per sequence from a keep-mask; a state cannot skip tokens in the middle."""
        keep = attention_mask.to(torch.int64)
        start = keep.shape[1] - keep.sum(-1)
        if not torch.equal(keep, (torch.arange(keep.shape[1], device=keep.device) >= start.unsqueeze(-1)).to(torch.int64)):
            raise ValueError("sequences must be padded on the left")
        return start.to(torch.int32).contiguous()

    @torch.no_grad()
    def forward(self, input_ids, attention_mask=None, position_ids=None, cache=None):
        """Logits of a call's tokens and the cache behind them. attention_mask [B, S] (1 = token, 0 = left padding) counts
        at a sequence's first call; positions follow from it."""
        cache = TppCache() if cache is None else cache
        cpp = cache.get_cpp()
        B, S = input_ids.shape
        if input_ids.numel() and (int(input_ids.min()) < 0 or int(input_ids.max()) >= self.shape.vocab_size):
            raise ValueError("token id outside the vocabulary")
        if cpp.get_seq_length() == 0:
            cpp.start = torch.zeros(B, dtype=torch.int32, device=input_ids.device) if attention_mask is None else self._padding(attention_mask)
        if cpp.start.shape[0] != B:
            raise ValueError(f"the cache holds {cpp.start.shape[0]} sequences, the call has {B}")
        s = self._embed(input_ids, None)
        for layer in self.layers:
            s = layer.forward([s, cpp.start], cpp, True)[0]
            if self.layer_outputs is not None:
                self.layer_outputs.append(self._stream_rows(s, layer, cpp, cpp.get_seq_length() - S))
        for lc in cpp.layers:
            lc.live = None
        return self._head(s), cache
