"""vui_b200: Vui Nano's per-codec-frame decode step as sm_100a CUDA behind the
reference's Engine / Row / GenConfig API, and token language models on the same slot engine."""

from .codec import CodecCtx, QwenCodecDecoder
from .codec_encoder import QwenCodecEncoder, StreamingCodecEncoder
from .engine import Engine, GenConfig, RenderRequest, Row, Segment
from .model import VuiB200, VuiShape
from .registry import load_model, open_engine
from .token_engine import TokenEngine, TokenGenConfig, TokenRow
from .token_lm import Medirax, TokenLM, Vidotar

__all__ = ["CodecCtx", "Engine", "GenConfig", "Medirax", "QwenCodecDecoder", "QwenCodecEncoder", "RenderRequest", "Row", "Segment",
           "StreamingCodecEncoder", "TokenEngine", "TokenGenConfig", "TokenLM", "TokenRow", "Vidotar", "VuiB200", "VuiShape",
           "load_model", "open_engine"]
