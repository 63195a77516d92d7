"""Parts of a layer.  Importing this package registers the built-in parts."""
from . import attention, block, branches, embedding, ffn, input_conv, latent_attention, mlstm, norm, recurrent, rope  # noqa: F401
from .base import BuildContext, EmbedAddition, FeedForward, Mixer, Norm, Part, PositionEncoding, StreamMix  # noqa: F401
