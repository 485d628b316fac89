"""Architectures by name: config.json -> decoder configuration, weights and decoder class.

`architecture` (or the first entry of `architectures`, as Hugging Face writes it) picks the entry; every entry turns the parsed
config and the checkpoint's state dict into a decoder.  Used by the command line and the trace runner."""
from . import checkpoint
from ._lib import PtError


def _llama(c, sd, batch, max_len, dtype, **kw):
    from .llama import LlamaConfig, LlamaDecoder
    if c.get("num_key_value_heads", c["num_attention_heads"]) != c["num_attention_heads"]:
        raise PtError("LlamaDecoder has no grouped key/value heads")
    cfg = LlamaConfig(c["num_hidden_layers"], c["hidden_size"], c["num_attention_heads"], c["intermediate_size"], c["vocab_size"],
                      eps=c.get("rms_norm_eps", 1e-5), max_len=max_len)
    return LlamaDecoder(cfg, checkpoint.llama_from_hf(sd), batch, **kw)


def _gpt2(c, sd, batch, max_len, dtype, **kw):
    from .gpt2 import GPT2Config, GPT2Decoder
    cfg = GPT2Config(n_layer=c["n_layer"], d_model=c["n_embd"], n_head=c["n_head"], vocab=c["vocab_size"], max_len=max_len, n_positions=c["n_positions"])
    return GPT2Decoder(cfg, checkpoint.gpt2_from_hf(sd, c["n_embd"], c["n_head"]), batch, **kw)


def _chatglm2(c, sd, batch, max_len, dtype, **kw):
    from .chatglm2 import ChatGLM2Config, ChatGLM2Decoder
    cfg = ChatGLM2Config(c["num_layers"], c["hidden_size"], c["num_attention_heads"], c["multi_query_group_num"], c["ffn_hidden_size"],
                         c["padded_vocab_size"], max_len, eps=c.get("layernorm_epsilon", 1e-5))
    return ChatGLM2Decoder(cfg, checkpoint.chatglm2_from_hf(sd, c["hidden_size"]), batch, **kw)


def _rwkv(c, sd, batch, max_len, dtype, **kw):
    from .rwkv import RWKVConfig, RWKVDecoder
    every = c.get("rescale_every", 6)
    cfg = RWKVConfig(c["num_hidden_layers"], c["hidden_size"], c.get("intermediate_size") or 4 * c["hidden_size"], c["vocab_size"], max_len,
                     rescale_every=every, eps=c.get("layer_norm_epsilon", 1e-5))
    return RWKVDecoder(cfg, checkpoint.rwkv_from_hf(sd, every), batch, **kw)


def _sabisun(c, sd, batch, max_len, dtype, **kw):
    from .sabisun import SabisunConfig, SabisunDecoder
    return SabisunDecoder(SabisunConfig(c, max_len), sd, batch, dtype=dtype, **kw)


def _padetar(c, sd, batch, max_len, dtype, **kw):
    from .padetar import PadetarConfig, PadetarDecoder
    return PadetarDecoder(PadetarConfig(c, max_len), sd, batch, dtype=dtype, **kw)


def _pivavik(c, sd, batch, max_len, dtype, **kw):
    from .pivavik import PivavikConfig, PivavikDecoder
    return PivavikDecoder(PivavikConfig(c, max_len), sd, batch, dtype=dtype, **kw)


def _puputar(c, sd, batch, max_len, dtype, **kw):
    from .puputar import PuputarConfig, PuputarDecoder
    return PuputarDecoder(PuputarConfig(c, max_len), sd, batch, dtype=dtype, **kw)


# name -> (builder, dtypes the decoder runs in; the first is the default)
ARCHITECTURES = {
    "LlamaForCausalLM": (_llama, ("float16",)),
    "GPT2LMHeadModel": (_gpt2, ("float16",)),
    "ChatGLMModel": (_chatglm2, ("float16",)),
    "ChatGLMForConditionalGeneration": (_chatglm2, ("float16",)),
    "RwkvForCausalLM": (_rwkv, ("float16",)),
    "Sabisun": (_sabisun, ("bfloat16", "float32")),
    "Padetar": (_padetar, ("bfloat16", "float32")),
    "Pivavik": (_pivavik, ("bfloat16", "float32")),
    "Puputar": (_puputar, ("bfloat16", "float32")),
}


class UnsupportedDtype(PtError):
    pass


def architecture(config):
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in ARCHITECTURES:
        raise PtError(f"unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return name


def dtypes(config):
    return ARCHITECTURES[architecture(config)][1]


def build_decoder(config, state_dict, batch, max_len, dtype=None, **kw):
    """The decoder of a model: `batch` rows of at most `max_len` tokens; further options go to the decoder's constructor."""
    builder, known = ARCHITECTURES[architecture(config)]
    dtype = known[0] if dtype is None else dtype
    if dtype not in known:
        raise UnsupportedDtype(f"{architecture(config)} runs in {' / '.join(known)}, not in {dtype}")
    return builder(config, state_dict, batch, max_len, dtype, **kw)


def load_decoder(model_dir, batch, max_len, dtype=None, **kw):
    config, sd = checkpoint.load_model_dir(model_dir)
    return build_decoder(config, sd, batch, max_len, dtype, **kw)
