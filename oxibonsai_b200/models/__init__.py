"""Model families.  ``qwen3`` (sub-2-bit GGUF), ``qwen3_generic`` (other GGUF block formats) and ``layered`` (decoders described
layer by layer in a ``config.json``); ``registry`` maps shapes to variants and architecture names to configuration readers."""
