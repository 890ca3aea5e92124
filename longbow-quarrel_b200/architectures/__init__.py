from . import fetorax, korazen, lavutar, llama, raritar, zoporax  # noqa: F401  (registers LlamaForCausalLM, Fetorax, Korazen, Lavutar, Raritar and Zoporax)
