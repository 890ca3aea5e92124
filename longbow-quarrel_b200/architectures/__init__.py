from . import fetorax, gevipel, korazen, lavutar, llama, raritar, zoporax  # noqa: F401  (registers LlamaForCausalLM, Fetorax, Gevipel, Korazen, Lavutar, Raritar and Zoporax)
