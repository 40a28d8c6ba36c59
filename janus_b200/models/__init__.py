from . import buludra, forisun, llama, mibezen, mugedra, ramolix, zivitar  # noqa: F401  (registers Buludra, Forisun, LlamaForCausalLM, Mibezen, Mugedra, Ramolix and Zivitar)
