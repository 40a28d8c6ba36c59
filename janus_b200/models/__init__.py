from . import buludra, forisun, llama, mugedra, ramolix, zivitar  # noqa: F401  (registers Buludra, Forisun, LlamaForCausalLM, Mugedra, Ramolix and Zivitar)
