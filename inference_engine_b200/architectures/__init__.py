from . import livitar, llama, puposun, ravapel, rugedra, vofanex  # noqa: F401 (register Livitar, LlamaForCausalLM, Puposun, Ravapel, Rugedra and Vofanex)
