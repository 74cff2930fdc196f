from . import kolisun, livitar, llama, puposun, ravapel, rugedra, vofanex  # noqa: F401 (register Kolisun, Livitar, LlamaForCausalLM, Puposun, Ravapel, Rugedra and Vofanex)
