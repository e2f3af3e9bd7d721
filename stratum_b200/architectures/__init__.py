from . import dabodra, getizen, llama, memipel, mokatar, nibelorn, vitinex  # noqa: F401  (registers the architectures)
