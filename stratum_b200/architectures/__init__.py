from . import dabodra, getizen, llama, mokatar, nibelorn, vitinex  # noqa: F401  (registers the architectures)
