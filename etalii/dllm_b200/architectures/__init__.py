from . import gaperax, llama, revupel, satavik, tezinex, tisalorn  # noqa: F401  (register the architectures)
