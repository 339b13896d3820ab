from . import gaperax, llama, revupel, satavik, tezinex, tisalorn, zivazen  # noqa: F401  (register the architectures)
