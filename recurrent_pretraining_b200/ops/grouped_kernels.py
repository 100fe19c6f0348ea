"""Bindings of the tensor-core kernels of grouped-query attention over a step's key stream (``csrc/latent_attention.cu``) and over
ring caches (``csrc/gqa_decode.cu``)."""


def prompt_supported(L, a) -> bool:
    return False


def decode_supported(L) -> bool:
    return False
