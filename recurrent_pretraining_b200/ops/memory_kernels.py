def prompt_supported(L, spec): return False
def chunk_supported(a, b): return False
def decode_supported(L): return False
