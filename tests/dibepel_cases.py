"""Small random models of the Dibepel design for the tests: sizes that are no multiples of tiles, single and equal
head counts, windows and chunks at and beside page borders, borrowed weights, layers without a feed-forward.
Queries are scaled up so that single keys dominate and a lost or extra key shows in the output."""

from flashrec_b200.dibepel import DibepelConfig, random_tensors


def diff(heads, kv, dim, vdim, size, keep, d=0.35, scale=None, ff=88, **extra):
    return dict(type="attention", mlp=None if ff is None else dict(kind="dense", ff=ff),
                mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, diff=d,
                           mask=dict(size=size, keep_first=keep)), **extra)


def talk(heads, kv, dim, vdim, size, conv, scale=None, ff=88, **extra):
    return dict(type="attention_2", mlp=None if ff is None else dict(kind="dense", ff=ff),
                mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, conv=conv,
                           mask=dict(size=size)), **extra)


def config(vocab, width, layers, eps=1e-5, scale=3.0):
    return dict(architecture="Dibepel", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale),
                layers=layers)


CASES = {
    # nothing a multiple of 16; three query heads per kv head; a layer without feed-forward; borrowed weights
    "ragged": config(131, 90, [diff(6, 2, 20, 24, 37, 3), talk(6, 3, 24, 40, 50, 3), talk(6, 2, 12, 20, 33, 5, ff=None),
                               diff(6, 2, 20, 24, 37, 3, weights_of=0), talk(6, 3, 24, 40, 50, 3, weights_of=1)]),
    # heads == kv heads, windows and chunks of exactly one page, nothing kept, one tap
    "equal": config(200, 128, [diff(2, 2, 64, 64, 64, 0, ff=160), talk(4, 4, 64, 64, 64, 1, ff=160)], eps=1e-3, scale=1.0),
    # one kv head, wide heads, a kept range beyond one page, a window and a chunk across pages
    "single_kv": config(97, 160, [talk(4, 1, 128, 128, 130, 4, ff=200), diff(4, 1, 96, 128, 100, 70, ff=64)]),
    # the whole sequence visible (window and chunk larger than it), one head, long convolution
    "one_head": config(67, 64, [diff(1, 1, 32, 48, 5000, 1, ff=40), talk(1, 1, 40, 16, 9999, 7, ff=None),
                                talk(1, 1, 40, 16, 9999, 7, ff=None, weights_of=1)]),
    # a window of one token besides the kept ones, chunks of three
    "narrow": config(80, 48, [diff(3, 1, 16, 32, 1, 2, ff=32), talk(2, 2, 16, 16, 3, 2, ff=32)]),
    # head sizes that only the row kernels take
    "wide_heads": config(64, 96, [diff(2, 1, 208, 224, 70, 5, ff=48), talk(2, 1, 200, 200, 40, 3, ff=48)]),
}


def make(name, seed=1, sharp=3.0):
    """(config dict, parsed config, bf16 tensors)"""
    raw = CASES[name]
    cfg = DibepelConfig.from_json(raw)
    tensors = random_tensors(cfg, seed)
    for k, t in tensors.items():
        if k.endswith("mix.q"):
            tensors[k] = (t.float() * sharp).to(t.dtype)
    return raw, cfg, tensors


def tokens(cfg, n, seed=0):
    import torch

    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg.vocab, (n,), generator=g).tolist()
