"""Small Tadalorn configurations for the tests: sizes that differ from one another in every place, values that happen to be 1 or
equal to one another, windows shorter than a page and longer than any prompt, kept tokens from none to more than a tile of keys,
layers that run with another layer's tensors."""
from __future__ import annotations


def mlstm(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def attention(heads, kv_heads, dim, taps, scale, window, keep, rot_dims, base=10000.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": taps, "scale": scale,
            "mask": None if window is None else {"size": window, "keep_first": keep}, "rot": {"base": base, "dims": rot_dims}}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
            "rot": {"base": base, "dims": rot_dim}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(kind, mixer, mlp, weights_of=None):
    out = {"type": kind, "mixer": mixer, "mlp": mlp}
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


def model(vocab, width, layers, residual_mult=0.6, softcap=20.0, eps=1e-5):
    return {"architecture": "Tadalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": residual_mult,
            "logit_softcap": softcap, "layers": layers}


def again(layers, source):
    """An entry that runs with the tensors of layer ``source``."""
    return dict(layers[source], weights_of=source)


# every mechanism at once: an attention and a memory that run again later with the same tensors, a window of 20 in the middle of
# pages with three kept tokens, routed and dense feed-forwards and none
_TA = [layer("attention", attention(4, 2, 16, 3, 0.4, 20, 3, 8), moe(5, 2, 24, shared=40)),
       layer("mlstm", mlstm(3, 16, 24, 6.0), dense(72)),
       layer("latent_attention", latent(2, 16, 8, 24, 40, 0.2), moe(6, 3, 16))]
TA = model(101, 64, _TA + [again(_TA, 0), layer("latent_attention", latent(3, 8, 4, 8, 24, 0.3, base=500.0), None), again(_TA, 1)])
# one head each, a convolution of one tap (which carries nothing), a window of one token without kept ones and an attention that
# sees everything, a router that takes every expert, no cap on the logits, sizes that are no multiple of 4
TB = model(131, 45, [layer("attention", attention(1, 1, 12, 1, 0.5, 1, 0, 2), moe(3, 3, 20, shared=24)),
                     layer("attention", attention(3, 1, 6, 2, 0.4, None, 0, 6), None),
                     layer("latent_attention", latent(1, 13, 6, 21, 36, 0.25, base=200000.0), dense(57)),
                     layer("mlstm", mlstm(1, 7, 9, 15.0), moe(4, 1, 12))], residual_mult=1.0, softcap=None, eps=1e-6)
# only state, no keys: memories whose first one runs three times, keys wider than values and narrower, a cap that bends every gate
_TC = [layer("mlstm", mlstm(2, 20, 12, 1.5), dense(30)), layer("mlstm", mlstm(4, 6, 22, 15.0), None)]
TC = model(60, 50, _TC + [again(_TC, 0), again(_TC, 0)], residual_mult=0.3, softcap=3.0)
# shapes of the tensor-core kernels, without routers (so that no row of bfloat16 is routed elsewhere): heads of two tiles of value
# columns, six query heads on one key head with nine kept tokens, a latent of 64, eight taps, a repeated attention
_TD = [layer("mlstm", mlstm(2, 40, 136, 8.0), dense(96)),
       layer("attention", attention(6, 1, 40, 8, 0.3, 70, 9, 16, base=1e6), dense(64)),
       layer("latent_attention", latent(4, 32, 16, 32, 64, 0.2, base=20000.0), None)]
TD = model(97, 96, _TD + [again(_TD, 1), layer("mlstm", mlstm(3, 64, 64, 15.0), dense(80))])
# more kept tokens than a tile of keys holds, a window of one tile and one more, more than sixteen query heads on a key head, a head
# of 128 turned over its whole width, a long convolution of eleven taps
TE = model(64, 72, [layer("attention", attention(20, 1, 16, 4, 0.4, 30, 70, 16), dense(48)),
                    layer("attention", attention(2, 2, 128, 11, 0.1, 65, 1, 128), None),
                    layer("mlstm", mlstm(5, 8, 16, 3.0), dense(40)),
                    layer("attention", attention(8, 4, 24, 2, 0.3, 64, 64, 10), dense(48))], residual_mult=0.8, softcap=30.0)
CONFIGS = {"TA": (TA, 61), "TB": (TB, 62), "TC": (TC, 63), "TD": (TD, 64), "TE": (TE, 65)}


def write_model(config, folder, seed, embed_gain=40.0, head_gain=20.0, decided=False):
    """A folder with random weights; the token table's and the head's rows are made larger than usual (the first sublayers read the
    table's rows as they are), and no norm's weight is 1.  ``decided``: the routers' biases decide nearly every choice, so that
    rounding changes none."""
    import torch
    from safetensors.torch import load_file, save_file
    from torchinferno_b200.weights.random_init import write_random_model
    folder = write_random_model(config, folder, seed)
    path = str(folder) + "/model.safetensors"
    tensors = load_file(path)
    generator = torch.Generator().manual_seed(seed)
    for name, t in tensors.items():
        if name in ("embed", "head"):
            tensors[name] = (t.float() * (embed_gain if name == "embed" else head_gain)).to(t.dtype)
        elif decided and name.endswith((".router", ".router.b")):
            tensors[name] = (t.float() * (10.0 if name.endswith(".b") else 0.1)).to(t.dtype)
        elif "norm" in name:
            tensors[name] = (1 + 0.2 * torch.randn(t.shape, generator=generator)).to(t.dtype)
    save_file(tensors, path)
    return folder
