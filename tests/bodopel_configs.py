"""Small Bodopel configurations for the tests: sizes that differ from one another in every place, values that happen to be 1
or equal to one another, windows shorter than a page and longer than any prompt, with and without a loop."""
from __future__ import annotations


def attention(heads, kv_heads, dim, vdim, scale, window, softcap):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
            "mask": None if window is None else {"size": window}}


def layer(mixer, ff):
    return {"type": "attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(vocab, width, taps, layers, loop=None, scale=6.0, eps=1e-5, max_positions=400):
    config = {"architecture": "Bodopel", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps},
              "embedding": {"scale": scale}, "canon": {"taps": taps}, "layers": layers}
    if loop is not None:
        config["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return config


# grouped heads with values wider than keys, a window of 20 in the middle of pages, a cap that bends most scores, a loop of
# two layers run twice, a layer without feed-forward inside the loop
BA = model(101, 64, 3, [layer(attention(4, 2, 16, 24, 0.4, 20, 2.0), 40), layer(attention(2, 2, 8, 8, 0.35, 33, 5.0), None),
                        layer(attention(4, 1, 24, 16, 0.2, 50, 30.0), 72), layer(attention(4, 2, 16, 24, 0.4, 20, 2.0), 24)], loop=(1, 3, 2))
# one head, a convolution of one tap (which carries nothing), no loop, no cap in one layer, a window of one token and one that
# sees everything, the last layer without feed-forward, sizes that are no multiple of 8
BB = model(131, 44, 1, [layer(attention(1, 1, 12, 20, 0.5, 1, 8.0), 36), layer(attention(3, 1, 6, 2, 0.4, None, None), 10),
                        layer(attention(1, 1, 20, 12, 0.3, 400, 3.0), None)], scale=1.0, eps=1e-6)
# nothing is a multiple of 4; the whole model is a loop of three passes; more taps than a two-token portion brings
BC = model(53, 50, 5, [layer(attention(6, 3, 10, 6, 0.3, 7, 4.0), 9), layer(attention(2, 1, 6, 14, 0.4, 64, 50.0), 30)], loop=(0, 2, 3))
# shapes of the tensor-core kernels: six query heads on one key head, as many key heads as query heads, a head of 128; a loop
# of one layer at the end, eight taps
BD = model(97, 96, 8, [layer(attention(6, 1, 40, 16, 0.3, 70, 6.0), 64), layer(attention(3, 3, 32, 32, 0.3, 64, 50.0), 96),
                       layer(attention(2, 1, 128, 104, 0.1, 65, 20.0), 128)], loop=(2, 3, 2), scale=10.0)
# many heads: twenty of them, each with keys of its own; forty on two key heads (more than sixteen query heads share one);
# a long convolution of eleven taps, a loop of one pass
BE = model(64, 72, 11, [layer(attention(20, 20, 8, 8, 0.5, 30, 10.0), 48), layer(attention(40, 2, 16, 8, 0.4, 40, 5.0), 48)], loop=(0, 1, 1))
CONFIGS = {"BA": (BA, 51), "BB": (BB, 52), "BC": (BC, 53), "BD": (BD, 54), "BE": (BE, 55)}


def write_model(config, folder, seed, embed_gain=25.0, head_gain=20.0):
    """A folder with random weights; the token table's and the head's rows are made larger than usual, so that tokens differ
    by as much as positions do and the logits are of a usual size."""
    from safetensors.torch import load_file, save_file
    from torchinferno_b200.weights.random_init import write_random_model
    folder = write_random_model(config, folder, seed)
    path = str(folder) + "/model.safetensors"
    tensors = load_file(path)
    tensors["embed"] = (tensors["embed"].float() * embed_gain).to(tensors["embed"].dtype)
    tensors["head"] = (tensors["head"].float() * head_gain).to(tensors["head"].dtype)
    save_file(tensors, path)
    return folder
