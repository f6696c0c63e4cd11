"""Small random Vemedra configurations and weights for the tests."""
import torch


def attention(heads=4, kv_heads=2, dim=24, vdim=40, chunk=13, rot_dims=16, base=5000.0, scale=0.3, softcap=7.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "rot": {"base": base, "dims": rot_dims},
            "scale": scale, "softcap": softcap}


def retention(heads=3, dim=20, vdim=28):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": [1 - 2.0 ** -(2 + 2 * h) for h in range(heads)]}


def parallel(ff=72, left=None, right=None, left_scale=0.7, right_scale=1.4, limit=1.3):
    return {"type": "parallel", "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit},
            "mixer": {"left": left or attention(), "right": right or retention(), "left_scale": left_scale, "right_scale": right_scale}}


def mingru(size=56, ff=None, limit=2.0):
    return {"type": "mingru", "mixer": {"width": size}, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers=None, width=48, vocab=97, taps=4, eps=1e-4, loop=(1, 3, 3)):
    c = {"architecture": "Vemedra", "width": width, "vocab": vocab, "canon": {"taps": taps}, "norm": {"eps": eps},
         "layers": layers if layers is not None else
         [parallel(ff=None), mingru(ff=40), parallel(left=attention(2, 2, 18, 10, 7, 18, 300.0), right=retention(1, 9, 33)), mingru(30)]}
    if loop is not None:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


def tensor_shapes(c):
    """Checkpoint tensor name -> shape, from the configuration alone."""
    W, taps = c["width"], c["canon"]["taps"]
    out = {"embed": (c["vocab"], W), "head": (c["vocab"], W), "final.norm": (W,)}
    if c.get("loop"):
        out["loop.step"] = (c["loop"]["times"], W)
    for i, lay in enumerate(c["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        out.update({p + "norm1": (W,), p + "canon1": (W, taps)})
        if lay["type"] == "mingru":
            n = m["width"]
            out.update({p + f"mix.{k}": (n, W) for k in "zxg"})
            out.update({p + "mix.z.b": (n,), p + "mix.x.b": (n,), p + "mix.o": (W, n)})
        else:
            a, r = m["left"], m["right"]
            q = p + "mix.left."
            out.update({q + "q": (a["heads"] * a["dim"], W), q + "k": (a["kv_heads"] * a["dim"], W), q + "v": (a["kv_heads"] * a["vdim"], W),
                        q + "sink": (a["heads"],), q + "o": (W, a["heads"] * a["vdim"])})
            q = p + "mix.right."
            out.update({q + "q": (r["heads"] * r["dim"], W), q + "k": (r["heads"] * r["dim"], W), q + "v": (r["heads"] * r["vdim"], W),
                        q + "g": (r["heads"] * r["vdim"], W), q + "o": (W, r["heads"] * r["vdim"])})
        if lay["mlp"] is not None:
            ff = lay["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "canon2": (W, taps), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def weights(c, seed=0):
    """bfloat16 tensors; projections a little larger than usual, so that gates, caps and clamps are reached."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(c).items():
        w = torch.randn(shape, generator=g)
        if "norm" in name:
            w = 1 + 0.2 * w
        elif "canon" in name:
            w = 0.4 * w
        elif name.endswith((".b", "sink")) or name == "loop.step":
            w = 0.5 * w
        elif name != "embed":
            w = 1.5 * w * shape[-1] ** -0.5
        out[name] = w.to(torch.bfloat16)
    # Keys of the retention lean towards its queries: where q.k is about zero at the first tokens, a head's output
    # almost vanishes, and its norm would blow up plain rounding to the size of the logits.
    for name in out:
        if name.endswith("right.k"):
            out[name] = (0.8 * out[name[:-1] + "q"].float() + 0.6 * out[name].float()).to(torch.bfloat16)
    return out


def build(c, w, device, dtype):
    from nanoquantization_b200.models import VemedraConfig, VemedraForCausalLM
    m = VemedraForCausalLM(VemedraConfig.from_dict(c), device=device, dtype=dtype)
    named = m.checkpoint_tensors()
    assert set(named) == set(w)
    for k, v in w.items():
        assert tuple(named[k].shape) == tuple(v.shape), k
        named[k].copy_(v)
    return m
