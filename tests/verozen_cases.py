"""Small random Verozen configurations and weights for the tests."""
import torch


def experts(ff=40, count=12, top=3, groups=3, keep=2, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": count, "groups": {"count": groups, "keep": keep}, "scale": scale, "top": top}}


def gla(heads=3, dim=24, vdim=40, tau=8.0, rank=5, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}, "mlp": mlp}


def attention(heads=6, kv_heads=2, dim=40, rot_dims=12, base=2000.0, scale=0.21, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                                           "rot": {"base": base, "dims": rot_dims}}, "mlp": mlp}


def retention(heads=2, dim=24, vdim=56, rot_dims=16, base=300.0, mlp=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": [1 - 2.0 ** -(3 + 2 * h) for h in range(heads)],
                                           "rot": {"base": base, "dims": rot_dims}}, "mlp": mlp}


def config(layers=None, width=60, vocab=101, norm_groups=3, eps=1e-4, alpha=1.6, side_dim=9):
    return {"architecture": "Verozen", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": norm_groups}, "postln_alpha": alpha,
            "token_side": {"dim": side_dim},
            "layers": layers if layers is not None else [attention(mlp=experts()), gla(mlp=experts(24, 8, 1, 4, 1)), retention(), gla(2, 40, 24, 1.0, 11)]}


def tensor_shapes(c):
    """Checkpoint tensor name -> shape, from the configuration alone."""
    W, L, n = c["width"], len(c["layers"]), c["token_side"]["dim"]
    out = {"embed": (c["vocab"], W), "side.embed": (c["vocab"], L * n), "head": (c["vocab"], W), "final.norm": (W,)}
    for i, lay in enumerate(c["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        q = p + "mix."
        out.update({p + "norm1": (W,), p + "side.gate": (n, W), p + "side.proj": (W, n), p + "side.norm": (W,)})
        H, D, V = m["heads"], m["dim"], m["vdim"]
        out.update({q + "q": (H * D, W), q + "o": (W, H * V)})
        if lay["type"] == "attention":
            out.update({q + "k": (m["kv_heads"] * D, W), q + "q.norm": (D,), q + "k.norm": (D,), q + "temp": (H,), q + "pb": (H,)})
        else:
            out.update({q + "k": (H * D, W), q + "v": (H * V, W), q + "g": (H * V, W)})
        if lay["type"] == "gla":
            out.update({q + "norm": (V,), q + "a1": (m["rank"], W), q + "a2": (H * D, m["rank"]), q + "a2.b": (H * D,)})
        if lay["mlp"] is not None:
            E, ff = lay["mlp"]["router"]["experts"], lay["mlp"]["expert"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.router": (E, W), p + "mlp.correction": (E,)})
            for e in range(E):
                out.update({f"{p}mlp.e{e}.up": (ff, W), f"{p}mlp.e{e}.down": (W, ff)})
    return out


def weights(c, seed=0):
    """bfloat16 tensors; projections a little larger than usual, so that gates and sigmoids are reached on both sides."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(c).items():
        w = torch.randn(shape, generator=g)
        if "norm" in name:
            w = 1 + 0.2 * w
        elif name.endswith("a2.b"):
            w = 2 + 1.5 * w          # slow and fast decays
        elif name.endswith("temp"):
            w = 1 + 0.3 * w
        elif name.endswith("pb"):
            w = -2 + 0.5 * w
        elif name.endswith("correction"):
            w = 0.3 * w              # some choices are negative
        elif name.endswith("router"):
            w = 2.0 * w * shape[-1] ** -0.5
        elif name.endswith(".down"):
            w = 0.6 * w * shape[-1] ** -0.5   # where rounding sends a token to another expert, it is not thrown far
        elif "embed" not in name:
            w = 1.3 * w * shape[-1] ** -0.5
        out[name] = w.to(torch.bfloat16)
    # Keys of the linear-attention mixers lean towards their queries: where q.k is about zero at the first tokens, a head's
    # output almost vanishes, and its norm would blow up plain rounding to the size of the logits.
    for name in out:
        if name.endswith("mix.k") and name[:-1] + "v" in out:
            out[name] = (0.8 * out[name[:-1] + "q"].float() + 0.6 * out[name].float()).to(torch.bfloat16)
    return out


def build(c, w, device, dtype):
    from nanoquantization_b200.models import VerozenConfig, VerozenForCausalLM
    m = VerozenForCausalLM(VerozenConfig.from_dict(c), device=device, dtype=dtype)
    named = m.checkpoint_tensors()
    assert set(named) == set(w)
    for k, v in w.items():
        assert tuple(named[k].shape) == tuple(v.shape), k
        named[k].copy_(v)
    return m
