"""Device buffers of the kernel tests."""
import numpy as np

from oracle.finuvik_ref import round_bf16


class Dev:
    """Uploads arrays in the element type of a test and keeps them alive."""

    def __init__(self, torch, ob, kind):
        self.torch, self.keep = torch, []
        self.dtype = ob.F32 if kind == "f32" else ob.BF16
        self.t = torch.float32 if kind == "f32" else torch.bfloat16

    def up(self, a):
        x = self.torch.from_numpy(np.ascontiguousarray(a, np.float32)).cuda().to(self.t)
        self.keep.append(x)
        return x

    def f32(self, a):
        x = self.torch.from_numpy(np.ascontiguousarray(a, np.float32)).cuda()
        self.keep.append(x)
        return x

    def i32(self, a):
        x = self.torch.from_numpy(np.ascontiguousarray(a, np.int32)).cuda()
        self.keep.append(x)
        return x

    def zeros(self, *shape, f32=False):
        x = self.torch.zeros(*shape, device="cuda", dtype=self.torch.float32 if f32 else self.t)
        self.keep.append(x)
        return x


def host(x):
    return x.float().cpu().numpy().astype(np.float64)


def rounded(a, kind):
    a = np.asarray(a, np.float32)
    return (round_bf16(a) if kind == "bf16" else a).astype(np.float64)
