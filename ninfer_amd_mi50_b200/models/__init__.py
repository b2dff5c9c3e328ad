from . import qwen2_moe, vekasun, difavik, fetezen, kopadra, pudizen  # noqa: F401  (registration)
