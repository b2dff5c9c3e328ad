from . import qwen2_moe, vekasun, difavik, fetezen, kopadra, pudizen, nolesun  # noqa: F401  (registration)
